"""Attention of a ragged batch over the paged cache, without host work per sequence.

The batch is described by the step's metadata in ``KVCacheContext``: ``cu_q`` row boundaries, context lengths, block
tables. Rows of sequences with one new token run on the decode kernel, all others on the prefill kernel (two launches
into one result, whichever are needed); 32-bit caches and head sizes outside the tensor-core kernels' range run on
``paged_attention_any``. In a decode step every sequence has one row and no boundaries are needed, so that the step can
be captured in a CUDA graph.
"""
from __future__ import annotations

from typing import Optional

import torch

from ..ops import _lib

TILE = 128               # query rows of a tile of the prefill kernel


def first_visible(pos: int, chunk: int = 0, window: int = 0) -> int:
    """The first position that a token at ``pos`` sees."""
    lo = pos - pos % chunk if chunk > 0 else 0
    return max(lo, pos - window + 1) if window > 0 else lo


def prefill_work(q_lens, context_lens, chunk: int = 0, window: int = 0):
    """Work list of the prefill kernel: ``[(sequence, first row of q, rows, position of the first row)]``, a 128-row tile
    each, of every sequence with more than one new row; the tiles that see the most key tiles come first."""
    items, q0 = [], 0
    for b, (n, ctx) in enumerate(zip(q_lens, context_lens)):
        for r in range(0, n if n > 1 else 0, TILE):
            pos, rows = ctx - n + r, min(TILE, n - r)
            items.append((first_visible(pos, chunk, window) // TILE - (pos + rows - 1) // TILE, (b, q0 + r, rows, pos)))
        q0 += n
    items.sort(key=lambda t: t[0])
    return [item for _, item in items]


# mean key tiles per query tile up to which the kernel's persistent form is used (``set_persistent_prefill`` fixes it)
_PERSISTENT_UP_TO = 8.0


def set_persistent_prefill(up_to: float) -> None:
    global _PERSISTENT_UP_TO
    _PERSISTENT_UP_TO = float(up_to)


def _work_tensor(items, chunk: int, window: int, device):
    """A work list as an int32 device tensor, and whether the persistent form of the kernel runs it."""
    keys = sum((p + n - 1) // TILE - first_visible(p, chunk, window) // TILE + 1 for _, _, n, p in items)
    return torch.tensor(items, dtype=torch.int32).to(device), keys <= _PERSISTENT_UP_TO * len(items)


def _work_on_device(cache, chunk: int, window: int):
    """The step's work list; made once per step (layers with the same mask share it)."""
    work = cache.prefill_work.get((chunk, window))
    if work is None:
        items = prefill_work(cache.q_lens_host, cache.context_lens_host, chunk, window)
        work = cache.prefill_work[(chunk, window)] = _work_tensor(items, chunk, window, cache.block_tables.device)
    return work


def _values(cache, layer: int):
    """The layer's value cache: its keys, where it has no values of its own."""
    return cache.key_cache[layer] if cache.value_cache[layer] is None else cache.value_cache[layer]


def _reference(q, cache, layer, scale, chunk, sink, softcap, out, out_scale, window, all_values):
    """Plain PyTorch body for CPU tensors."""
    from .paged_attention import _gather
    B = cache.context_lens.shape[0]
    cu = cache.cu_q if cache.is_prefill else list(range(B + 1))
    lens = cache.context_lens.tolist()
    Hq = q.shape[1]
    out.zero_()
    for b in range(B):
        a, e = cu[b], cu[b + 1]
        if e == a or lens[b] <= 0:
            continue
        k = _gather(cache.key_cache[layer], cache.block_tables[b], lens[b], cache.block_size).float()
        v = _gather(_values(cache, layer), cache.block_tables[b], lens[b], cache.block_size).float()
        reps = Hq // k.shape[1]
        s = torch.einsum("qhd,khd->hqk", q[a:e].float(), k.repeat_interleave(reps, 1)) * scale
        if softcap > 0:
            s = softcap * torch.tanh(s / softcap)
        qp = torch.arange(lens[b] - (e - a), lens[b]).unsqueeze(1)
        kp = torch.arange(lens[b]).unsqueeze(0)
        hide = kp > qp
        if chunk > 0:
            hide = hide | (kp < qp - qp % chunk)
        if window > 0:
            hide = hide | (kp <= qp - window)
        s = s.masked_fill(hide, float("-inf"))
        if sink is not None:
            s = torch.cat((s, sink.float()[:, None, None].expand(Hq, e - a, 1)), dim=-1)
        p = torch.softmax(s, dim=-1)[..., :lens[b]]
        if all_values:
            o = torch.einsum("hqk,kgd->qhgd", p, v) * out_scale
        else:
            o = torch.einsum("hqk,khd->qhd", p, v.repeat_interleave(reps, 1)) * out_scale
        out[a:e] = o.reshape(e - a, -1).to(q.dtype)
    return out


def _prefill_tc(lib, q, k, ld_k, k_heads, k_rows, v, ld_v, work, persistent, tables, sink, out, D, DV, block_size, chunk, window,
                all_values, scale, softcap, out_scale):
    """One launch of the tensor-core prefill kernel; ``k`` / ``v`` are addresses of ``[k_rows, k_heads, D | DV]``, rows ``ld_k`` /
    ``ld_v`` elements apart."""
    T, Hq = q.shape[0], q.shape[1]
    rc = lib.mfb_paged_prefill_tc(q.data_ptr(), k, v, work.data_ptr(), work.shape[0], int(persistent), tables.data_ptr(),
                                  _lib.ptr(sink), out.data_ptr(), T, Hq, k_heads, D, DV, k_rows // block_size, block_size,
                                  tables.shape[1], int(chunk), int(window), int(all_values), ld_k, ld_v, float(scale), softcap,
                                  out.stride(0), float(out_scale), _lib.status_word(q.device).data_ptr(), _lib.stream_ptr())
    _lib.check(rc, "mfb_paged_prefill_tc")
    _lib.count_launch()


def _scratch(cache, name: str, need: int, device):
    """The scratch of decode steps keeps its address once a step was captured; ragged steps, whose number of splits varies,
    have one of their own."""
    buf = getattr(cache, name, None)
    if buf is None or buf.numel() * 4 < need:
        buf = torch.empty((need + 3) // 4, dtype=torch.float32, device=device)
        setattr(cache, name, buf)
    return buf


def ragged_attention(q: torch.Tensor, cache, layer: int, scale: float, chunk: int = 0,
                     sink: Optional[torch.Tensor] = None, softcap: float = 0.0, out: Optional[torch.Tensor] = None,
                     out_scale: float = 1.0, window: int = 0, all_values: bool = False, singles: bool = True) -> torch.Tensor:
    """q ``[T, heads, dim]`` of the step's new tokens, whose keys and values are in the cache already → ``[T, heads *
    v_dim]``. ``chunk`` > 0: a position sees its own chunk of that many positions (counted from 0) only; ``window`` > 0: it sees
    itself and the ``window - 1`` positions before it. ``sink [heads]`` fp32: adds ``exp(sink)`` to the softmax denominator.
    ``softcap`` > 0: scores become ``softcap * tanh(score / softcap)``. ``all_values``: every head's weights are applied to the
    values of every key / value head: ``[T, heads * kv_heads * v_dim]``. A layer without values of its own attends over its keys.
    ``singles`` False: the result of sequences with one new row in a ragged step may be left undefined.
    ``out``: a matrix (any row pitch that keeps rows on 16 bytes) to write to; the result is multiplied by ``out_scale``."""
    kc, vc = cache.key_cache[layer], _values(cache, layer)
    T, Hq, D = q.shape
    Hkv, DV = vc.shape[2], vc.shape[3]
    softcap, V = float(softcap or 0.0), Hkv if all_values else 1
    if out is None:
        out = torch.empty((T, Hq * V * DV), dtype=q.dtype, device=q.device)
    elif out.dtype != q.dtype or out.shape != (T, Hq * V * DV) or out.stride(1) != 1:
        raise TypeError("ragged_attention: out must be a [T, heads * v_dim] matrix of q's dtype with unit column stride")
    if not q.is_cuda:
        return _reference(q, cache, layer, scale, chunk, sink, softcap, out, out_scale, window, all_values)
    if not q.is_contiguous():
        raise TypeError("ragged_attention: q must be contiguous")
    lib = _lib.get_lib()
    B, max_blocks = cache.block_tables.shape
    ragged = cache.is_prefill
    bs, nb = cache.block_size, kc.shape[0]
    cu = cache.cu_q_dev.data_ptr() if ragged else 0
    tables, lens, snk = cache.block_tables.data_ptr(), cache.context_lens.data_ptr(), _lib.ptr(sink)
    if q.dtype != torch.bfloat16 or out.stride(0) % 8 or out.data_ptr() % 16 \
            or not lib.mfb_paged_prefill_tc_supported(Hq, Hkv, D, DV, bs):
        rc = lib.mfb_paged_attention_any(q.data_ptr(), kc.data_ptr(), vc.data_ptr(), tables, lens, cu, snk, out.data_ptr(), T, B,
                                         Hq, Hkv, D, DV, bs, max_blocks, int(chunk), int(window), int(all_values), float(scale),
                                         softcap, out.stride(0), float(out_scale), int(q.dtype == torch.float32), _lib.stream_ptr())
        _lib.check(rc, "mfb_paged_attention_any")
        _lib.count_launch()
        return out
    status = _lib.status_word(q.device).data_ptr()
    if ragged and cache.n_long_rows:
        work, persistent = _work_on_device(cache, int(chunk), int(window))
        _prefill_tc(lib, q, kc.data_ptr(), Hkv * D, Hkv, nb * bs, vc.data_ptr(), Hkv * DV, work, persistent, cache.block_tables, sink,
                    out, D, DV, bs, chunk, window, all_values, scale, softcap, out_scale)
    if not ragged or (cache.n_single_rows and singles):
        reach = max_blocks * bs
        for span in (chunk, window):
            if span > 0:
                reach = min(reach, span + 128)          # it may straddle one key tile more than it fills
        groups = -(-(Hq // Hkv) // 16)
        splits = lib.mfb_paged_decode_tc_splits(cache.n_single_rows if ragged else B, Hkv * groups * V, reach)
        need = lib.mfb_paged_decode_scratch_bytes(B, Hq * V, DV, splits)
        scratch = _scratch(cache, "_ragged_scratch" if ragged else "_decode_scratch", need, q.device)
        rc = lib.mfb_paged_decode_attention_tc_ex(
            q.data_ptr(), kc.data_ptr(), vc.data_ptr(), tables, lens, cu, snk, out.data_ptr(), scratch.data_ptr(), splits, T, B,
            Hq, Hkv, D, DV, nb, bs, max_blocks, int(chunk), int(window), int(all_values), float(scale), softcap, out.stride(0),
            float(out_scale), status, _lib.stream_ptr())
        _lib.check(rc, "mfb_paged_decode_attention_tc_ex")
        _lib.count_launch(2)
    return out


def talking_attention(q: torch.Tensor, cache, layer: int, scale: float, talk: torch.Tensor, gate: Optional[torch.Tensor] = None,
                      window: int = 0) -> torch.Tensor:
    """Attention whose softmax weights are mixed over heads (head h uses ``sum_g talk[h, g] weights_g`` on the values of its own
    key / value head), times ``sigmoid(gate)``: q ``[T, heads, dim]``, talk ``[heads, heads]`` fp32, gate ``[T, heads * v_dim]`` →
    ``[T, heads * v_dim]``. Decoded rows are one kernel and its merge; portions apply every head's weights to the values of every
    key / value head and mix the results."""
    from ..ops import stream
    T, H, D = q.shape
    G, DV = cache.value_cache[layer].shape[2:]
    lib = _lib.get_lib() if q.is_cuda else None
    fused = lib is not None and q.dtype == torch.bfloat16 and lib.mfb_paged_talk_decode_supported(H, G, D, DV, cache.block_size)
    if cache.is_prefill or not fused:
        o = ragged_attention(q, cache, layer, scale, window=window, all_values=True, singles=not fused)
        out = stream.talk_mix(o.view(T, H, G, DV), talk, gate)
        if not fused or not cache.n_single_rows:
            return out
    else:
        out = torch.empty((T, H * DV), dtype=q.dtype, device=q.device)
    if gate is not None and (gate.dtype != q.dtype or gate.shape != out.shape or gate.stride(1) != 1):
        raise TypeError("talking_attention: the gate must be a [T, heads * v_dim] matrix of q's dtype with unit column stride")
    kc, vc = cache.key_cache[layer], cache.value_cache[layer]
    B, max_blocks = cache.block_tables.shape
    reach = max_blocks * cache.block_size if window <= 0 else min(max_blocks * cache.block_size, window + 128)
    splits = lib.mfb_paged_talk_decode_splits(cache.n_single_rows if cache.is_prefill else B, reach)
    scratch = _scratch(cache, "_ragged_talk_scratch" if cache.is_prefill else "_talk_scratch",
                       lib.mfb_paged_talk_decode_scratch_bytes(B, H, G, DV, splits), q.device)
    rc = lib.mfb_paged_talk_decode(q.data_ptr(), kc.data_ptr(), vc.data_ptr(), cache.block_tables.data_ptr(),
                                   cache.context_lens.data_ptr(), cache.cu_q_dev.data_ptr() if cache.is_prefill else 0, talk.data_ptr(),
                                   _lib.ptr(gate), 0 if gate is None else gate.stride(0), out.data_ptr(), scratch.data_ptr(), splits, T,
                                   B, H, G, D, DV, kc.shape[0], cache.block_size, max_blocks, int(window), float(scale),
                                   _lib.status_word(q.device).data_ptr(), _lib.stream_ptr())
    _lib.check(rc, "mfb_paged_talk_decode")
    _lib.count_launch(2)
    return out


# ---- latent attention: the cache holds one latent per token, keys and values are linear in it -----------------------------------
class _Rows:
    """Some rows of a step as a decode step of their own (one row per sequence)."""
    is_prefill = False

    def __init__(self, cache, seqs, rows):
        self.block_size, self.key_cache, self.value_cache = cache.block_size, cache.key_cache, cache.value_cache
        device = cache.block_tables.device
        self.rows = torch.tensor(rows, dtype=torch.int64).to(device)
        seqs = torch.tensor(seqs, dtype=torch.int64).to(device)
        self.block_tables, self.context_lens = cache.block_tables[seqs], cache.context_lens[seqs]
        self.n_single_rows = len(rows)


def _single_rows(cache) -> _Rows:
    """The sequences of a ragged step with one new row; made once per step."""
    rows = cache.prefill_work.get("single")
    if rows is None:
        seqs = [b for b, n in enumerate(cache.q_lens_host) if n == 1]
        rows = cache.prefill_work["single"] = _Rows(cache, seqs, [cache.cu_q[b] for b in seqs])
    return rows


def _expansion(cache, window: int):
    """Which cached rows the step's portions see, laid out sequence by sequence in pages of their own: ``(rows of the cache,
    block tables of the copy, work list, persistent)``; made once per step and window."""
    plan = cache.prefill_work.get(("latent", window))
    if plan is None:
        bs, dev = cache.block_size, cache.block_tables.device
        items, rows, tables, at, q0 = [], [], [], 0, 0
        within = torch.arange(bs, device=dev)
        for b, (n, ctx) in enumerate(zip(cache.q_lens_host, cache.context_lens_host)):
            own = torch.zeros(0, dtype=torch.int32)
            if n > 1:
                base = first_visible(ctx - n, 0, window) // TILE * TILE
                blocks = cache.block_tables[b, base // bs:-(-ctx // bs)].long()
                rows.append((blocks[:, None] * bs + within).reshape(-1))
                own = torch.arange(at, at + blocks.numel(), dtype=torch.int32)
                at += blocks.numel()
                items += [(b, q0 + r, min(TILE, n - r), ctx - n + r - base) for r in range(0, n, TILE)]
            tables.append(own)
            q0 += n
        width = max(1, max(t.numel() for t in tables))
        table = torch.stack([torch.nn.functional.pad(t, (0, width - t.numel())) for t in tables]).to(dev)
        items.sort(key=lambda t: first_visible(t[3], 0, window) // TILE - (t[3] + t[2] - 1) // TILE)
        plan = cache.prefill_work[("latent", window)] = (torch.cat(rows), table) + _work_tensor(items, 0, window, dev)
    return plan


def _absorbed(q, cache, layer, w_uk, w_uv, scale, window, sink):
    """Queries through the key factor, attention over the cached rows themselves, results through the value factor, which may act
    on fewer columns: ``[T, heads * v_dim]``."""
    T, H = q.shape[0], q.shape[1]
    R, DV, RV = w_uk.shape[2], w_uv.shape[1], w_uv.shape[2]
    q_lat = torch.empty((T, H, R), dtype=q.dtype, device=q.device)
    torch.bmm(q.transpose(0, 1), w_uk, out=q_lat.transpose(0, 1))
    lib = _lib.get_lib() if q.is_cuda else None
    if lib is not None and q.dtype == torch.bfloat16 and not cache.is_prefill \
            and lib.mfb_latent_decode_supported(R, RV, cache.block_size):
        o_lat = torch.empty((T, H, RV), dtype=q.dtype, device=q.device)
        B, max_blocks = cache.block_tables.shape
        reach = max_blocks * cache.block_size if window <= 0 else min(max_blocks * cache.block_size, window + 128)
        splits = lib.mfb_latent_decode_splits(B, H, reach)
        scratch = _scratch(cache, "_latent_scratch", lib.mfb_latent_decode_scratch_bytes(B, H, RV, splits), q.device)
        kc = cache.key_cache[layer]
        rc = lib.mfb_latent_decode(q_lat.data_ptr(), kc.data_ptr(), cache.block_tables.data_ptr(), cache.context_lens.data_ptr(),
                                   _lib.ptr(sink), o_lat.data_ptr(), scratch.data_ptr(), splits, B, H, R, RV, kc.shape[0],
                                   cache.block_size, max_blocks, int(window), float(scale),
                                   _lib.status_word(q.device).data_ptr(), _lib.stream_ptr())
        _lib.check(rc, "mfb_latent_decode")
        _lib.count_launch(2)
    else:
        o_lat = ragged_attention(q_lat, cache, layer, scale, sink=sink, window=window).view(T, H, R)[:, :, :RV]
    out = torch.empty((T, H, DV), dtype=q.dtype, device=q.device)
    torch.bmm(o_lat.transpose(0, 1), w_uv.transpose(1, 2), out=out.transpose(0, 1))
    return out.view(T, H * DV)


def latent_attention(q: torch.Tensor, cache, layer: int, w_kv: torch.Tensor, v_dim: int, scale: float, window: int = 0,
                     sink: Optional[torch.Tensor] = None, v_rank: Optional[int] = None) -> torch.Tensor:
    """q ``[T, heads, dim]`` against cached latents ``[.., 1, rank]``, of which the first ``heads * dim`` rows of ``w_kv [heads *
    (dim + v_dim), rank]`` make the keys and the others the values (of the first ``v_rank`` columns alone, where the cached rows
    also hold a key part) → ``[T, heads * v_dim]``. Decoded rows attend over the latents (the factors are absorbed into query and
    result); portions expand the keys and values that they see, once per call."""
    T, H, D = q.shape
    R = w_kv.shape[1]
    w_uk, w_uv = w_kv[:H * D].view(H, D, R), w_kv[H * D:].view(H, v_dim, R)[:, :, :v_rank]
    lib = _lib.get_lib() if q.is_cuda else None
    expand = lib is not None and q.dtype == torch.bfloat16 and cache.is_prefill and cache.n_long_rows \
        and lib.mfb_paged_prefill_tc_wide_supported(H, H, D, v_dim, cache.block_size)
    if not expand:
        return _absorbed(q, cache, layer, w_uk, w_uv, scale, window, sink)
    from ..ops import functional as Fn
    out = torch.empty((T, H * v_dim), dtype=q.dtype, device=q.device)
    rows, tables, work, persistent = _expansion(cache, int(window))
    kv = Fn.linear(cache.key_cache[layer].view(-1, R).index_select(0, rows), w_kv)
    if not q.is_contiguous():
        q = q.contiguous()
    _prefill_tc(lib, q, kv.data_ptr(), kv.stride(0), H, kv.shape[0], kv.data_ptr() + 2 * H * D, kv.stride(0), work, persistent, tables,
                sink, out, D, v_dim, cache.block_size, 0, window, False, scale, 0.0, 1.0)
    if cache.n_single_rows:
        single = _single_rows(cache)
        out[single.rows] = _absorbed(q[single.rows], single, layer, w_uk, w_uv, scale, window, sink)
    return out
