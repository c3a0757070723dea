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


def prefill_work(q_lens, context_lens, chunk: int = 0):
    """Work list of the prefill kernel: ``[(sequence, first row of q, rows, position of the first row)]``, a 128-row tile
    each, of every sequence with more than one new row; the tiles that see the most key tiles come first."""
    items, q0 = [], 0
    for b, (n, ctx) in enumerate(zip(q_lens, context_lens)):
        for r in range(0, n if n > 1 else 0, TILE):
            pos, rows = ctx - n + r, min(TILE, n - r)
            lo = pos - pos % chunk if chunk > 0 else 0
            items.append((lo // TILE - (pos + rows - 1) // TILE, (b, q0 + r, rows, pos)))
        q0 += n
    items.sort(key=lambda t: t[0])
    return [item for _, item in items]


# mean key tiles per query tile up to which the kernel's persistent form is used (``set_persistent_prefill`` fixes it)
_PERSISTENT_UP_TO = 8.0


def set_persistent_prefill(up_to: float) -> None:
    global _PERSISTENT_UP_TO
    _PERSISTENT_UP_TO = float(up_to)


def _work_on_device(cache, chunk: int):
    """The step's work list for ``chunk`` as an int32 device tensor, and whether the persistent form of the kernel runs it;
    made once per step (layers with the same chunk share it)."""
    work = cache.prefill_work.get(chunk)
    if work is None:
        items = prefill_work(cache.q_lens_host, cache.context_lens_host, chunk)
        keys = sum((p + n - 1) // TILE - (p - p % chunk if chunk > 0 else 0) // TILE + 1 for _, _, n, p in items)
        work = (torch.tensor(items, dtype=torch.int32).to(cache.block_tables.device), keys <= _PERSISTENT_UP_TO * len(items))
        cache.prefill_work[chunk] = work
    return work


def _reference(q, cache, layer, scale, chunk, sink, softcap, out, out_scale):
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
        v = _gather(cache.value_cache[layer], cache.block_tables[b], lens[b], cache.block_size).float()
        reps = Hq // k.shape[1]
        s = torch.einsum("qhd,khd->hqk", q[a:e].float(), k.repeat_interleave(reps, 1)) * scale
        if softcap > 0:
            s = softcap * torch.tanh(s / softcap)
        qp = torch.arange(lens[b] - (e - a), lens[b]).unsqueeze(1)
        kp = torch.arange(lens[b]).unsqueeze(0)
        hide = kp > qp
        if chunk > 0:
            hide = hide | (kp < qp - qp % chunk)
        s = s.masked_fill(hide, float("-inf"))
        if sink is not None:
            s = torch.cat((s, sink.float()[:, None, None].expand(Hq, e - a, 1)), dim=-1)
        p = torch.softmax(s, dim=-1)[..., :lens[b]]
        o = torch.einsum("hqk,khd->qhd", p, v.repeat_interleave(reps, 1)) * out_scale
        out[a:e] = o.reshape(e - a, -1).to(q.dtype)
    return out


def ragged_attention(q: torch.Tensor, cache, layer: int, scale: float, chunk: int = 0,
                     sink: Optional[torch.Tensor] = None, softcap: float = 0.0, out: Optional[torch.Tensor] = None,
                     out_scale: float = 1.0) -> torch.Tensor:
    """q ``[T, heads, dim]`` of the step's new tokens, whose keys and values are in the cache already → ``[T, heads *
    v_dim]``. ``chunk`` > 0: a position sees its own chunk of that many positions (counted from 0) only. ``sink [heads]``
    fp32: adds ``exp(sink)`` to the softmax denominator. ``softcap`` > 0: scores become ``softcap * tanh(score / softcap)``.
    ``out``: a matrix (any row pitch that keeps rows on 16 bytes) to write to; the result is multiplied by ``out_scale``."""
    kc, vc = cache.key_cache[layer], cache.value_cache[layer]
    T, Hq, D = q.shape
    Hkv, DV = vc.shape[2], vc.shape[3]
    softcap = float(softcap or 0.0)
    if out is None:
        out = torch.empty((T, Hq * DV), dtype=q.dtype, device=q.device)
    elif out.dtype != q.dtype or out.shape != (T, Hq * DV) or out.stride(1) != 1:
        raise TypeError("ragged_attention: out must be a [T, heads * v_dim] matrix of q's dtype with unit column stride")
    if not q.is_cuda:
        return _reference(q, cache, layer, scale, chunk, sink, softcap, out, out_scale)
    lib = _lib.get_lib()
    B, max_blocks = cache.block_tables.shape
    ragged = cache.is_prefill
    bs, nb = cache.block_size, kc.shape[0]
    cu = cache.cu_q_dev.data_ptr() if ragged else 0
    tables, lens, snk = cache.block_tables.data_ptr(), cache.context_lens.data_ptr(), _lib.ptr(sink)
    if q.dtype != torch.bfloat16 or out.stride(0) % 8 or out.data_ptr() % 16 \
            or not lib.mfb_paged_prefill_tc_supported(Hq, Hkv, D, DV, bs):
        rc = lib.mfb_paged_attention_any(q.data_ptr(), kc.data_ptr(), vc.data_ptr(), tables, lens, cu, snk, out.data_ptr(), T, B,
                                         Hq, Hkv, D, DV, bs, max_blocks, int(chunk), float(scale), softcap, out.stride(0),
                                         float(out_scale), int(q.dtype == torch.float32), _lib.stream_ptr())
        _lib.check(rc, "mfb_paged_attention_any")
        _lib.count_launch()
        return out
    status = _lib.status_word(q.device).data_ptr()
    if ragged and cache.n_long_rows:
        work, persistent = _work_on_device(cache, int(chunk))
        rc = lib.mfb_paged_prefill_tc(q.data_ptr(), kc.data_ptr(), vc.data_ptr(), work.data_ptr(), work.shape[0], int(persistent),
                                      tables, snk, out.data_ptr(), T, Hq, Hkv, D, DV, nb, bs, max_blocks, int(chunk),
                                      float(scale), softcap, out.stride(0), float(out_scale), status, _lib.stream_ptr())
        _lib.check(rc, "mfb_paged_prefill_tc")
        _lib.count_launch()
    if not ragged or cache.n_single_rows:
        reach = max_blocks * bs
        if chunk > 0:
            reach = min(reach, chunk + 128)          # a chunk may straddle one key tile more than it fills
        groups = -(-(Hq // Hkv) // 16)
        splits = lib.mfb_paged_decode_tc_splits(cache.n_single_rows if ragged else B, Hkv * groups, reach)
        need = lib.mfb_paged_decode_scratch_bytes(B, Hq, DV, splits)
        # the scratch of decode steps keeps its address once a step was captured; ragged steps, whose number of splits
        # varies, have one of their own
        name = "_ragged_scratch" if ragged else "_decode_scratch"
        scratch = getattr(cache, name, None)
        if scratch is None or scratch.numel() * 4 < need:
            scratch = torch.empty((need + 3) // 4, dtype=torch.float32, device=q.device)
            setattr(cache, name, scratch)
        rc = lib.mfb_paged_decode_attention_tc_ex(
            q.data_ptr(), kc.data_ptr(), vc.data_ptr(), tables, lens, cu, snk, out.data_ptr(), scratch.data_ptr(), splits, T, B,
            Hq, Hkv, D, DV, nb, bs, max_blocks, int(chunk), float(scale), softcap, out.stride(0), float(out_scale), status,
            _lib.stream_ptr())
        _lib.check(rc, "mfb_paged_decode_attention_tc_ex")
        _lib.count_launch(2)
    return out
