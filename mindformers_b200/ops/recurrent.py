"""Recurrent mixers over ragged batches: the gated delta rule (short convolutions, unit keys, decays, the recurrence, its norm
and gate), the matrix memory (capped log gates, running maximum, memory and normaliser, norm and gate) and the state space with a
scalar decay per head (short convolution, step sizes, the recurrence, gate and grouped norm).

``delta_rule``, ``matrix_memory`` and ``state_space`` have two bodies like the ops of ``functional.py``: the sm_100a kernels
(``csrc/delta_rule.cu``, ``csrc/matrix_memory.cu``, ``csrc/state_space.cu``), always taken for CUDA tensors (bf16 or fp32
activations; state and recurrence are fp32), and a plain PyTorch body for CPU tensors. They are inference ops: they advance the
state in place and have no gradients.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Tuple

import torch
import torch.nn.functional as F

from . import _lib


@dataclass
class DeltaWeights:
    """Per-layer weights beside the projections, all fp32: ``conv [taps, 2 G D + H DV]`` (q, k, v channels; the last row
    belongs to the current token), ``a_log [H]``, ``dt_bias [H]`` or ``[H D]`` (decays per key channel), ``norm [DV]``."""
    conv: torch.Tensor
    a_log: torch.Tensor
    dt_bias: torch.Tensor
    norm: torch.Tensor


@dataclass
class DeltaShape:
    heads: int
    kv_heads: int
    dim: int
    v_dim: int
    taps: int
    by_channel: bool         # one decay per head and key channel (else per head)
    gate_silu: bool          # the read-out's gate is silu (else sigmoid)

    @property
    def channels(self) -> int:
        return 2 * self.kv_heads * self.dim + self.heads * self.v_dim


def _rows(t: torch.Tensor, dtype, rows: int, cols: int, what: str):
    if t.dtype != dtype or t.dim() != 2 or t.shape[0] != rows or t.shape[1] < cols or t.stride(1) != 1:
        raise TypeError(f"{what} must be a {dtype} matrix of {rows} rows and at least {cols} columns with unit stride")


def _sequences(cache, T: int):
    """``(slot, first row, rows, position of the first row)`` of every sequence with rows in the step."""
    lens = cache.context_lens.tolist()
    if cache.is_prefill:
        cu = cache.cu_q
        return [(b, cu[b], cu[b + 1] - cu[b], lens[b] - (cu[b + 1] - cu[b])) for b in range(len(lens)) if cu[b + 1] > cu[b]]
    slots = cache.slot_mapping.tolist()
    return [(b, b, 1, lens[b] - 1) for b in range(T) if slots[b] >= 0]


def _reference(x, b, a, gate, w: DeltaWeights, s: DeltaShape, ring, state, cache, eps, out, out_scale):
    H, G, D, DV = s.heads, s.kv_heads, s.dim, s.v_dim
    if not cache.is_prefill:
        out.zero_()
    for slot, r0, n, start in _sequences(cache, x.shape[0]):
        rows = slice(r0, r0 + n)
        xs = x[rows, :s.channels]
        before = torch.zeros(s.taps - 1, s.channels, dtype=torch.float32)
        for d in range(1, s.taps):
            if start - d >= 0:
                before[s.taps - 1 - d] = ring[slot, (start - d) % s.taps].float()
        seq = torch.cat((before, xs.float()))
        y = F.silu(sum(seq[j:j + n] * w.conv[j] for j in range(s.taps)))
        for p in range(max(start, start + n - s.taps), start + n):
            ring[slot, p % s.taps] = xs[p - start]
        q, k, v = y[:, :G * D].view(n, G, D), y[:, G * D:2 * G * D].view(n, G, D), y[:, 2 * G * D:].view(n, H, DV)
        q = q * torch.rsqrt(q.pow(2).sum(-1, keepdim=True) + 1e-6) * D ** -0.5
        k = k * torch.rsqrt(k.pow(2).sum(-1, keepdim=True) + 1e-6)
        q, k = q.repeat_interleave(H // G, 1), k.repeat_interleave(H // G, 1)
        raw = a[rows, :w.dt_bias.numel()].float() + w.dt_bias
        g = torch.exp(-torch.exp(w.a_log)[:, None] * F.softplus(raw).view(n, H, -1)).expand(n, H, D)
        beta = torch.sigmoid(b[rows, :H].float())
        S = state[slot].clone() if start > 0 else torch.zeros(H, D, DV)
        o = torch.empty(n, H, DV)
        for t in range(n):
            S = S * g[t, :, :, None]
            u = beta[t, :, None] * (v[t] - (S * k[t, :, :, None]).sum(1))
            S = S + k[t, :, :, None] * u[:, None]
            o[t] = (S * q[t, :, :, None]).sum(1)
        state[slot] = S
        o = o * torch.rsqrt(o.pow(2).mean(-1, keepdim=True) + eps) * w.norm
        z = gate[rows, :H * DV].float().view(n, H, DV)
        z = F.silu(z) if s.gate_silu else torch.sigmoid(z)
        out[rows] = (o * z * out_scale).reshape(n, H * DV).to(out.dtype)


def delta_rule(x: torch.Tensor, b: torch.Tensor, a: torch.Tensor, gate: torch.Tensor, w: DeltaWeights, s: DeltaShape,
               state: Tuple[torch.Tensor, torch.Tensor], cache, eps: float, out: Optional[torch.Tensor] = None,
               out_scale: float = 1.0) -> torch.Tensor:
    """``x [T, channels]`` (inputs of the convolutions: q | k | v), ``b [T, H]`` (raw step size), ``a [T, H]`` or ``[T, H D]``
    (raw decay), ``gate [T, H DV]``, all of the step's rows in the order of ``cache`` (``KVCacheContext``), with any row
    pitch; ``state``: the layer's ``(S [slots, H, D, DV] fp32, ring [slots, taps, channels])``, advanced in place. Returns
    (in ``out``, when given) ``[T, H DV]``: the gated, normalised read-out times ``out_scale``."""
    T, dtype = x.shape[0], x.dtype
    S, ring = state
    H, G, D, DV = s.heads, s.kv_heads, s.dim, s.v_dim
    if out is None:
        out = torch.empty((T, H * DV), dtype=dtype, device=x.device)
    if not x.is_cuda:
        _reference(x, b, a, gate, w, s, ring, S, cache, eps, out, out_scale)
        return out
    if dtype not in (torch.bfloat16, torch.float32):
        raise TypeError(f"bfloat16 or float32 activations expected, got {dtype}")
    for t, cols, what in ((x, s.channels, "x"), (b, H, "b"), (a, H * D if s.by_channel else H, "a"), (gate, H * DV, "gate"),
                          (out, H * DV, "out")):
        _rows(t, dtype, T, cols, what)
    slots_n = S.shape[0]
    if tuple(S.shape[1:]) != (H, D, DV) or S.dtype != torch.float32 or not S.is_contiguous() \
            or tuple(ring.shape) != (slots_n, s.taps, s.channels) or ring.dtype != dtype or not ring.is_contiguous():
        raise TypeError("delta_rule: the state does not have the layer's shape")
    if b.stride(0) != x.stride(0) or cache.context_lens.numel() > slots_n:
        raise ValueError("delta_rule: b must share the row pitch of x, and every sequence needs a state slot")
    for t, n in ((w.conv, s.taps * s.channels), (w.a_log, H), (w.dt_bias, H * D if s.by_channel else H), (w.norm, DV)):
        if t.dtype != torch.float32 or t.numel() != n or not t.is_contiguous():
            raise TypeError("delta_rule: weights beside the projections are contiguous fp32 tensors")
    lib = _lib.get_lib()
    B = cache.context_lens.numel()
    decode = not cache.is_prefill and lib.mfb_delta_decode_supported(D, DV)
    cu = 0
    if cache.is_prefill:
        cu = cache.cu_q_dev.data_ptr()
    elif not decode:          # one row per slot, as portions: idle slots run on rows nobody reads, so their state is kept aside
        return _decode_as_portions(x, b, a, gate, w, s, state, cache, eps, out, out_scale)
    scratch = 0
    if not decode:
        need = lib.mfb_delta_scratch_floats(T, H, G, D, DV, int(s.by_channel))
        buf = torch.empty(need, dtype=torch.float32, device=x.device)
        scratch = buf.data_ptr()
    _launch(lib, x, b, a, gate, w, s, ring, S, cu, cache.context_lens, cache.slot_mapping, scratch, out, T, B, eps, out_scale)
    _lib.count_launch(1 if decode else 4)
    return out


def _launch(lib, x, b, a, gate, w, s, ring, S, cu, lens, slots, scratch, out, T, B, eps, out_scale):
    rc = lib.mfb_delta_rule(
        x.data_ptr(), x.stride(0), b.data_ptr(), a.data_ptr(), a.stride(0), gate.data_ptr(), gate.stride(0), w.conv.data_ptr(),
        w.a_log.data_ptr(), w.dt_bias.data_ptr(), w.norm.data_ptr(), ring.data_ptr(), S.data_ptr(), cu, lens.data_ptr(),
        slots.data_ptr(), scratch, out.data_ptr(), out.stride(0), T, B, s.heads, s.kv_heads, s.dim, s.v_dim, s.taps,
        int(s.by_channel), int(s.gate_silu), float(eps), float(out_scale), int(x.dtype == torch.float32), _lib.stream_ptr())
    _lib.check(rc, "mfb_delta_rule")


def _decode_as_portions(x, b, a, gate, w, s, state, cache, eps, out, out_scale):
    """A decode step of head sizes that the one-kernel step does not take: portions of one row. Idle slots would advance
    too, so they get their state back (no host read: the step may be captured in a graph)."""
    lib = _lib.get_lib()
    S, ring = state
    B = cache.context_lens.numel()
    idle = cache.slot_mapping[:B] < 0
    keep = S[:B].clone(), ring[:B].clone()
    cu = getattr(cache, "_unit_rows", None)
    if cu is None or cu.numel() != B + 1:
        cu = cache._unit_rows = torch.arange(B + 1, dtype=torch.int32, device=x.device)
    buf = torch.empty(lib.mfb_delta_scratch_floats(B, s.heads, s.kv_heads, s.dim, s.v_dim, int(s.by_channel)), dtype=torch.float32,
                      device=x.device)
    lens = cache.context_lens.clamp(min=1)
    _launch(lib, x, b, a, gate, w, s, ring, S, cu.data_ptr(), lens, cache.slot_mapping, buf.data_ptr(), out, B, B, eps, out_scale)
    _lib.count_launch(4)
    S[:B].copy_(torch.where(idle[:, None, None, None], keep[0], S[:B]))
    ring[:B].copy_(torch.where(idle[:, None, None], keep[1], ring[:B]))
    return out


# ---- matrix memory ------------------------------------------------------------------------------------------------------------
@dataclass
class MemoryShape:
    heads: int
    dim: int
    v_dim: int
    gate_cap: float


def _memory_reference(proj, bi, bf, norm, s: MemoryShape, state, cache, eps, out):
    H, D, DV, cap = s.heads, s.dim, s.v_dim, s.gate_cap
    S_all, n_all, m_all = state
    if not cache.is_prefill:
        out.zero_()
    for slot, r0, n, start in _sequences(cache, proj.shape[0]):
        rows = slice(r0, r0 + n)
        q, k, v, z, i, f = torch.split(proj[rows].float(), (H * D, H * D, H * DV, H * DV, H, H), dim=1)
        q, k, v = q.view(n, H, D) * D ** -0.5, k.view(n, H, D), v.view(n, H, DV)
        i = cap * torch.tanh((i + bi) / cap)
        f = F.logsigmoid(cap * torch.tanh((f + bf) / cap))
        S, nv, m = (t[slot].clone() if start > 0 else torch.zeros_like(t[slot]) for t in state)
        o = torch.empty(n, H, DV)
        for t in range(n):
            new = torch.maximum(f[t] + m, i[t])
            keep, put = torch.exp(f[t] + m - new), torch.exp(i[t] - new)
            S = keep[:, None, None] * S + (put[:, None] * k[t])[:, :, None] * v[t][:, None]
            nv = keep[:, None] * nv + put[:, None] * k[t]
            m = new
            size = torch.maximum((nv * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
            o[t] = (S * q[t][:, :, None]).sum(1) / size[:, None]
        S_all[slot], n_all[slot], m_all[slot] = S, nv, m
        o = o * torch.rsqrt(o.pow(2).mean(-1, keepdim=True) + eps) * norm.view(H, DV)
        out[rows] = (o.reshape(n, H * DV) * torch.sigmoid(z)).to(out.dtype)


def matrix_memory(proj: torch.Tensor, input_bias: torch.Tensor, forget_bias: torch.Tensor, norm: torch.Tensor, s: MemoryShape,
                  state: Tuple[torch.Tensor, torch.Tensor, torch.Tensor], cache, eps: float) -> torch.Tensor:
    """``proj [T, >= 2 H D + 2 H DV + 2 H]`` (q | k | v | output gate | input gate | forget gate, any row pitch), all of the step's
    rows in the order of ``cache`` (``KVCacheContext``). Per head, with ``q`` times ``D ** -0.5`` and the log gates ``i = cap
    tanh((x_i + b_i) / cap)``, ``f = log_sigmoid(cap tanh((x_f + b_f) / cap))``::

        m' = max(f + m, i);  S' = e^(f + m - m') S + e^(i - m') k v^T;  n' the same with k alone
        o  = S'^T q / (max(|n' . q|, e^(-m')) + 1e-6)

    Returns ``[T, H DV]``: ``o`` RMS-normed per head, times ``norm`` and the sigmoid of the output gate. ``state``: the layer's
    ``(S [slots, H, D, DV], n [slots, H, D], m [slots, H])`` in fp32, advanced in place."""
    T, dtype = proj.shape[0], proj.dtype
    H, D, DV = s.heads, s.dim, s.v_dim
    out = torch.empty((T, H * DV), dtype=dtype, device=proj.device)
    if not proj.is_cuda:
        _memory_reference(proj, input_bias, forget_bias, norm, s, state, cache, eps, out)
        return out
    if dtype not in (torch.bfloat16, torch.float32):
        raise TypeError(f"bfloat16 or float32 activations expected, got {dtype}")
    _rows(proj, dtype, T, 2 * H * (D + DV) + 2 * H, "proj")
    S, n, m = state
    slots = S.shape[0]
    for t, shape in ((S, (slots, H, D, DV)), (n, (slots, H, D)), (m, (slots, H)), (input_bias, (H,)), (forget_bias, (H,)),
                     (norm, (H * DV,))):
        if t.dtype != torch.float32 or tuple(t.shape) != shape or not t.is_contiguous():
            raise TypeError("matrix_memory: states, biases and the norm's weight are contiguous fp32 tensors of the layer's shape")
    B = cache.context_lens.numel()
    if B > slots:
        raise ValueError("matrix_memory: every sequence needs a state slot")
    lib = _lib.get_lib()
    f32 = int(dtype == torch.float32)
    cu, scratch = 0, 0
    if cache.is_prefill:
        cu = cache.cu_q_dev.data_ptr()
        longest = max(cache.q_lens_host, default=0)
        buf = torch.empty(lib.mfb_matrix_memory_scratch_floats(T, B, H, D, DV), dtype=torch.float32, device=proj.device)
        scratch = buf.data_ptr()
    else:
        longest = 1
    rc = lib.mfb_matrix_memory(proj.data_ptr(), proj.stride(0), input_bias.data_ptr(), forget_bias.data_ptr(), norm.data_ptr(),
                               S.data_ptr(), n.data_ptr(), m.data_ptr(), cu, cache.context_lens.data_ptr(),
                               cache.slot_mapping.data_ptr(), scratch, out.data_ptr(), T, B, H, D, DV, longest, s.gate_cap, float(eps),
                               f32, _lib.stream_ptr())
    _lib.check(rc, "mfb_matrix_memory")
    _lib.count_launch(3 if cache.is_prefill else 1)
    return out


# ---- state space --------------------------------------------------------------------------------------------------------------
@dataclass
class StateSpaceWeights:
    """Per-layer weights beside the projections, all fp32: ``conv [taps, H P + 2 G N]`` (x, B, C channels; the last row belongs to
    the current token), ``conv_bias``, ``dt_bias [H]``, ``a_log [H]``, ``skip [H]``, ``norm [H P]``."""
    conv: torch.Tensor
    conv_bias: torch.Tensor
    dt_bias: torch.Tensor
    a_log: torch.Tensor
    skip: torch.Tensor
    norm: torch.Tensor


@dataclass
class StateSpaceShape:
    heads: int
    head_dim: int
    state: int
    groups: int
    taps: int
    norm_groups: int

    @property
    def inner(self) -> int:
        return self.heads * self.head_dim

    @property
    def channels(self) -> int:
        return self.inner + 2 * self.groups * self.state

    @property
    def columns(self) -> int:
        """Columns of the input projection: gate, x, B, C, step sizes."""
        return self.inner + self.channels + self.heads


def _state_space_reference(proj, w: StateSpaceWeights, s: StateSpaceShape, state, ring, cache, eps, out):
    H, P, N, G = s.heads, s.head_dim, s.state, s.groups
    if not cache.is_prefill:
        out.zero_()
    for slot, r0, n, start in _sequences(cache, proj.shape[0]):
        z, xs, dt = torch.split(proj[r0:r0 + n, :s.columns], (s.inner, s.channels, H), dim=1)
        before = torch.zeros(s.taps - 1, s.channels, dtype=torch.float32)
        for d in range(1, s.taps):
            if start - d >= 0:
                before[s.taps - 1 - d] = ring[slot, (start - d) % s.taps].float()
        seq = torch.cat((before, xs.float()))
        y = F.silu(sum(seq[j:j + n] * w.conv[j] for j in range(s.taps)) + w.conv_bias).to(proj.dtype).float()
        for p in range(max(start, start + n - s.taps), start + n):
            ring[slot, p % s.taps] = xs[p - start]
        x, B, C = y[:, :s.inner].view(n, H, P), y[:, s.inner:s.inner + G * N], y[:, s.inner + G * N:]
        B, C = (t.view(n, G, N).repeat_interleave(H // G, 1) for t in (B, C))
        dt = F.softplus(dt.float() + w.dt_bias, threshold=1e9)
        keep = torch.exp(-torch.exp(w.a_log) * dt)
        S = state[slot].clone() if start > 0 else torch.zeros(H, N, P)
        o = torch.empty(n, H, P)
        for t in range(n):
            S = keep[t, :, None, None] * S + (dt[t, :, None] * B[t])[:, :, None] * x[t][:, None]
            o[t] = (S * C[t][:, :, None]).sum(1) + w.skip[:, None] * x[t]
        state[slot] = S
        o = (o.reshape(n, s.inner) * F.silu(z.float())).unflatten(1, (s.norm_groups, -1))
        o = o * torch.rsqrt(o.pow(2).mean(-1, keepdim=True) + eps)
        out[r0:r0 + n] = (o.flatten(1) * w.norm).to(out.dtype)


def state_space(proj: torch.Tensor, w: StateSpaceWeights, s: StateSpaceShape, state: Tuple[torch.Tensor, torch.Tensor], cache,
                eps: float) -> torch.Tensor:
    """``proj [T, >= columns]`` (gate z | x | B | C | raw step size, any row pitch), all of the step's rows in the order of ``cache``
    (``KVCacheContext``). x, B and C pass a causal convolution per channel and silu; per head (which shares B and C with its
    group), with ``dt = softplus(raw + dt_bias)``::

        S' = e^(-e^a_log dt) S + dt B x^T,   y = S'^T C + skip x

    Returns ``[T, H P]``: ``y * silu(z)``, RMS-normed in ``norm_groups`` parts, times ``norm``. ``state``: the layer's ``(S [slots,
    H, N, P] fp32, ring [slots, taps, channels])``, advanced in place."""
    T, dtype = proj.shape[0], proj.dtype
    S, ring = state
    H, P, N = s.heads, s.head_dim, s.state
    out = torch.empty((T, s.inner), dtype=dtype, device=proj.device)
    if not proj.is_cuda:
        _state_space_reference(proj, w, s, S, ring, cache, eps, out)
        return out
    if dtype not in (torch.bfloat16, torch.float32):
        raise TypeError(f"bfloat16 or float32 activations expected, got {dtype}")
    _rows(proj, dtype, T, s.columns, "proj")
    slots = S.shape[0]
    if tuple(S.shape[1:]) != (H, N, P) or S.dtype != torch.float32 or not S.is_contiguous() \
            or tuple(ring.shape) != (slots, s.taps, s.channels) or ring.dtype != dtype or not ring.is_contiguous():
        raise TypeError("state_space: the state does not have the layer's shape")
    for t, n in ((w.conv, s.taps * s.channels), (w.conv_bias, s.channels), (w.dt_bias, H), (w.a_log, H), (w.skip, H), (w.norm, s.inner)):
        if t.dtype != torch.float32 or t.numel() != n or not t.is_contiguous():
            raise TypeError("state_space: weights beside the projections are contiguous fp32 tensors")
    B = cache.context_lens.numel()
    if B > slots:
        raise ValueError("state_space: every sequence needs a state slot")
    lib = _lib.get_lib()
    cu, scratch, conv_out, pitch, longest = 0, None, None, 0, 1
    if cache.is_prefill:
        cu, longest = cache.cu_q_dev.data_ptr(), max(cache.q_lens_host, default=0)
        scratch = torch.empty(lib.mfb_state_space_scratch_floats(T, H, P, N), dtype=torch.float32, device=proj.device)
        pitch = s.channels + -s.channels % 8
        conv_out = torch.empty((T, pitch), dtype=dtype, device=proj.device)
    rc = lib.mfb_state_space(proj.data_ptr(), proj.stride(0), w.conv.data_ptr(), w.conv_bias.data_ptr(), w.dt_bias.data_ptr(),
                             w.a_log.data_ptr(), w.skip.data_ptr(), w.norm.data_ptr(), ring.data_ptr(), S.data_ptr(), cu,
                             cache.context_lens.data_ptr(), cache.slot_mapping.data_ptr(), _lib.ptr(scratch), _lib.ptr(conv_out),
                             out.data_ptr(), pitch, T, B, H, P, N, s.groups, s.taps, s.norm_groups, longest, float(eps),
                             int(dtype == torch.float32), _lib.stream_ptr())
    _lib.check(rc, "mfb_state_space")
    _lib.count_launch(4 if cache.is_prefill else 2)
    return out
