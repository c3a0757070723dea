"""Serving ops of decoders that keep a 32-bit residual stream (or several) beside 16-bit activations.

Like the ops of ``functional.py`` every op has two bodies: the sm_100a kernel, always taken for CUDA tensors (bf16 or
fp32), and a plain PyTorch body for CPU tensors. They are inference ops: no gradients.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Tuple

import torch
import torch.nn.functional as F

from . import _lib
from . import functional as Fn

_DTYPES = (torch.bfloat16, torch.float32)


def _typed(*tensors, dtype):
    for t in tensors:
        if t is not None and (t.dtype != dtype or not t.is_contiguous()):
            raise TypeError(f"contiguous {dtype} tensors expected, got {t.dtype} with strides {t.stride()}")


def _check_dtype(dtype):
    if dtype not in _DTYPES:
        raise TypeError(f"bfloat16 or float32 activations expected, got {dtype}")


def norm_reference(x, w, b, eps, layer_norm):
    """fp32 layer norm (or RMS norm) of the last axis, with weight ``w`` and optional bias ``b``."""
    x = x.float()
    if layer_norm:
        x = x - x.mean(-1, keepdim=True)
    y = x * torch.rsqrt(x.pow(2).mean(-1, keepdim=True) + eps) * w.float()
    return y if b is None else y + b.float()


def add_normed(residual: torch.Tensor, y: torch.Tensor, y_bias: Optional[torch.Tensor], w: torch.Tensor,
               b: Optional[torch.Tensor], scale: Optional[torch.Tensor], eps: float, layer_norm: bool,
               inplace: bool = False) -> Tuple[torch.Tensor, torch.Tensor]:
    """``x = residual + scale * (norm(y + y_bias) * w + b)``; returns ``(x in the dtype of y, x in fp32)``.

    ``residual`` is the fp32 stream (updated in place by the kernel with ``inplace``) or, for the first sub-layer, the
    embedding in the dtype of ``y``. With fp32 activations both results are one tensor."""
    dtype = y.dtype
    if not y.is_cuda:
        yy = y.float() if y_bias is None else y.float() + y_bias.float()
        o = norm_reference(yy, w, b, eps, layer_norm)
        x = residual.float() + (o if scale is None else o * scale.float())
        return x.to(dtype), x
    _check_dtype(dtype)
    T, W = y.shape
    _typed(y_bias, w, b, scale, dtype=dtype)
    f32_stream = residual.dtype == torch.float32
    if residual.dtype not in (torch.float32, dtype) or not residual.is_contiguous() or y.stride(1) != 1:
        raise TypeError("the residual must be a contiguous fp32 stream or an embedding in the activation dtype")
    x = residual if inplace and f32_stream else torch.empty((T, W), dtype=torch.float32, device=y.device)
    copy = None if dtype == torch.float32 else torch.empty((T, W), dtype=dtype, device=y.device)
    rc = _lib.get_lib().mfb_add_normed(
        y.data_ptr(), y.stride(0), _lib.ptr(y_bias), w.data_ptr(), _lib.ptr(b), _lib.ptr(scale), residual.data_ptr(),
        int(f32_stream), x.data_ptr(), _lib.ptr(copy), T, W, int(layer_norm), float(eps), int(dtype == torch.float32),
        _lib.stream_ptr())
    _lib.check(rc, "mfb_add_normed")
    _lib.count_launch()
    return (x if copy is None else copy), x


def norm_stream(x: torch.Tensor, w: torch.Tensor, b: Optional[torch.Tensor], eps: float, layer_norm: bool) -> torch.Tensor:
    """Norm of the fp32 stream, returned in the dtype of ``w``."""
    if not x.is_cuda:
        return norm_reference(x, w, b, eps, layer_norm).to(w.dtype)
    _check_dtype(w.dtype)
    _typed(w, b, dtype=w.dtype)
    _typed(x, dtype=torch.float32)
    y = torch.empty(x.shape, dtype=w.dtype, device=x.device)
    rc = _lib.get_lib().mfb_norm_stream(x.data_ptr(), w.data_ptr(), _lib.ptr(b), y.data_ptr(), x.shape[0], x.shape[1],
                                        int(layer_norm), float(eps), int(w.dtype == torch.float32), _lib.stream_ptr())
    _lib.check(rc, "mfb_norm_stream")
    _lib.count_launch()
    return y


def residual_streams(x: torch.Tensor, n: int, y: Optional[torch.Tensor], mix: Optional[torch.Tensor],
                     write: Optional[torch.Tensor], read: Optional[torch.Tensor], w: torch.Tensor, eps: float,
                     keep: bool = True) -> Tuple[torch.Tensor, Optional[torch.Tensor]]:
    """One step of ``n`` fp32 residual streams: ``x_t <- sum_s mix[s, t] x_s + write[t] y`` (without ``y``: no update), then
    the next sub-layer's input ``rms_norm(sum_t read[t] x_t) * w`` (``read`` None: the sum of the streams).

    ``x``: the streams ``[T, n, W]`` fp32 (updated in place) or, before the first update, the embedding ``[T, W]`` in the dtype
    of ``w``, to which all streams are equal. Returns ``(input [T, W], streams)``; ``keep=False`` drops the streams, and
    without an update they are ``x`` itself."""
    embedded = x.dim() == 2
    T, W, dtype = x.shape[0], x.shape[-1], w.dtype
    if not x.is_cuda:
        xs = x.float()[:, None].expand(T, n, W) if embedded else x
        if y is not None:
            xs = torch.einsum("sd,tsw->tdw", mix, xs) + write[:, None] * y.float()[:, None]
        u = xs.sum(1) if read is None else (read[:, None] * xs).sum(1)
        return norm_reference(u, w, None, eps, False).to(dtype), (x if y is None else xs if keep else None)
    _check_dtype(dtype)
    if x.dtype != (dtype if embedded else torch.float32) or not x.is_contiguous() or not (embedded or x.shape[1] == n) \
            or (y is not None and (y.dtype != dtype or y.shape != (T, W) or y.stride(1) != 1)):
        raise TypeError("residual_streams: fp32 streams (or the embedding) and a sub-layer output in the activation dtype expected")
    _typed(mix, write, read, dtype=torch.float32)
    h = torch.empty((T, W), dtype=dtype, device=x.device)
    out = None
    if y is not None and keep:
        out = torch.empty((T, n, W), dtype=torch.float32, device=x.device) if embedded else x
    rc = _lib.get_lib().mfb_residual_streams(
        x.data_ptr(), int(embedded), _lib.ptr(y), 0 if y is None else y.stride(0), _lib.ptr(mix), _lib.ptr(write), _lib.ptr(read),
        w.data_ptr(), _lib.ptr(out), h.data_ptr(), T, n, W, float(eps), int(dtype == torch.float32), _lib.stream_ptr())
    _lib.check(rc, "mfb_residual_streams")
    _lib.count_launch()
    return h, (x if y is None else out)


def sinusoidal_frequencies(width: int) -> torch.Tensor:
    """fp64 ``[ceil(width / 2)]``: frequency i is ``10000 ** (-2 i / width)``."""
    i = torch.arange((width + 1) // 2, dtype=torch.float64)
    return torch.pow(torch.tensor(10000.0, dtype=torch.float64), -2.0 * i / width)


def embed(ids: torch.Tensor, table: torch.Tensor, scale: float, positions: torch.Tensor,
          freqs: Optional[torch.Tensor]) -> torch.Tensor:
    """``scale * table[ids]`` in fp32, plus (with ``freqs``) the position vector whose entries 2i and 2i + 1 are the sine and
    cosine of ``position * freqs[i]``. The angles are fp64 until they are within one turn."""
    T, W = ids.numel(), table.shape[1]
    if not table.is_cuda:
        x = table[ids].float() * scale
        if freqs is not None:
            a = positions.to(torch.float64)[:, None] * freqs[None, :]
            x = x + torch.stack((torch.sin(a), torch.cos(a)), dim=-1).flatten(1)[:, :W].float()
        return x
    _check_dtype(table.dtype)
    if ids.dtype != torch.int64 or positions.dtype != torch.int64 or positions.numel() != T or not table.is_contiguous() \
            or not ids.is_contiguous() or (freqs is not None and (freqs.dtype != torch.float64 or freqs.numel() != (W + 1) // 2)):
        raise TypeError("embed: int64 ids and positions, a contiguous table and fp64 frequencies expected")
    x = torch.empty((T, W), dtype=torch.float32, device=table.device)
    rc = _lib.get_lib().mfb_embed_stream(ids.data_ptr(), table.data_ptr(), positions.contiguous().data_ptr(), _lib.ptr(freqs),
                                         x.data_ptr(), T, W, table.shape[0], float(scale), int(table.dtype == torch.float32),
                                         _lib.stream_ptr())
    _lib.check(rc, "mfb_embed_stream")
    _lib.count_launch()
    return x


@dataclass
class Carry:
    """Token shift of one layer run: ``mu [W]`` and the cache that keeps the last token's vector per sequence slot."""
    mu: torch.Tensor
    cache: object
    run: int


def _shift_reference(h, carry: Carry):
    from .recurrent import _sequences
    cache, out = carry.cache, h.clone()
    state = cache.carry[carry.run]
    for slot, r0, n, start in _sequences(cache, h.shape[0]):
        first = state[slot] if start > 0 else torch.zeros_like(state[slot])
        before = torch.cat((first[None], h[r0:r0 + n - 1]))
        out[r0:r0 + n] = h[r0:r0 + n] + (before - h[r0:r0 + n]) * carry.mu.float()
        state[slot] = h[r0 + n - 1]
    return out


def normed_step(x: torch.Tensor, y: Optional[torch.Tensor], w_in: Optional[torch.Tensor], step: Optional[torch.Tensor],
                w_out: torch.Tensor, eps: float, zero_centered: bool, carry: Optional[Carry] = None,
                keep: bool = True) -> Tuple[torch.Tensor, Optional[torch.Tensor]]:
    """One step of an fp32 residual stream ``x [T, W]`` with norms on both sides of a sub-layer: ``x' = x + rms_norm(y; w_in) +
    step`` (without ``y`` or ``step``: without that term), then the next sub-layer's input ``h = rms_norm(x'; w_out)``, with
    ``carry`` shifted by a token: ``h + (h of the sequence's token before - h) * mu`` (zeros before the first token; the last
    ``h`` of a portion stays in ``cache.carry``). ``zero_centered``: the norms' weights are ``1 + w``.

    Returns ``(h in the dtype of w_out, x')``; ``x`` is not changed; ``keep=False`` drops ``x'``."""
    T, W, dtype = x.shape[0], x.shape[1], w_out.dtype
    if not x.is_cuda:
        one = 1.0 if zero_centered else 0.0
        if y is not None:
            x = x + norm_reference(y, w_in.float() + one, None, eps, False)
        if step is not None:
            x = x + step.float()
        h = norm_reference(x, w_out.float() + one, None, eps, False)
        if carry is not None:
            h = _shift_reference(h, carry)
        return h.to(dtype), (x if keep else None)
    _check_dtype(dtype)
    _typed(w_in, step, w_out, None if carry is None else carry.mu, dtype=dtype)
    if x.dtype != torch.float32 or not x.is_contiguous() or (y is not None and (
            y.dtype != dtype or y.shape != (T, W) or y.stride(1) != 1 or w_in is None)):
        raise TypeError("normed_step: a contiguous fp32 stream and a sub-layer output in the activation dtype expected")
    h = torch.empty((T, W), dtype=dtype, device=x.device)
    same = y is None and step is None
    out = torch.empty_like(x) if keep and not same else None
    B, cu, lens, slots, before, after = 0, 0, 0, 0, 0, 0
    if carry is not None:
        c = carry.cache
        state = c.carry[carry.run]
        B = c.context_lens.numel()
        if state.dtype != torch.float32 or state.shape[1] != W or not state.is_contiguous() or B > state.shape[0]:
            raise ValueError("normed_step: the carry does not have the stream's width, or a sequence has no slot")
        cu = c.cu_q_dev.data_ptr() if c.is_prefill else 0
        lens, slots, after = c.context_lens.data_ptr(), c.slot_mapping.data_ptr(), state.data_ptr()
        before = c.carry_before[carry.run].data_ptr() if c.is_prefill else after
    rc = _lib.get_lib().mfb_normed_step(
        x.data_ptr(), _lib.ptr(y), 0 if y is None else y.stride(0), _lib.ptr(w_in), _lib.ptr(step), w_out.data_ptr(), _lib.ptr(out),
        h.data_ptr(), None if carry is None else carry.mu.data_ptr(), before, after, cu, lens, slots, T, W, B, int(zero_centered),
        float(eps), int(dtype == torch.float32), _lib.stream_ptr())
    _lib.check(rc, "mfb_normed_step")
    _lib.count_launch()
    return h, (x if same else out) if keep else None


@dataclass
class InputConv:
    """Causal convolution of one layer run: ``w [taps, W]`` fp32 (the last row meets the current token) and the cache that keeps
    the last ``taps - 1`` rows per sequence slot."""
    w: torch.Tensor
    cache: object
    run: int

    def rows(self, before: bool = False):
        """``[slots, taps - 1, W]`` of this run (``before``: as they were before a prefill step)."""
        t = self.cache.carry_before if before else self.cache.carry
        taps, W = self.w.shape
        return None if t is None else t[self.run].view(-1, taps - 1, W)


def _input_conv_reference(h, conv: InputConv):
    from .recurrent import _sequences
    out, (taps, W) = h.clone(), conv.w.shape
    state = conv.rows()
    for slot, r0, n, start in _sequences(conv.cache, h.shape[0]):
        seq = h[r0:r0 + n]
        if taps > 1:
            first = state[slot] if start > 0 else torch.zeros_like(state[slot])
            seq = torch.cat((first, seq))
            state[slot] = seq[n:]
        out[r0:r0 + n] = h[r0:r0 + n] + sum(seq[j:j + n] * conv.w[j] for j in range(taps))
    return out


def grouped_norm_reference(x, w, groups, eps):
    """fp32 RMS norm of ``groups`` neighbouring parts of the last axis, each by its own root mean square."""
    parts = x.float().unflatten(-1, (groups, -1))
    return (parts * torch.rsqrt(parts.pow(2).mean(-1, keepdim=True) + eps)).flatten(-2) * w.float()


def joint_step(x: torch.Tensor, ys, base: Optional[torch.Tensor], step: Optional[torch.Tensor], w: Optional[torch.Tensor],
               groups: int, eps: float, dtype: torch.dtype, conv: Optional[InputConv] = None, want_h: bool = True,
               keep: bool = True) -> Tuple[Optional[torch.Tensor], Optional[torch.Tensor], Optional[torch.Tensor]]:
    """One step of an fp32 residual stream ``x [T, W]`` whose sub-layers run side by side: ``x' = x + sum(ys) + base + step``
    (``ys``: up to two outputs in the activation dtype; ``base [T, W]`` fp32; ``step [W]``; all optional), ``h`` its RMS norm in
    ``groups`` parts times ``w`` (``w`` None: ``x'`` itself) and, with ``conv``, ``h + conv(h)``: a causal convolution per channel
    (zeros before the first token; the last rows of a portion stay in ``cache.carry``).

    Returns ``(h, h + conv(h), x')``, the first two in ``dtype``; ``want_h=False`` / ``keep=False`` drop ``h`` / ``x'``. ``x`` is
    not changed."""
    T, W = x.shape
    ys = [y for y in ys if y is not None]
    if not x.is_cuda:
        for t in ys + [base, step]:
            x = x if t is None else x + t.float()
        h = x if w is None else grouped_norm_reference(x, w, groups, eps)
        hc = None if conv is None else _input_conv_reference(h, conv).to(dtype)
        return (h.to(dtype) if want_h else None), hc, (x if keep else None)
    _check_dtype(dtype)
    _typed(step, w, dtype=dtype)
    if x.dtype != torch.float32 or not x.is_contiguous() or len(ys) > 2 or any(
            y.dtype != dtype or y.shape != (T, W) or y.stride(1) != 1 for y in ys) or (base is not None and (
            base.dtype != torch.float32 or base.shape != (T, W) or base.stride(1) != 1)):
        raise TypeError("joint_step: a contiguous fp32 stream and sub-layer outputs in the activation dtype expected")
    h = torch.empty((T, W), dtype=dtype, device=x.device) if want_h else None
    hc = torch.empty((T, W), dtype=dtype, device=x.device) if conv is not None else None
    same = not ys and base is None and step is None
    out = torch.empty_like(x) if keep and not same else None
    B, cu, lens, slots, before, after, taps = 0, 0, 0, 0, 0, 0, 0
    if conv is not None:
        c, taps = conv.cache, conv.w.shape[0]
        B = c.context_lens.numel()
        if conv.w.dtype != torch.float32 or conv.w.shape[1] != W or not conv.w.is_contiguous():
            raise TypeError("joint_step: the convolution's weights are a contiguous fp32 [taps, W] tensor")
        cu = c.cu_q_dev.data_ptr() if c.is_prefill else 0
        lens, slots = c.context_lens.data_ptr(), c.slot_mapping.data_ptr()
        if taps > 1:
            state = conv.rows()
            if B > state.shape[0]:
                raise ValueError("joint_step: a sequence has no slot")
            after = state.data_ptr()
            before = conv.rows(before=True).data_ptr() if c.is_prefill else after
    y0, y1 = (ys + [None, None])[:2]
    rc = _lib.get_lib().mfb_joint_step(
        x.data_ptr(), _lib.ptr(y0), 0 if y0 is None else y0.stride(0), _lib.ptr(y1), 0 if y1 is None else y1.stride(0),
        _lib.ptr(base), 0 if base is None else base.stride(0), _lib.ptr(step), _lib.ptr(w), _lib.ptr(out), _lib.ptr(h), _lib.ptr(hc),
        None if conv is None else conv.w.data_ptr(), before, after, cu, lens, slots, T, W, B, int(groups), taps, float(eps),
        int(dtype == torch.float32), _lib.stream_ptr())
    _lib.check(rc, "mfb_joint_step")
    _lib.count_launch()
    return h, hc, (x if same else out) if keep else None


def relu2(x: torch.Tensor) -> torch.Tensor:
    """``max(x, 0)^2``"""
    if not x.is_cuda or (torch.is_grad_enabled() and x.requires_grad):
        return F.relu(x).square()
    _check_dtype(x.dtype)
    x2 = x.reshape(-1, x.shape[-1])
    if x2.stride(-1) != 1:
        x2 = x2.contiguous()
    y = torch.empty(x2.shape, dtype=x.dtype, device=x.device)
    rc = _lib.get_lib().mfb_relu2(x2.data_ptr(), y.data_ptr(), x2.shape[0], x2.shape[1], x2.stride(0),
                                  int(x.dtype == torch.float32), _lib.stream_ptr())
    _lib.check(rc, "mfb_relu2")
    _lib.count_launch()
    return y.view(x.shape)


def softcap_(x: torch.Tensor, cap: float) -> torch.Tensor:
    """``cap * tanh(x / cap)`` of an fp32 matrix, in place."""
    if not x.is_cuda:
        return x.div_(cap).tanh_().mul_(cap)
    if x.dtype != torch.float32 or x.dim() != 2 or x.stride(1) != 1:
        raise TypeError("softcap_ needs an fp32 matrix")
    rc = _lib.get_lib().mfb_softcap(x.data_ptr(), x.shape[0], x.shape[1], x.stride(0), float(cap), _lib.stream_ptr())
    _lib.check(rc, "mfb_softcap")
    _lib.count_launch()
    return x


_ACTS = {None: 0, "relu2": 1, "softcap": 2}


def linear(x: torch.Tensor, w: torch.Tensor, *, act: Optional[str] = None, cap: float = 0.0,
           out_dtype: Optional[torch.dtype] = None) -> torch.Tensor:
    """``act(x W^T)``: ``act`` None, ``"relu2"`` or ``"softcap"`` (``cap``; the result is then fp32). ``out_dtype`` fp32
    keeps the accumulators unrounded. bf16 calls of up to 64 rows apply the activation in the GEMM's epilogue. Any
    width: rows that do not start on 16 bytes are padded (operands) or allocated with a padded pitch (result)."""
    if act not in _ACTS:
        raise ValueError(f"unknown activation {act!r}")
    dtype = torch.float32 if act == "softcap" else (out_dtype or x.dtype)
    M, N, K = x.shape[0], w.shape[0], x.shape[1]
    if x.is_cuda and x.dtype == torch.bfloat16 and w.dtype == torch.bfloat16 and Fn.get_gemm_backend() == "tcgen05":
        if M == 0:
            return torch.empty((0, N), dtype=dtype, device=x.device)
        if Fn._decode_gemm_ok(M, K, x, w):
            x, w = (t if Fn._aligned(t) else t.contiguous() for t in (x, w))
            out = torch.empty((M, N), dtype=dtype, device=x.device)
            rc = _lib.get_lib().mfb_gemm_bf16_decode_ex(
                x.data_ptr(), w.data_ptr(), out.data_ptr(), None, M, N, K, x.stride(0), w.stride(0), out.stride(0),
                Fn._DECODE_GEMM_KS, int(dtype == torch.float32), _ACTS[act], float(cap),
                _lib.status_word(x.device).data_ptr(), _lib.stream_ptr())
            _lib.check(rc, "mfb_gemm_bf16_decode_ex")
            _lib.count_launch()
            return out
        out = Fn.gemm(x, w, out_dtype=dtype)
    else:                                                  # fp32, CPU tensors, or the library GEMM backend
        out = F.linear(x, w).to(dtype)
    if act == "relu2":
        return relu2(out)
    if act == "softcap":
        return softcap_(out, cap)
    return out


def _rotate_reference(x, positions, freqs, amplitude, rot, interleaved):
    if not rot:
        return x
    a = positions.to(torch.float32)[:, None] * freqs[None, :]
    c, s = (a.cos() * amplitude)[:, None], (a.sin() * amplitude)[:, None]
    xr = x[..., :rot]
    if interleaved:
        u, v = xr[..., 0::2], xr[..., 1::2]
        y = torch.stack((u * c - v * s, v * c + u * s), dim=-1).flatten(-2)
    else:
        u, v = xr[..., :rot // 2], xr[..., rot // 2:]
        y = torch.cat((u * c - v * s, v * c + u * s), dim=-1)
    return torch.cat((y, x[..., rot:]), dim=-1)


def qkv_rope_cache(qkv: torch.Tensor, bias: Optional[torch.Tensor], q_norm: Optional[torch.Tensor],
                   k_norm: Optional[torch.Tensor], eps: float, freqs: torch.Tensor, amplitude: float, interleaved: bool,
                   positions: torch.Tensor, slots: torch.Tensor, key_cache: torch.Tensor, value_cache: torch.Tensor,
                   heads: int, kv_heads: int, dim: int, v_dim: int, unit_qk: bool = False, unit_v: bool = False) -> torch.Tensor:
    """Everything between the QKV projection and attention over the paged cache: projection bias, per-head RMS norm of q
    and k (``None``: no norm; ``unit_qk``: a norm without a weight) and of v (``unit_v``, without a weight), rotation of the
    first ``2 * len(freqs)`` dimensions by ``position * freqs`` (cos and sin times ``amplitude``) and the write of k and v into the cache rows ``slots`` (negative: not written).

    ``qkv [T, heads * dim + kv_heads * (dim + v_dim)]`` → q ``[T, heads, dim]``."""
    T, dtype, rot = qkv.shape[0], qkv.dtype, 2 * freqs.numel()
    nq, nk = heads * dim, kv_heads * dim
    if not qkv.is_cuda:
        x = qkv.float() if bias is None else qkv.float() + bias.float()
        q, k = x[:, :nq].view(T, heads, dim), x[:, nq:nq + nk].view(T, kv_heads, dim)
        v = x[:, nq + nk:]
        one = torch.ones(())
        if q_norm is not None or unit_qk:
            q = norm_reference(q, one if unit_qk else q_norm, None, eps, False)
        if k_norm is not None or unit_qk:
            k = norm_reference(k, one if unit_qk else k_norm, None, eps, False)
        if unit_v:
            v = norm_reference(v.reshape(T, kv_heads, v_dim), one, None, eps, False).reshape(T, -1)
        q = _rotate_reference(q, positions, freqs, amplitude, rot, interleaved)
        k = _rotate_reference(k, positions, freqs, amplitude, rot, interleaved)
        keep = slots >= 0
        at = slots[keep].long()
        key_cache.view(-1, nk)[at] = k.reshape(T, nk)[keep].to(key_cache.dtype)
        value_cache.view(-1, kv_heads * v_dim)[at] = v[keep].to(value_cache.dtype)
        return q.to(dtype)
    _check_dtype(dtype)
    _typed(bias, q_norm, k_norm, key_cache, value_cache, dtype=dtype)
    if qkv.stride(1) != 1 or qkv.shape[1] != nq + nk + kv_heads * v_dim or positions.dtype != torch.int64 \
            or slots.dtype != torch.int32 or (unit_qk and (q_norm is not None or k_norm is not None)) \
            or freqs.dtype != torch.float32 or positions.numel() != T or slots.numel() != T:
        raise TypeError("qkv_rope_cache: unexpected shapes or dtypes")
    q = torch.empty((T, heads, dim), dtype=dtype, device=qkv.device)
    rc = _lib.get_lib().mfb_qkv_rope_cache(
        qkv.data_ptr(), qkv.stride(0), _lib.ptr(bias), _lib.ptr(q_norm), _lib.ptr(k_norm), float(eps), freqs.data_ptr(),
        float(amplitude), rot, int(interleaved or not rot), positions.data_ptr(), slots.data_ptr(), q.data_ptr(), key_cache.data_ptr(),
        value_cache.data_ptr(), T, heads, kv_heads, dim, v_dim, int(unit_qk) + 2 * int(unit_v), int(dtype == torch.float32),
        _lib.stream_ptr())
    _lib.check(rc, "mfb_qkv_rope_cache")
    _lib.count_launch()
    return q


def latent_norm_cache(proj: torch.Tensor, q_norm: torch.Tensor, kv_norm: torch.Tensor, eps: float, slots: torch.Tensor,
                      cache: torch.Tensor, freqs: Optional[torch.Tensor] = None, positions: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Between the down projections of latent attention and what follows: ``proj [T, >= Q + R + P]`` (query latent | key / value
    latent | key part with positions, any row pitch) → the RMS-normed query latent ``[T, Q]``; the normed key / value latent and,
    with ``freqs [P / 2]``, the last part rotated (neighbouring dimensions, by ``position * freqs``) go to the rows ``slots`` of
    ``cache [.., R + P]`` (negative: not written)."""
    T, dtype, Q, R = proj.shape[0], proj.dtype, q_norm.numel(), kv_norm.numel()
    P = 0 if freqs is None else 2 * freqs.numel()
    if not proj.is_cuda:
        c = norm_reference(proj[:, Q:Q + R], kv_norm, None, eps, False)
        if P:
            k = _rotate_reference(proj[:, None, Q + R:Q + R + P].float(), positions, freqs, 1.0, P, True)[:, 0]
            c = torch.cat((c, k), dim=1)
        keep = slots >= 0
        cache.view(-1, R + P)[slots[keep].long()] = c[keep].to(cache.dtype)
        return norm_reference(proj[:, :Q], q_norm, None, eps, False).to(dtype)
    _check_dtype(dtype)
    _typed(q_norm, kv_norm, cache, dtype=dtype)
    if proj.stride(1) != 1 or proj.shape[1] < Q + R + P or slots.dtype != torch.int32 or slots.numel() != T \
            or cache.shape[-1] != R + P or (P and (freqs.dtype != torch.float32 or positions.dtype != torch.int64
                                                   or positions.numel() != T or not positions.is_contiguous())):
        raise TypeError("latent_norm_cache: unexpected shapes or dtypes")
    q = torch.empty((T, Q), dtype=dtype, device=proj.device)
    rc = _lib.get_lib().mfb_latent_norm_cache(proj.data_ptr(), proj.stride(0), q_norm.data_ptr(), kv_norm.data_ptr(), float(eps),
                                              slots.data_ptr(), q.data_ptr(), cache.data_ptr(), _lib.ptr(freqs),
                                              _lib.ptr(positions) if P else 0, T, Q, R, P,
                                              int(dtype == torch.float32), _lib.stream_ptr())
    _lib.check(rc, "mfb_latent_norm_cache")
    _lib.count_launch()
    return q


def rotate_tail_(x: torch.Tensor, freqs: torch.Tensor, positions: torch.Tensor) -> torch.Tensor:
    """The last ``2 * len(freqs)`` dimensions of every head of ``x [T, heads, dim]`` rotated by ``position * freqs`` (neighbouring
    dimensions are pairs), in place."""
    T, H, D = x.shape
    P = 2 * freqs.numel()
    if not x.is_cuda:
        x[..., D - P:] = _rotate_reference(x[..., D - P:].float(), positions, freqs, 1.0, P, True).to(x.dtype)
        return x
    _check_dtype(x.dtype)
    if not x.is_contiguous() or P > D or freqs.dtype != torch.float32 or positions.dtype != torch.int64 or positions.numel() != T \
            or not positions.is_contiguous():
        raise TypeError("rotate_tail_: contiguous heads, fp32 frequencies and int64 positions expected")
    rc = _lib.get_lib().mfb_rotate_tail(x.data_ptr(), freqs.data_ptr(), positions.data_ptr(), T, H, D, P,
                                        int(x.dtype == torch.float32), _lib.stream_ptr())
    _lib.check(rc, "mfb_rotate_tail")
    _lib.count_launch()
    return x


def gate_heads_(x: torch.Tensor, gate: torch.Tensor) -> torch.Tensor:
    """``x [T, n]`` times ``sigmoid(gate [T, m])``, in place: a gate per column (m = n) or per n / m neighbouring columns."""
    T, n = x.shape
    m = gate.shape[1]
    if n % m or gate.shape[0] != T:
        raise ValueError(f"{m} gates for {n} columns")
    if not x.is_cuda:
        return x.copy_((x.float().view(T, m, n // m) * torch.sigmoid(gate.float())[..., None]).view(T, n))
    _check_dtype(x.dtype)
    if gate.dtype != x.dtype or x.stride(1) != 1 or gate.stride(1) != 1:
        raise TypeError("gate_heads_: matrices of one dtype with unit column stride expected")
    rc = _lib.get_lib().mfb_gate_heads(x.data_ptr(), x.stride(0), gate.data_ptr(), gate.stride(0), T, n, m,
                                       int(x.dtype == torch.float32), _lib.stream_ptr())
    _lib.check(rc, "mfb_gate_heads")
    _lib.count_launch()
    return x


def talk_mix(o: torch.Tensor, talk: torch.Tensor, gate: Optional[torch.Tensor]) -> torch.Tensor:
    """Softmax weights mixed over heads, applied after the products with the values: ``o [T, H, G, DV]`` holds head g's weights
    on the values of every key / value head; result ``[T, H * DV]``, head h ``sum_g talk[h, g] o[:, g, own head of h]`` times
    ``sigmoid(gate [T, H * DV])``."""
    T, H, G, DV = o.shape
    if not o.is_cuda:
        own = torch.arange(H) // (H // G)
        y = torch.einsum("hg,tghv->thv", talk.float(), o.float()[:, :, own])
        y = y.reshape(T, H * DV)
        return (y if gate is None else y * torch.sigmoid(gate.float())).to(o.dtype)
    _check_dtype(o.dtype)
    if talk.dtype != torch.float32 or talk.shape != (H, H) or not talk.is_contiguous() or not o.is_contiguous() or (
            gate is not None and (gate.dtype != o.dtype or gate.shape != (T, H * DV) or gate.stride(1) != 1)):
        raise TypeError("talk_mix: unexpected shapes or dtypes")
    y = torch.empty((T, H * DV), dtype=o.dtype, device=o.device)
    rc = _lib.get_lib().mfb_talk_mix(o.data_ptr(), talk.data_ptr(), _lib.ptr(gate), 0 if gate is None else gate.stride(0),
                                     y.data_ptr(), T, H, G, DV, int(o.dtype == torch.float32), _lib.stream_ptr())
    _lib.check(rc, "mfb_talk_mix")
    _lib.count_launch()
    return y
