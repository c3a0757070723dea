"""Serving ops of decoders that keep a 32-bit residual stream (or several) beside 16-bit activations.

Like the ops of ``functional.py`` every op has two bodies: the sm_100a kernel, always taken for CUDA tensors (bf16 or
fp32), and a plain PyTorch body for CPU tensors. They are inference ops: no gradients.
"""
from __future__ import annotations

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
                   heads: int, kv_heads: int, dim: int, v_dim: int) -> torch.Tensor:
    """Everything between the QKV projection and attention over the paged cache: projection bias, per-head RMS norm of q
    and k (``None``: no norm), rotation of the first ``2 * len(freqs)`` dimensions by ``position * freqs`` (cos and sin
    times ``amplitude``) and the write of k and v into the cache rows ``slots`` (negative: not written).

    ``qkv [T, heads * dim + kv_heads * (dim + v_dim)]`` → q ``[T, heads, dim]``."""
    T, dtype, rot = qkv.shape[0], qkv.dtype, 2 * freqs.numel()
    nq, nk = heads * dim, kv_heads * dim
    if not qkv.is_cuda:
        x = qkv.float() if bias is None else qkv.float() + bias.float()
        q, k = x[:, :nq].view(T, heads, dim), x[:, nq:nq + nk].view(T, kv_heads, dim)
        v = x[:, nq + nk:]
        if q_norm is not None:
            q = norm_reference(q, q_norm, None, eps, False)
        if k_norm is not None:
            k = norm_reference(k, k_norm, None, eps, False)
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
            or slots.dtype != torch.int32 or freqs.dtype != torch.float32 or positions.numel() != T or slots.numel() != T:
        raise TypeError("qkv_rope_cache: unexpected shapes or dtypes")
    q = torch.empty((T, heads, dim), dtype=dtype, device=qkv.device)
    rc = _lib.get_lib().mfb_qkv_rope_cache(
        qkv.data_ptr(), qkv.stride(0), _lib.ptr(bias), _lib.ptr(q_norm), _lib.ptr(k_norm), float(eps), freqs.data_ptr(),
        float(amplitude), rot, int(interleaved), positions.data_ptr(), slots.data_ptr(), q.data_ptr(), key_cache.data_ptr(),
        value_cache.data_ptr(), T, heads, kv_heads, dim, v_dim, int(dtype == torch.float32), _lib.stream_ptr())
    _lib.check(rc, "mfb_qkv_rope_cache")
    _lib.count_launch()
    return q
