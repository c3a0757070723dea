"""Self-attention over a paged cache for ragged batches: whole prompts, portions of prompts and decoded tokens together.

``RaggedSelfAttention`` is the serving counterpart of ``SelfAttention`` for models whose attention has one or more of:
key and value sizes that differ, per-layer sizes and rotary settings, a chunked mask (``attention_chunk_size``), a
softmax sink (``attention_sink``), soft-capped scores (``attention_softcap``), no rotation at all (``rotary_dim = 0``), a
sliding window (``attention_window``), norms without weights (``qk_unit_norm``, ``value_unit_norm``), weights mixed over heads
(``attention_talk``), an output gate (``attention_output_gate``), projection biases folded into the following kernel. Parameter
names are those of ``SelfAttention`` plus ``sink [heads]`` and ``talk [heads, heads]`` (fp32). ``RaggedLatentAttention`` caches
one latent per token instead of keys and values. ``RaggedAttentionCore`` is what lies between the projections, for mixers that
share them with something else. One kernel applies bias, q / k norm and rotation and writes the cache
(``ops/stream.py::qkv_rope_cache``); one call attends for all sequences of the batch
(``inference/ragged_attention.py``).
"""
from __future__ import annotations

import math

import torch
import torch.nn as nn

from ...ops import stream
from .. import parallel_state as ps
from .attention import AttnMeta, _local_heads
from .norm import RMSNorm
from .rotary import RotaryFrequencies
from .tensor_parallel import ColumnParallelLinear, RowParallelLinear, _mark_tp


def cache_layer(meta: AttnMeta, layer_number: int) -> int:
    """Index of the running layer's cache: ``meta.layer_run`` names the run (layers that share weights have a cache each)."""
    if meta.cache is None:
        raise RuntimeError("this mixer serves from a cache: generate() or the serving engine provide one")
    return (meta.layer_run if meta.layer_run is not None else layer_number - 1) - meta.cache.layer_offset


class RaggedAttentionCore(nn.Module):
    """Norms and rotation of q and k, cache write and attention; ``sections`` are the rows of the q | k | v projection."""

    def __init__(self, config, layer_number: int = 1, device=None):
        super().__init__()
        self.config, self.layer_number = config, layer_number
        H, G, D = config.num_attention_heads, config.num_query_groups, config.kv_channels
        DV = config.v_channels or D
        self.dim, self.v_dim = D, DV
        if H % G:
            raise ValueError(f"layer {layer_number}: {H} query heads do not divide over {G} key / value heads")
        self.nq, self.nkv = _local_heads(config)
        self.sections = (H * D, G * D, G * DV)
        dev = device or getattr(config, "device", None) or ("cuda" if torch.cuda.is_available() else "cpu")
        tp = ps.get_tensor_model_parallel_world_size()
        self.q_layernorm = RMSNorm(config, D, config.layernorm_epsilon) if config.qk_layernorm else None
        self.k_layernorm = RMSNorm(config, D, config.layernorm_epsilon) if config.qk_layernorm else None
        if config.attention_sink:
            self.sink = nn.Parameter(torch.zeros(self.nq, dtype=torch.float32, device=dev))
            _mark_tp(self.sink, tp > 1, 0)
        else:
            self.register_parameter("sink", None)
        rot = config.rotary_dim if config.rotary_dim is not None else int(D * config.rotary_percent)
        if rot % 2 or rot > D:
            raise ValueError(f"layer {layer_number}: {rot} rotary dimensions of heads of {D}")
        self.rotary = RotaryFrequencies(rot, config.rotary_base, config.rope_scaling, device=dev)
        self.scale = config.softmax_scale or 1.0 / math.sqrt(D)
        self.chunk = int(config.attention_chunk_size or 0)
        self.softcap = float(config.attention_softcap or 0.0)
        self.window = int(config.attention_window or 0)
        self.unit_qk, self.unit_v = bool(config.qk_unit_norm), bool(config.value_unit_norm)
        if self.unit_qk and config.qk_layernorm:
            raise ValueError(f"layer {layer_number}: qk_unit_norm and qk_layernorm exclude one another")
        if config.attention_talk and (tp > 1 or self.chunk or self.softcap or config.attention_sink):
            raise NotImplementedError("softmax weights mixed over heads: one tensor-parallel rank, no chunks, no soft cap, no sink")
        self.register_parameter("talk", nn.Parameter(torch.eye(H, dtype=torch.float32, device=dev)) if config.attention_talk else None)

    def cache_shape(self):
        """``(kv heads, key size, value size)`` of this rank's cache."""
        return self.nkv, self.dim, self.v_dim

    def attend(self, qkv, bias, meta: AttnMeta, out=None, out_scale: float = 1.0, gate=None):
        """``qkv [T, sum(sections)]`` (this rank's rows; any row pitch) → ``[T, heads * v_dim]`` times ``out_scale``, in ``out``
        when given; ``gate``: times its sigmoid."""
        from ...inference.ragged_attention import ragged_attention, talking_attention
        cache, layer = meta.cache, cache_layer(meta, self.layer_number)
        qn = self.q_layernorm.weight if self.q_layernorm is not None else None
        kn = self.k_layernorm.weight if self.k_layernorm is not None else None
        q = stream.qkv_rope_cache(qkv, bias, qn, kn, self.config.layernorm_epsilon, self.rotary.freqs, self.rotary.amplitude,
                                  self.config.rotary_interleaved, meta.positions, cache.slot_mapping,
                                  cache.key_cache[layer], cache.value_cache[layer], self.nq, self.nkv, self.dim, self.v_dim,
                                  self.unit_qk, self.unit_v)
        if self.talk is not None:
            if out is not None or out_scale != 1.0:
                raise NotImplementedError("softmax weights mixed over heads write a result of their own")
            return talking_attention(q, cache, layer, self.scale, self.talk, gate, self.window)
        out = ragged_attention(q, cache, layer, self.scale, self.chunk, self.sink, self.softcap, out, out_scale, self.window)
        return out if gate is None else stream.gate_heads_(out, gate)


class RaggedSelfAttention(RaggedAttentionCore):
    """Returns ``(output without bias, output bias)``: the step behind the sub-layer adds the bias. With an output gate its
    rows follow those of q, k and v in the input projection, and the bias of q, k and v is a parameter of its own."""

    def __init__(self, config, layer_number: int = 1):
        super().__init__(config, layer_number)
        bias = bool(config.add_qkv_bias or config.add_bias_linear)
        H, tp = config.num_attention_heads, ps.get_tensor_model_parallel_world_size()
        gates = {None: 0, "head": H, "channel": H * self.v_dim}[config.attention_output_gate]
        if gates and tp > 1:
            raise NotImplementedError("gated ragged attention runs on one tensor-parallel rank")
        sections = self.sections + ((gates,) if gates else ())
        self.linear_qkv = ColumnParallelLinear(config.hidden_size, sum(sections), config=config, bias=bias and not gates,
                                               skip_bias_add=True, partition_sections=sections)
        self.n_qkv = sum(self.sections) // tp if not gates else sum(self.sections)
        self.gated = gates > 0
        w = self.linear_qkv.weight
        self.register_parameter("qkv_bias", nn.Parameter(torch.zeros(sum(self.sections), dtype=w.dtype, device=w.device))
                                if bias and gates else None)
        self.linear_proj = RowParallelLinear(config.num_attention_heads * self.v_dim, config.hidden_size, config=config,
                                             skip_bias_add=True,
                                             bias=config.add_attention_output_bias or config.add_bias_linear)

    def forward(self, hidden, rotary, meta: AttnMeta):
        cache_layer(meta, self.layer_number)
        qkv, bias = self.linear_qkv(hidden)
        if self.gated:
            return self.linear_proj(self.attend(qkv[:, :self.n_qkv], self.qkv_bias, meta, gate=qkv[:, self.n_qkv:]))
        return self.linear_proj(self.attend(qkv, bias, meta))


def expand_kv_up(w_uk: torch.Tensor, w_uv: torch.Tensor, heads: int, dim: int, rot: int) -> torch.Tensor:
    """Factors of keys ``[heads * dim, rank]`` and values ``[heads * v_dim, rank]`` → rows that act on a cached latent with a rotated
    key part of ``rot`` numbers behind it: a head's key rows are followed by ``rot`` unit vectors."""
    rank = w_uk.shape[1]
    k = w_uk.new_zeros(heads, dim + rot, rank + rot)
    k[:, :dim, :rank] = w_uk.view(heads, dim, rank)
    k[:, dim:, rank:] = torch.eye(rot, dtype=w_uk.dtype, device=w_uk.device)
    return torch.cat((k.view(-1, rank + rot), torch.nn.functional.pad(w_uv, (0, rot))))


def split_kv_up(w: torch.Tensor, heads: int, dim: int, rot: int, rank: int):
    """Inverse of ``expand_kv_up``: ``(w_uk, w_uv)``."""
    n = heads * (dim + rot)
    return w[:n].view(heads, dim + rot, rank + rot)[:, :dim, :rank].reshape(heads * dim, rank), w[n:, :rank].contiguous()


class RaggedLatentAttention(nn.Module):
    """Latent attention: queries through a normed latent, keys and values linear in one cached, normed latent of
    ``kv_lora_rank`` numbers per token. With ``rotary_dim`` each head's query has as many dimensions more, which are rotated, and so
    has its key: one rotated part for all heads, cached behind the latent. Returns ``(output, None)``.

    One projection makes the query latent, the key / value latent, the rotated key part and the output gates; one kernel norms both
    latents, rotates the key part and writes the cache (``ops/stream.py::latent_norm_cache``). The rows of ``linear_kv_up`` (keys,
    then values, head by head) act on the whole cached row: those that make a key's rotated part are unit vectors, so that keys of
    all heads, expanded or absorbed into the queries, are one product."""

    def __init__(self, config, layer_number: int = 1):
        super().__init__()
        if ps.get_tensor_model_parallel_world_size() > 1:
            raise NotImplementedError("ragged latent attention runs on one tensor-parallel rank")
        self.layer_number, self.eps = layer_number, config.layernorm_epsilon
        H, D, DV, Q, R = (config.num_attention_heads, config.kv_channels, config.v_channels or config.kv_channels, config.q_lora_rank,
                          config.kv_lora_rank)
        P = int(config.rotary_dim or 0)
        if P % 2 or (P and not config.rotary_interleaved):
            raise ValueError(f"layer {layer_number}: {P} rotary dimensions (an even number of interleaved ones)")
        self.heads, self.dim, self.v_dim, self.rank, self.rot = H, D + P, DV, R, P
        self.scale, self.window = config.softmax_scale or 1.0 / math.sqrt(D + P), int(config.attention_window or 0)
        gates = {None: 0, "head": H, "channel": H * DV}[config.attention_output_gate]
        self.sections = (Q, R + P) + ((gates,) if gates else ())
        linear = lambda cols, rows: ColumnParallelLinear(cols, rows, config=config, bias=False)
        self.linear_in = linear(config.hidden_size, sum(self.sections))
        self.q_latent_norm, self.kv_latent_norm = RMSNorm(config, Q, self.eps), RMSNorm(config, R, self.eps)
        self.linear_q_up, self.linear_kv_up = linear(Q, H * (D + P)), linear(R + P, H * (D + P + DV))
        dev = self.linear_in.weight.device
        self.rotary = RotaryFrequencies(P, config.rotary_base, config.rope_scaling, device=dev) if P else None
        if P:
            if self.rotary.amplitude != 1.0:
                raise NotImplementedError("the rotation of latent attention has no amplitude")
            with torch.no_grad():
                self.linear_kv_up.weight.copy_(expand_kv_up(*split_kv_up(self.linear_kv_up.weight, H, D, P, R), H, D, P))
        self.register_parameter("sink", nn.Parameter(torch.zeros(H, dtype=torch.float32, device=dev)) if config.attention_sink else None)
        self.linear_proj = RowParallelLinear(H * DV, config.hidden_size, config=config)

    def cache_shape(self):
        return 1, self.rank + self.rot, 0

    def forward(self, hidden, rotary, meta: AttnMeta):
        from ...inference.ragged_attention import latent_attention
        freqs = None if self.rotary is None else self.rotary.freqs
        cache, layer = meta.cache, cache_layer(meta, self.layer_number)
        proj, _ = self.linear_in(hidden)
        n = sum(self.sections[:2])
        c = stream.latent_norm_cache(proj[:, :n], self.q_latent_norm.weight, self.kv_latent_norm.weight, self.eps, cache.slot_mapping,
                                     cache.key_cache[layer], freqs, meta.positions)
        q = self.linear_q_up(c)[0].contiguous().view(-1, self.heads, self.dim)
        if freqs is not None:
            q = stream.rotate_tail_(q, freqs, meta.positions)
        out = latent_attention(q, cache, layer, self.linear_kv_up.weight, self.v_dim, self.scale, self.window, self.sink, self.rank)
        if len(self.sections) > 2:
            out = stream.gate_heads_(out, proj[:, n:])
        return self.linear_proj(out)
