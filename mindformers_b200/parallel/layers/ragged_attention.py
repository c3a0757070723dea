"""Self-attention over a paged cache for ragged batches: whole prompts, portions of prompts and decoded tokens together.

``RaggedSelfAttention`` is the serving counterpart of ``SelfAttention`` for models whose attention has one or more of:
key and value sizes that differ, per-layer sizes and rotary settings, a chunked mask (``attention_chunk_size``), a
softmax sink (``attention_sink``), soft-capped scores (``attention_softcap``), no rotation at all (``rotary_dim = 0``),
projection biases folded into the following kernel. Parameter names are those of ``SelfAttention`` plus ``sink [heads]``
(fp32). ``RaggedAttentionCore`` is what lies between the projections, for mixers that share them with something else. One kernel applies bias, q / k norm and rotation and writes the cache
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

    def cache_shape(self):
        """``(kv heads, key size, value size)`` of this rank's cache."""
        return self.nkv, self.dim, self.v_dim

    def attend(self, qkv, bias, meta: AttnMeta, out=None, out_scale: float = 1.0):
        """``qkv [T, sum(sections)]`` (this rank's rows; any row pitch) → ``[T, heads * v_dim]`` times ``out_scale``, in ``out``
        when given."""
        from ...inference.ragged_attention import ragged_attention
        cache, layer = meta.cache, cache_layer(meta, self.layer_number)
        qn = self.q_layernorm.weight if self.q_layernorm is not None else None
        kn = self.k_layernorm.weight if self.k_layernorm is not None else None
        q = stream.qkv_rope_cache(qkv, bias, qn, kn, self.config.layernorm_epsilon, self.rotary.freqs, self.rotary.amplitude,
                                  self.config.rotary_interleaved, meta.positions, cache.slot_mapping,
                                  cache.key_cache[layer], cache.value_cache[layer], self.nq, self.nkv, self.dim, self.v_dim)
        return ragged_attention(q, cache, layer, self.scale, self.chunk, self.sink, self.softcap, out, out_scale)


class RaggedSelfAttention(RaggedAttentionCore):
    """Returns ``(output without bias, output bias)``: the step behind the sub-layer adds the bias."""

    def __init__(self, config, layer_number: int = 1):
        super().__init__(config, layer_number)
        self.linear_qkv = ColumnParallelLinear(config.hidden_size, sum(self.sections), config=config,
                                               bias=config.add_qkv_bias or config.add_bias_linear, skip_bias_add=True,
                                               partition_sections=self.sections)
        self.linear_proj = RowParallelLinear(config.num_attention_heads * self.v_dim, config.hidden_size, config=config,
                                             skip_bias_add=True,
                                             bias=config.add_attention_output_bias or config.add_bias_linear)

    def forward(self, hidden, rotary, meta: AttnMeta):
        cache_layer(meta, self.layer_number)
        qkv, bias = self.linear_qkv(hidden)
        return self.linear_proj(self.attend(qkv, bias, meta))
