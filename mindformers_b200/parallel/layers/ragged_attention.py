"""Self-attention over a paged cache for ragged batches: whole prompts, portions of prompts and decoded tokens together.

``RaggedSelfAttention`` is the serving counterpart of ``SelfAttention`` for models whose attention has one or more of:
key and value sizes that differ, per-layer sizes and rotary settings, a chunked mask (``attention_chunk_size``), a
softmax sink (``attention_sink``), projection biases folded into the following kernel. Parameter names are those of
``SelfAttention`` plus ``sink [heads]`` (fp32). One kernel applies bias, q / k norm and rotation and writes the cache
(``ops/stream.py::qkv_rope_cache``); one call attends for all sequences of the batch
(``inference/ragged_attention.py``).
"""
from __future__ import annotations

import math

import torch
import torch.nn as nn

from ...ops import stream
from .attention import AttnMeta, _local_heads
from .norm import RMSNorm
from .rotary import RotaryFrequencies
from .tensor_parallel import ColumnParallelLinear, RowParallelLinear, _mark_tp


class RaggedSelfAttention(nn.Module):
    """Returns ``(output without bias, output bias)``: the norm behind the sub-layer adds the bias. ``meta.layer_run``
    names the cache of the run (layers that share weights have a cache each)."""

    def __init__(self, config, layer_number: int = 1):
        super().__init__()
        self.config, self.layer_number = config, layer_number
        H, G, D = config.num_attention_heads, config.num_query_groups, config.kv_channels
        DV = config.v_channels or D
        self.dim, self.v_dim = D, DV
        if H % G:
            raise ValueError(f"layer {layer_number}: {H} query heads do not divide over {G} key / value heads")
        self.nq, self.nkv = _local_heads(config)
        sections = (H * D, G * D, G * DV)
        self.linear_qkv = ColumnParallelLinear(config.hidden_size, sum(sections), config=config,
                                               bias=config.add_qkv_bias or config.add_bias_linear, skip_bias_add=True,
                                               partition_sections=sections)
        self.q_layernorm = RMSNorm(config, D, config.layernorm_epsilon) if config.qk_layernorm else None
        self.k_layernorm = RMSNorm(config, D, config.layernorm_epsilon) if config.qk_layernorm else None
        dev = self.linear_qkv.weight.device
        if config.attention_sink:
            self.sink = nn.Parameter(torch.zeros(self.nq, dtype=torch.float32, device=dev))
            _mark_tp(self.sink, self.linear_qkv.tp > 1, 0)
        else:
            self.register_parameter("sink", None)
        rot = config.rotary_dim if config.rotary_dim is not None else int(D * config.rotary_percent)
        if rot % 2 or rot > D:
            raise ValueError(f"layer {layer_number}: {rot} rotary dimensions of heads of {D}")
        self.rotary = RotaryFrequencies(rot, config.rotary_base, config.rope_scaling, device=dev)
        self.scale = config.softmax_scale or 1.0 / math.sqrt(D)
        self.chunk = int(config.attention_chunk_size or 0)
        self.linear_proj = RowParallelLinear(H * DV, config.hidden_size, config=config, skip_bias_add=True,
                                             bias=config.add_attention_output_bias or config.add_bias_linear)

    def cache_shape(self):
        """``(kv heads, key size, value size)`` of this rank's cache."""
        return self.nkv, self.dim, self.v_dim

    def forward(self, hidden, rotary, meta: AttnMeta):
        cache = meta.cache
        if cache is None:
            raise RuntimeError("RaggedSelfAttention serves from a paged cache: generate() or the serving engine provide one")
        from ...inference.ragged_attention import ragged_attention
        layer = (meta.layer_run if meta.layer_run is not None else self.layer_number - 1) - cache.layer_offset
        qkv, bias = self.linear_qkv(hidden)
        qn = self.q_layernorm.weight if self.q_layernorm is not None else None
        kn = self.k_layernorm.weight if self.k_layernorm is not None else None
        q = stream.qkv_rope_cache(qkv, bias, qn, kn, self.config.layernorm_epsilon, self.rotary.freqs, self.rotary.amplitude,
                                  self.config.rotary_interleaved, meta.positions, cache.slot_mapping,
                                  cache.key_cache[layer], cache.value_cache[layer], self.nq, self.nkv, self.dim, self.v_dim)
        ctx = ragged_attention(q, cache, layer, self.scale, self.chunk, self.sink)
        out, bias = self.linear_proj(ctx)
        return out, bias
