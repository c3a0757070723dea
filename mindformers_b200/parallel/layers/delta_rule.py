"""Mixers with a recurrent state: the gated delta rule, alone or beside softmax attention.

``DeltaCore`` is what lies between the projections (``ops/recurrent.py``): short convolutions, unit keys, decays (per head, or
per key channel from a low-rank projection), the recurrence, its norm and its gate (one projection or a low-rank one).
``GatedDeltaMixer`` is a sub-layer of it; ``ParallelMixer`` runs ``RaggedAttentionCore`` and a ``DeltaCore`` on the same input.
Both have one input projection for everything that reads the hidden state and one output projection: the cores write side by
side into its operand, scaled, so that the weighted sum of the two outputs is part of that product.

The state of a sequence (``KVCacheContext.recurrent``) belongs to its row in the batch; the kernels take whole prompts,
portions and decoded tokens of any mix of sequences. Heads are split over tensor-parallel ranks, low-rank factors are
replicated up to their head-wise half. Serving layers: no gradients.
"""
from __future__ import annotations

import torch
import torch.nn as nn

from ...ops import functional as Fn
from ...ops import recurrent
from .. import parallel_state as ps
from .attention import AttnMeta
from .ragged_attention import RaggedAttentionCore, cache_layer
from .tensor_parallel import ColumnParallelLinear, RowParallelLinear, _init_weight, _mark_tp, default_init, section_local_sizes, \
    shard_sections


class DeltaCore(nn.Module):
    """``sections`` / ``groups``: rows of the input projection this core reads (q, k, v, gate, low-rank factors, step size,
    decay), in order, and the number of heads each splits over (1: replicated)."""

    def __init__(self, config, layer_number: int = 1):
        super().__init__()
        H, G, D, DV = config.delta_heads, config.delta_kv_heads, config.delta_key_dim, config.delta_value_dim
        if not H or not G or H % G:
            raise ValueError(f"layer {layer_number}: {H} heads do not divide over {G} query / key heads")
        tp, rank = ps.get_tensor_model_parallel_world_size(), ps.get_tensor_model_parallel_rank()
        self.layer_number, self.eps, self.tp = layer_number, config.layernorm_epsilon, tp
        dev = getattr(config, "device", None) or ("cuda" if torch.cuda.is_available() else "cpu")
        channel, gate_rank = config.delta_decay == "channel", config.delta_gate_rank
        if channel and not config.delta_decay_rank:
            raise ValueError(f"layer {layer_number}: decays per key channel need delta_decay_rank")
        parts = [("q", G * D, G), ("k", G * D, G), ("v", H * DV, H)]
        parts += [] if gate_rank else [("gate", H * DV, H)]
        parts += [("decay_down", config.delta_decay_rank, 1)] if channel else []
        parts += [("gate_down", gate_rank, 1)] if gate_rank else []
        parts += [("beta", H, H)]
        parts += [] if channel else [("decay", H, H)]
        self.names, self.sections, self.groups = (tuple(x) for x in zip(*parts))
        self.local = dict(zip(self.names, section_local_sizes(self.sections, tp, self.groups) if tp > 1 else self.sections))
        self.shape = recurrent.DeltaShape(H // tp, max(1, G // tp), D, DV, config.delta_conv_taps, channel,
                                          config.delta_gate == "silu")

        def small(full, dim=0, sections=None, groups=None):
            """fp32 parameter, split over the heads of the tensor-parallel ranks."""
            t = full if tp == 1 else (shard_sections(full, sections, dim, rank, tp, groups) if sections else full.chunk(tp, dim)[rank])
            p = nn.Parameter(t.contiguous())
            _mark_tp(p, tp > 1, dim)
            p.partition_sections, p.partition_groups = sections, groups
            return p

        def rand(*shape, mean=0.0, std=0.02):
            return torch.empty(*shape, dtype=torch.float32, device=dev).normal_(mean, std)
        conv = self.sections[:3]
        self.conv = small(rand(config.delta_conv_taps, sum(conv), std=config.delta_conv_taps ** -0.5), 1, conv, self.groups[:3])
        self.a_log = small(rand(H).uniform_(0.0, 1.0))
        self.dt_bias = small(rand(H * D if channel else H, mean=-3.0, std=1.0))
        self.norm = nn.Parameter(torch.ones(DV, dtype=torch.float32, device=dev))
        init = default_init(config.init_method_std)

        def up(rows, cols):
            p = _init_weight((rows // tp, cols), init, config.params_dtype, dev, partition_dim=0, full_shape=(rows, cols), rank=rank,
                             world=tp)
            _mark_tp(p, tp > 1, 0)
            return p
        self.register_parameter("decay_up", up(H * D, config.delta_decay_rank) if channel else None)
        self.register_parameter("gate_up", up(H * DV, gate_rank) if gate_rank else None)

    @property
    def width(self) -> int:
        """Columns of this rank's read-out."""
        return self.shape.heads * self.shape.v_dim

    def state_shape(self):
        """``(heads, key size, value size, conv channels, conv taps)`` of this rank's state."""
        s = self.shape
        return s.heads, s.dim, s.v_dim, s.channels, s.taps

    def forward(self, proj: torch.Tensor, meta: AttnMeta, out=None, out_scale: float = 1.0) -> torch.Tensor:
        """``proj [T, sum(local sections)]`` (any row pitch) → ``[T, heads * v_dim]`` times ``out_scale``, in ``out`` when given."""
        view, at = {}, 0
        for n in self.names:
            view[n] = proj[:, at:at + self.local[n]]
            at += self.local[n]
        x = proj[:, :self.shape.channels]
        a = view["decay"] if self.decay_up is None else Fn.linear(view["decay_down"], self.decay_up)
        gate = view["gate"] if self.gate_up is None else Fn.linear(view["gate_down"], self.gate_up)
        w = recurrent.DeltaWeights(self.conv, self.a_log, self.dt_bias, self.norm)
        state = meta.cache.recurrent[cache_layer(meta, self.layer_number)]
        return recurrent.delta_rule(x, view["beta"], a, gate, w, self.shape, state, meta.cache, self.eps, out, out_scale)


class GatedDeltaMixer(nn.Module):
    """``W_o core(W_in h)``. Returns ``(output, None)``."""

    def __init__(self, config, layer_number: int = 1):
        super().__init__()
        self.layer_number = layer_number
        self.core = DeltaCore(config, layer_number)
        c = self.core
        self.linear_in = ColumnParallelLinear(config.hidden_size, sum(c.sections), config=config, bias=False,
                                              partition_sections=c.sections, partition_groups=c.groups)
        self.linear_proj = RowParallelLinear(config.delta_heads * config.delta_value_dim, config.hidden_size, config=config)

    def cache_shape(self):
        return None

    def state_shape(self):
        return self.core.state_shape()

    def forward(self, hidden, rotary, meta: AttnMeta):
        cache_layer(meta, self.layer_number)
        proj, _ = self.linear_in(hidden)
        return self.linear_proj(self.core(proj, meta))


class ParallelMixer(nn.Module):
    """``left_scale * attention(h) + right_scale * delta_rule(h)``. Returns ``(output, None)``."""

    def __init__(self, config, layer_number: int = 1):
        super().__init__()
        self.layer_number = layer_number
        self.left, self.right = RaggedAttentionCore(config, layer_number), DeltaCore(config, layer_number)
        self.scales = tuple(float(x) for x in config.parallel_scales or (1.0, 1.0))
        tp = ps.get_tensor_model_parallel_world_size()
        if config.num_query_groups % tp:
            raise ValueError(f"layer {layer_number}: {config.num_query_groups} key / value heads do not divide over {tp} ranks")
        groups = (config.num_attention_heads, config.num_query_groups, config.num_query_groups)
        self.linear_in = ColumnParallelLinear(config.hidden_size, sum(self.left.sections + self.right.sections), config=config,
                                              bias=False, partition_sections=self.left.sections + self.right.sections,
                                              partition_groups=groups + self.right.groups)
        cols = (config.num_attention_heads * self.left.v_dim, config.delta_heads * config.delta_value_dim)
        self.linear_proj = RowParallelLinear(sum(cols), config.hidden_size, config=config, partition_sections=cols)
        self.left_rows = sum(self.left.sections) // tp
        self.left_cols = cols[0] // tp

    def cache_shape(self):
        return self.left.cache_shape()

    def state_shape(self):
        return self.right.state_shape()

    def forward(self, hidden, rotary, meta: AttnMeta):
        cache_layer(meta, self.layer_number)
        proj, _ = self.linear_in(hidden)
        n = self.left_cols + self.right.width
        both = torch.empty((proj.shape[0], n + -n % 8), dtype=proj.dtype, device=proj.device)[:, :n]      # rows start on 16 bytes
        self.left.attend(proj[:, :self.left_rows], None, meta, both[:, :self.left_cols], self.scales[0])
        self.right(proj[:, self.left_rows:], meta, both[:, self.left_cols:], self.scales[1])
        return self.linear_proj(both)
