"""Mixer with a state space per head whose decay is a scalar (Mamba-2).

One projection makes the gate, x, B, C and the step sizes; ``ops/recurrent.py::state_space`` is everything up to the output
projection. The state of a sequence (``KVCacheContext.recurrent``: ``S`` in fp32 and a ring of the last conv inputs) belongs to its
row in the batch; whole prompts, portions and decoded tokens of any mix of sequences are one call. A serving layer: no gradients.
"""
from __future__ import annotations

import torch
import torch.nn as nn

from ...ops import recurrent
from .. import parallel_state as ps
from .attention import AttnMeta
from .ragged_attention import cache_layer
from .tensor_parallel import ColumnParallelLinear, RowParallelLinear


class StateSpaceMixer(nn.Module):
    """Returns ``(output, None)``."""

    def __init__(self, config, layer_number: int = 1):
        super().__init__()
        if ps.get_tensor_model_parallel_world_size() > 1:
            raise NotImplementedError("the state-space mixer runs on one tensor-parallel rank")
        s = self.shape = recurrent.StateSpaceShape(config.ssm_heads, config.ssm_head_dim, config.ssm_state, config.ssm_groups,
                                                   config.ssm_conv_taps, config.ssm_norm_groups)
        if min(s.heads, s.head_dim, s.state, s.groups, s.taps, s.norm_groups) < 1 or s.heads % s.groups or s.inner % s.norm_groups:
            raise ValueError(f"layer {layer_number}: state space of {s}")
        self.layer_number, self.eps = layer_number, config.layernorm_epsilon
        self.linear_in = ColumnParallelLinear(config.hidden_size, s.columns, config=config, bias=False)
        dev = self.linear_in.weight.device

        def rand(*shape, mean=0.0, std=1.0):
            return nn.Parameter(torch.empty(*shape, dtype=torch.float32, device=dev).normal_(mean, std))
        self.conv, self.conv_bias = rand(s.taps, s.channels, std=s.taps ** -0.5), rand(s.channels, std=0.02)
        self.dt_bias, self.a_log = rand(s.heads, mean=-3.0), rand(s.heads, std=0.5)
        self.skip = nn.Parameter(torch.ones(s.heads, dtype=torch.float32, device=dev))
        self.norm = nn.Parameter(torch.ones(s.inner, dtype=torch.float32, device=dev))
        self.linear_proj = RowParallelLinear(s.inner, config.hidden_size, config=config)

    def cache_shape(self):
        return None

    def state_shape(self):
        """``(heads, state size, channels per head, conv channels, conv taps)``."""
        s = self.shape
        return s.heads, s.state, s.head_dim, s.channels, s.taps

    def forward(self, hidden, rotary, meta: AttnMeta):
        layer = cache_layer(meta, self.layer_number)
        proj, _ = self.linear_in(hidden)
        w = recurrent.StateSpaceWeights(self.conv, self.conv_bias, self.dt_bias, self.a_log, self.skip, self.norm)
        return self.linear_proj(recurrent.state_space(proj, w, self.shape, meta.cache.recurrent[layer], meta.cache, self.eps))
