"""Mixer with a matrix memory per head (the mLSTM of xLSTM): exponential input gate, sigmoid forget gate, running maximum.

One projection makes queries, keys, values, the output gate and both log gates; ``ops/recurrent.py::matrix_memory`` is everything
up to the output projection. The state of a sequence (``KVCacheContext.recurrent``: memory, normaliser, running maximum, fp32)
belongs to its row in the batch; whole prompts, portions and decoded tokens of any mix of sequences are one call. A serving layer:
no gradients.
"""
from __future__ import annotations

import torch
import torch.nn as nn

from ...ops import recurrent
from .. import parallel_state as ps
from .attention import AttnMeta
from .ragged_attention import cache_layer
from .tensor_parallel import ColumnParallelLinear, RowParallelLinear


class MatrixMemoryMixer(nn.Module):
    """Returns ``(output, None)``."""

    def __init__(self, config, layer_number: int = 1):
        super().__init__()
        if ps.get_tensor_model_parallel_world_size() > 1:
            raise NotImplementedError("the matrix-memory mixer runs on one tensor-parallel rank")
        H, D, DV = config.memory_heads, config.memory_key_dim, config.memory_value_dim
        if min(H, D, DV) < 1 or not config.memory_gate_cap > 0:
            raise ValueError(f"layer {layer_number}: {H} heads of {D} x {DV}, gates capped at {config.memory_gate_cap}")
        self.layer_number, self.eps = layer_number, config.layernorm_epsilon
        self.shape = recurrent.MemoryShape(H, D, DV, float(config.memory_gate_cap))
        self.sections = (H * D, H * D, H * DV, H * DV, H, H)           # q, k, v, output gate, input gate, forget gate
        self.linear_in = ColumnParallelLinear(config.hidden_size, sum(self.sections), config=config, bias=False)
        dev = self.linear_in.weight.device
        new = lambda n, value: nn.Parameter(torch.full((n,), value, dtype=torch.float32, device=dev))
        self.input_bias, self.forget_bias, self.norm = new(H, 0.0), new(H, 3.0), new(H * DV, 1.0)
        self.linear_proj = RowParallelLinear(H * DV, config.hidden_size, config=config)

    def cache_shape(self):
        return None

    def state_shape(self):
        """Shapes of the state's tensors."""
        s = self.shape
        return [(s.heads, s.dim, s.v_dim), (s.heads, s.dim), (s.heads,)]

    def forward(self, hidden, rotary, meta: AttnMeta):
        layer = cache_layer(meta, self.layer_number)
        proj, _ = self.linear_in(hidden)
        out = recurrent.matrix_memory(proj, self.input_bias, self.forget_bias, self.norm, self.shape, meta.cache.recurrent[layer],
                                      meta.cache, self.eps)
        return self.linear_proj(out)
