"""Pre-LN transformer layer and the layer stack.

Reference: ``training_graph/transformer/transformer_layer.py`` (:74-250: input_layernorm →
self_attention → residual add → pre_mlp_layernorm → mlp → residual add, returning the extra (MoE) loss)
and ``transformer_block.py`` (:79-197: per-layer specs, final norm, loss threading), plus the layer →
pipeline-stage assignment with ``offset`` of ``training_graph/transformer/utils.py:93-159``.

The residual add of each sub-layer is folded into the following RMSNorm kernel: a layer receives the
pending sub-layer output and the residual stream and returns the same pair.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, List, Optional

import torch
import torch.nn as nn
from torch.utils.checkpoint import checkpoint

from .. import parallel_state as ps
from ...ops import stream
from ..spec_utils import build_module
from .attention import AttnMeta
from .moe import MoELayer
from .norm import build_norm


@dataclass
class TransformerLayerSubmodules:
    """What a layer is made of, as ``ModuleSpec`` entries (``gpt_layer_specs.py`` fills them in). Norm entries are
    built with ``(config)``, the attention and an MoE ``mlp`` with ``(config, layer_number)``, a dense ``mlp`` with
    ``(config)``; ``None`` for a post-norm leaves it out."""
    input_layernorm: Any = None
    self_attention: Any = None
    pre_mlp_layernorm: Any = None
    mlp: Any = None
    post_attn_layernorm: Any = None
    post_mlp_layernorm: Any = None


class TransformerLayer(nn.Module):
    """Pre-LN block: ``input_layernorm`` → ``self_attention`` → ``pre_mlp_layernorm`` → ``mlp`` (dense or MoE), optional
    sandwich norms; the residual adds are folded into the norms. Built from a ``TransformerLayerSubmodules`` spec
    (reference ``training_graph/transformer/transformer_layer.py:74-250``)."""

    def __init__(self, config, layer_number: int = 1, is_moe: bool = False,
                 submodules: Optional[TransformerLayerSubmodules] = None):
        super().__init__()
        self.config = config
        self.layer_number = layer_number
        if submodules is None:     # the layer that the configuration describes
            from .gpt_layer_specs import get_gpt_layer_spec_for_config
            submodules = get_gpt_layer_spec_for_config(config, is_moe).submodules
        self.input_layernorm = build_module(submodules.input_layernorm, config)
        self.self_attention = build_module(submodules.self_attention, config, layer_number)
        self.pre_mlp_layernorm = build_module(submodules.pre_mlp_layernorm, config)
        mlp_spec = submodules.mlp
        mlp_cls = getattr(mlp_spec, "module", mlp_spec)
        self.is_moe = isinstance(mlp_cls, type) and issubclass(mlp_cls, MoELayer)
        self.mlp = build_module(mlp_spec, config, layer_number) if self.is_moe else build_module(mlp_spec, config)
        self.post_attn_layernorm = (build_module(submodules.post_attn_layernorm, config)
                                    if submodules.post_attn_layernorm is not None else None)
        self.post_mlp_layernorm = (build_module(submodules.post_mlp_layernorm, config)
                                   if submodules.post_mlp_layernorm is not None else None)
        self.hidden_dropout = float(getattr(config, "hidden_dropout", 0.0) or 0.0)

    def _dropout(self, x):
        """Hidden dropout on a sub-layer output before it joins the residual (reference ``bias_dropout_add``,
        ``transformer_layer.py:215-250``). Under sequence parallelism every tensor-parallel rank holds other tokens, so
        the mask comes from the tensor-parallel random stream (different per rank); otherwise the ranks hold the same
        activations and draw the same mask from the default stream."""
        if self.hidden_dropout <= 0.0 or not self.training:
            return x
        cfg = self.config
        if cfg.sequence_parallel and ps.get_tensor_model_parallel_world_size() > 1:
            from ...modules.rng import get_rng_tracker
            tracker = get_rng_tracker()
            if "model-parallel-rng" in tracker.states:
                with tracker.fork():
                    return torch.nn.functional.dropout(x, self.hidden_dropout, True)
        return torch.nn.functional.dropout(x, self.hidden_dropout, True)

    def forward(self, pending, residual, rotary, meta: AttnMeta):
        """``pending``: sub-layer output not yet added to ``residual`` (``residual`` None for the first layer)."""
        if residual is None:
            residual = pending
            normed = self.input_layernorm(pending)
        else:
            normed, residual = self.input_layernorm(pending, residual)
        attn_out, _ = self.self_attention(normed, rotary, meta)
        if self.post_attn_layernorm is not None:
            attn_out = self.post_attn_layernorm(attn_out)
        attn_out = self._dropout(attn_out)
        normed, residual = self.pre_mlp_layernorm(attn_out, residual)
        aux = None
        if self.is_moe:
            mlp_out, aux = self.mlp(normed)
        else:
            mlp_out, _ = self.mlp(normed)
        if self.post_mlp_layernorm is not None:
            mlp_out = self.post_mlp_layernorm(mlp_out)
        return self._dropout(mlp_out), residual, aux


class OutputNormTransformerLayer(nn.Module):
    """Layer with a 32-bit residual stream and norms on the sub-layer OUTPUTS only: ``x <- x + scale1 * norm1(attention(x))``,
    then ``x <- x + scale2 * norm2(mlp(x))`` (no second half without an ``mlp``; no scales without ``config.layer_scale``).
    A serving layer: projection bias, norm, scale and residual add are one kernel (``ops/stream.py::add_normed``).

    ``forward(pending, residual, ...)`` takes and returns the stream twice: ``pending`` in the activation dtype (the next
    sub-layer's input) and ``residual`` in fp32 (None before the first layer)."""

    stream_in_residual = True      # the result is ``residual`` alone; nothing is left to be added

    def __init__(self, config, layer_number: int = 1, submodules: Optional[TransformerLayerSubmodules] = None):
        super().__init__()
        self.config, self.layer_number = config, layer_number
        self.self_attention = build_module(submodules.self_attention, config, layer_number)
        self.post_attn_layernorm = build_module(submodules.post_attn_layernorm, config)
        self.mlp = build_module(submodules.mlp, config) if submodules.mlp is not None else None
        self.post_mlp_layernorm = build_module(submodules.post_mlp_layernorm, config) if self.mlp is not None else None

        def scale():
            ref = self.post_attn_layernorm.weight
            return nn.Parameter(torch.ones_like(ref)) if config.layer_scale else None
        self.register_parameter("attn_layer_scale", scale())
        self.register_parameter("mlp_layer_scale", scale() if self.mlp is not None else None)

    def _add(self, residual, pending, y, bias, norm, scale):
        return stream.add_normed(pending if residual is None else residual, y, bias, norm.weight, getattr(norm, "bias", None),
                                 scale, norm.eps, hasattr(norm, "bias"), inplace=residual is not None)

    def forward(self, pending, residual, rotary, meta: AttnMeta):
        y, bias = self.self_attention(pending, rotary, meta)
        pending, residual = self._add(residual, pending, y, bias, self.post_attn_layernorm, self.attn_layer_scale)
        if self.mlp is not None:
            y, bias = self.mlp(pending)
            pending, residual = self._add(residual, pending, y, bias, self.post_mlp_layernorm, self.mlp_layer_scale)
        return pending, residual, None


class StreamConnection(nn.Module):
    """How one sub-layer is tied to ``n`` residual streams: its input is ``sum_s read[s] x_s``, and its output ``y`` enters as
    ``x_t <- sum_s mix[s, t] x_s + write[t] y``. fp32."""

    def __init__(self, n: int, device=None):
        super().__init__()
        def param(t):
            return nn.Parameter(t.to(device))
        self.read = param(torch.full((n,), 1.0 / n))
        self.write = param(torch.ones(n))
        self.mix = param(torch.eye(n))


@dataclass
class ResidualStreams:
    """The streams ``x`` (``[T, n, W]`` fp32, or the embedding before the first update) and the connection of the sub-layer
    whose output has not entered them yet."""
    x: torch.Tensor
    link: Optional[StreamConnection] = None


class StreamTransformerLayer(nn.Module):
    """Pre-norm layer on several fp32 residual streams (hyper-connections): mixer, then a feed-forward (dense or MoE; none
    without an ``mlp``), each with a ``StreamConnection``. A serving layer: between two sub-layers, the update of the
    streams, the next read and its norm are one kernel (``ops/stream.py::residual_streams``), across layers too, since the
    output of a layer's last sub-layer stays pending."""

    residual_streams = True       # ``residual`` is a ``ResidualStreams`` that still lacks ``pending``

    def __init__(self, config, layer_number: int = 1, submodules: Optional[TransformerLayerSubmodules] = None):
        super().__init__()
        self.config, self.layer_number = config, layer_number
        dev = getattr(config, "device", None)
        self.input_layernorm = build_module(submodules.input_layernorm, config)
        self.self_attention = build_module(submodules.self_attention, config, layer_number)
        self.mixer_connection = StreamConnection(config.residual_streams, dev)
        self.mlp = self.pre_mlp_layernorm = self.mlp_connection = None
        if submodules.mlp is not None:
            mlp_cls = getattr(submodules.mlp, "module", submodules.mlp)
            self.is_moe = isinstance(mlp_cls, type) and issubclass(mlp_cls, MoELayer)
            self.pre_mlp_layernorm = build_module(submodules.pre_mlp_layernorm, config)
            self.mlp = build_module(submodules.mlp, config, layer_number) if self.is_moe else build_module(submodules.mlp, config)
            self.mlp_connection = StreamConnection(config.residual_streams, dev)

    def _enter(self, pending, streams: ResidualStreams, link: StreamConnection, norm):
        """Let ``pending`` enter the streams; returns the input of the sub-layer behind ``link`` and the streams it leaves."""
        old = streams.link
        h, x = stream.residual_streams(streams.x, self.config.residual_streams, pending if old is not None else None,
                                       None if old is None else old.mix, None if old is None else old.write, link.read,
                                       norm.weight, norm.eps)
        return h, ResidualStreams(x, link)

    def forward(self, pending, residual: Optional[ResidualStreams], rotary, meta: AttnMeta):
        if residual is None:                       # the embedding: every stream is equal to it
            residual = ResidualStreams(pending)
        h, residual = self._enter(pending, residual, self.mixer_connection, self.input_layernorm)
        pending, _ = self.self_attention(h, rotary, meta)
        aux = None
        if self.mlp is not None:
            h, residual = self._enter(pending, residual, self.mlp_connection, self.pre_mlp_layernorm)
            pending, aux = self.mlp(h)
        return pending, residual, aux if self.mlp is not None and self.is_moe else None


@dataclass
class NormedResidual:
    """The fp32 stream and the norm through which the pending sub-layer output has yet to enter it (None: nothing pends)."""
    x: torch.Tensor
    norm: Any = None


class SandwichTransformerLayer(nn.Module):
    """Layer with an fp32 residual stream and norms on both sides of every sub-layer: ``x <- x + norm_b(mixer(norm_a(x)))``,
    then the same with the feed-forward (dense or MoE; none without an ``mlp``). With ``config.token_shift`` the mixer reads
    ``h + (h of the token before - h) * mu``. A serving layer: entering the stream, the next norm and the shift are one kernel
    (``ops/stream.py::normed_step``), across layers too, since a layer's last output stays pending."""

    normed_residual = True        # ``residual`` is a ``NormedResidual`` that still lacks ``pending``

    def __init__(self, config, layer_number: int = 1, submodules: Optional[TransformerLayerSubmodules] = None):
        super().__init__()
        self.config, self.layer_number = config, layer_number
        self.input_layernorm = build_module(submodules.input_layernorm, config)
        self.self_attention = build_module(submodules.self_attention, config, layer_number)
        self.post_attn_layernorm = build_module(submodules.post_attn_layernorm, config)
        self.register_parameter("token_shift", nn.Parameter(torch.zeros_like(self.input_layernorm.weight))
                                if config.token_shift else None)
        self.mlp = self.pre_mlp_layernorm = self.post_mlp_layernorm = None
        self.is_moe = False
        if submodules.mlp is not None:
            mlp_cls = getattr(submodules.mlp, "module", submodules.mlp)
            self.is_moe = isinstance(mlp_cls, type) and issubclass(mlp_cls, MoELayer)
            self.pre_mlp_layernorm = build_module(submodules.pre_mlp_layernorm, config)
            self.mlp = build_module(submodules.mlp, config, layer_number) if self.is_moe else build_module(submodules.mlp, config)
            self.post_mlp_layernorm = build_module(submodules.post_mlp_layernorm, config)

    def _enter(self, pending, res: NormedResidual, norm, meta: AttnMeta, step=None, shift=None):
        """Let ``pending`` enter the stream; returns the input of the sub-layer behind ``norm`` and the new stream."""
        carry = None
        if shift is not None:
            if meta.cache is None:
                raise RuntimeError("token shift serves from a cache: generate() or the serving engine provide one")
            carry = stream.Carry(shift, meta.cache, meta.layer_run - meta.cache.layer_offset)
        return stream.normed_step(res.x, pending if res.norm is not None else None, res.norm.weight if res.norm is not None else None,
                                  step, norm.weight, norm.eps, self.config.layernorm_zero_centered_gamma, carry)

    def forward(self, pending, residual: Optional[NormedResidual], rotary, meta: AttnMeta):
        if residual is None:
            residual = NormedResidual(pending)
        h, x = self._enter(pending, residual, self.input_layernorm, meta, meta.loop_step, self.token_shift)
        pending, _ = self.self_attention(h, rotary, meta)
        residual, aux = NormedResidual(x, self.post_attn_layernorm), None
        if self.mlp is not None:
            h, x = self._enter(pending, residual, self.pre_mlp_layernorm, meta)
            pending, aux = self.mlp(h)
            residual = NormedResidual(x, self.post_mlp_layernorm)
        return pending, residual, aux if self.is_moe else None


@dataclass
class JointResidual:
    """The fp32 stream and the mixer's output that has yet to enter it beside the pending one of the feed-forward."""
    x: torch.Tensor
    mixed: Optional[torch.Tensor] = None


class ParallelTransformerLayer(nn.Module):
    """Layer with an fp32 residual stream whose sub-layers read one norm and run side by side: ``x <- x + (mixer(h') + mlp(h))``
    with ``h`` the RMS norm of ``x`` in ``config.norm_groups`` parts, and ``h' = h + conv(h)``, a causal convolution per channel,
    with ``config.input_conv_taps`` (else ``h``). The feed-forward is dense, MoE or absent. A serving layer: entering the stream,
    the next norm and the convolution are one kernel (``ops/stream.py::joint_step``), across layers too, since a layer's outputs
    stay pending. Before the first layer of a pass of a loop, ``x <- W [x; embedding output] + step`` (``AttnMeta.loop_entry``)."""

    joint_residual = True         # ``residual`` is a ``JointResidual`` that still lacks ``pending``

    def __init__(self, config, layer_number: int = 1, submodules: Optional[TransformerLayerSubmodules] = None):
        super().__init__()
        self.config, self.layer_number = config, layer_number
        self.input_layernorm = build_module(submodules.input_layernorm, config)
        self.self_attention = build_module(submodules.self_attention, config, layer_number)
        taps, w = int(config.input_conv_taps or 0), self.input_layernorm.weight
        self.register_parameter("input_conv", nn.Parameter(torch.empty(taps, w.numel(), dtype=torch.float32, device=w.device)
                                                           .normal_(0.0, 0.3)) if taps else None)
        self.mlp, self.is_moe = None, False
        if submodules.mlp is not None:
            mlp_cls = getattr(submodules.mlp, "module", submodules.mlp)
            self.is_moe = isinstance(mlp_cls, type) and issubclass(mlp_cls, MoELayer)
            self.mlp = build_module(submodules.mlp, config, layer_number) if self.is_moe else build_module(submodules.mlp, config)

    def forward(self, pending, residual: Optional[JointResidual], rotary, meta: AttnMeta):
        x, ys = (pending, ()) if residual is None else (residual.x, (pending, residual.mixed))
        norm, base, step = self.input_layernorm, None, meta.loop_step
        dtype, groups = norm.weight.dtype, self.config.norm_groups
        if meta.loop_step is not None and meta.loop_entry is not None:
            w, base = meta.loop_entry
            x, ys = stream.linear(stream.joint_step(x, ys, None, None, None, 1, 0.0, dtype, keep=False)[0], w,
                                  out_dtype=torch.float32).contiguous(), ()        # rows of odd widths lie in a padded matrix
        conv = None
        if self.input_conv is not None:
            if meta.cache is None:
                raise RuntimeError("the convolution serves from a cache: generate() or the serving engine provide one")
            conv = stream.InputConv(self.input_conv, meta.cache, meta.layer_run - meta.cache.layer_offset)
        h, mixed, x = stream.joint_step(x, ys, base, step, norm.weight, groups, norm.eps, dtype, conv,
                                        want_h=conv is None or self.mlp is not None)
        mixed, _ = self.self_attention(h if conv is None else mixed, rotary, meta)
        if self.mlp is None:
            return mixed, JointResidual(x), None
        pending, aux = self.mlp(h)
        return pending, JointResidual(x, mixed), aux if self.is_moe else None


def pipeline_layer_split(num_layers: int, pp: int, vpp: int = 1, offset=0) -> List[List[List[int]]]:
    """Layer ids of every (pp stage, virtual chunk). ``offset`` adds/removes layers per stage
    (list of pp values, or vpp lists of pp values), as the reference's ``LayerSetting`` does."""
    vpp = vpp or 1
    chunks = pp * vpp
    base = num_layers // chunks
    if isinstance(offset, int):
        if offset != 0:
            raise ValueError("a scalar offset must be 0; give a list with one value per stage")
        off = [[0] * pp for _ in range(vpp)]
    else:
        off = [list(o) for o in offset] if offset and isinstance(offset[0], (list, tuple)) else [list(offset)]
        if len(off) != vpp or any(len(o) != pp for o in off):
            raise ValueError(f"offset must hold {vpp} x {pp} values, got {offset!r}")
    counts = [[base + off[v][s] for s in range(pp)] for v in range(vpp)]
    if sum(sum(c) for c in counts) != num_layers:
        raise ValueError(f"layers per stage {counts} do not add up to num_layers={num_layers}")
    out = [[[] for _ in range(vpp)] for _ in range(pp)]
    nxt = 0
    for v in range(vpp):
        for s in range(pp):
            out[s][v] = list(range(nxt, nxt + counts[v][s]))
            nxt += counts[v][s]
    return out


class StageLayers(nn.Module):
    """The layers of one pipeline stage, registered under their GLOBAL layer number: a parameter of the sixth layer of
    the model is ``layers.5.…`` on whichever stage owns it, so checkpoints, weight loaders and resharding tools see
    one name space for every pipeline layout (the reference numbers layers globally per stage,
    ``training_graph/transformer/utils.py:129-159``). Iteration and integer indexing are over the stage's own
    layers in order (``layers[0]`` is the first layer of this stage), as with a ``ModuleList``."""

    def __init__(self, layer_ids, modules):
        super().__init__()
        self.layer_ids = list(layer_ids)
        for gid, mod in zip(self.layer_ids, modules):
            self.add_module(str(gid), mod)

    def __len__(self):
        return len(self.layer_ids)

    def __iter__(self):
        return (self._modules[str(g)] for g in self.layer_ids)

    def __getitem__(self, idx):
        if isinstance(idx, slice):
            return [self._modules[str(g)] for g in self.layer_ids[idx]]
        return self._modules[str(self.layer_ids[idx])]


class TransformerBlock(nn.Module):
    """The layers owned by this pipeline stage (and virtual chunk) plus, on the last stage, the final norm."""

    def __init__(self, config, pre_process: bool = True, post_process: bool = True, vp_stage: Optional[int] = None,
                 base_seed: Optional[int] = None):
        super().__init__()
        self.config = config
        base_seed = torch.initial_seed() if base_seed is None else base_seed
        dev = getattr(config, "device", None)
        pp = ps.get_pipeline_model_parallel_world_size()
        pp_rank = ps.get_pipeline_model_parallel_rank()
        vpp = config.virtual_pipeline_model_parallel_size or 1
        split = pipeline_layer_split(config.num_layers, pp, vpp, config.offset or 0)
        self.layer_ids = split[pp_rank][vp_stage or 0]
        from .gpt_layer_specs import get_gpt_decoder_block_spec
        layer_specs = get_gpt_decoder_block_spec(config)      # one spec per layer of the whole model
        from ..init_method import module_rng
        built = []
        owners = [config.shares_weights_with(i) for i in self.layer_ids]
        if any(o not in self.layer_ids for o in owners):
            raise NotImplementedError("layers that share weights must be on one pipeline stage")
        own_ids = [i for i, o in zip(self.layer_ids, owners) if o == i]
        for i in own_ids:
            with module_rng(base_seed, 100 + i, dev):     # a layer's initial weights depend on its number only
                built.append(build_module(layer_specs[i], config.for_layer(i), layer_number=i + 1))
        self.layers = StageLayers(own_ids, built)
        # the layers in running order: a layer that shares weights is its owner's module once more, a looped layer runs in
        # every pass; every run has a number (``run_ids``), and with it a cache, of its own
        self.run_order, self.run_ids = [own_ids.index(o) for o in owners], list(self.layer_ids)
        self.run_steps = [None] * len(self.run_order)
        self.register_parameter("loop_step", None)
        self.register_parameter("loop_in", None)
        if config.layer_loop is not None:
            if pp * vpp > 1:
                raise NotImplementedError("looped layers stay on one pipeline stage")
            runs = config.layer_runs()
            self.run_order, self.run_ids = [own_ids.index(i) for i, _ in runs], list(range(len(runs)))
            self.run_steps = [t for _, t in runs]
            with module_rng(base_seed, 90, dev):
                def rand(*shape):
                    return nn.Parameter(torch.empty(*shape, dtype=torch.float32,
                                                    device=dev or ("cuda" if torch.cuda.is_available() else "cpu"))
                                        .normal_(0.0, config.init_method_std).to(config.params_dtype))
                self.loop_step = rand(int(config.layer_loop[2]), config.hidden_size)
                if config.loop_input:
                    self.loop_in = rand(config.hidden_size, 2 * config.hidden_size)
        self.final_layernorm = build_norm(config) if post_process else None
        self.recompute = bool(config.recompute) if not isinstance(config.recompute, (list, tuple)) else True
        self._recompute_layers = self._resolve_recompute(config.recompute)
        self._setup_selective_recompute_and_offload(config)
        # ``grads_final_hook(layer_id)``: set by the optimizer for the forward pass of a step's last micro-batch; it is
        # called during the backward pass as soon as every gradient of that layer's parameters has been written
        self.grads_final_hook = None
        # ``params_ready_hook(layer_id)``: set by the optimizer while it still publishes updated parameters; called
        # before a layer runs, it makes the stream wait for that layer's parameters
        self.params_ready_hook = None

    # reference defaults of ``select_recompute: true`` (``training_graph/transformer/utils.py:107-110``): the gated
    # activation of the MLP and of the shared experts; here these, the norms and the rotary embedding are what a
    # selectively recomputed layer runs twice, whatever the patterns say, because nothing else is cheap
    _DEFAULT_SELECT = (r"mlp\.mul", r"mlp\.activation_func\.silu", r"mlp\.shared_experts\.mul",
                       r"mlp\.shared_experts\.activation_func\.silu", r".*\.norm")

    @property
    def num_runs(self) -> int:
        """Layer runs of this stage (each has a cache of its own); above ``len(layers)`` when layers share weights."""
        return len(self.run_order)

    def cache_shapes(self):
        """``(kv heads, key size, value size)`` per layer run (None: it caches no keys), or None for attention without
        per-layer cache shapes."""
        shapes = [getattr(self.layers[at].self_attention, "cache_shape", None) for at in self.run_order]
        return [s() for s in shapes] if shapes and all(s is not None for s in shapes) else None

    def state_shapes(self):
        """Per layer run the recurrent state's shape (``KVCacheContext``) or None; None when no layer has one."""
        shapes = [getattr(self.layers[at].self_attention, "state_shape", lambda: None)() for at in self.run_order]
        return shapes if any(s is not None for s in shapes) else None

    def carry_width(self) -> int:
        """Width of the vector that every layer run carries from one token of a sequence to the next (0: none): one row of the
        width for a token shift, ``taps - 1`` rows for a convolution in front of the mixers."""
        rows = [1 if getattr(layer, "token_shift", None) is not None else 0 for layer in self.layers]
        rows += [layer.input_conv.shape[0] - 1 for layer in self.layers if getattr(layer, "input_conv", None) is not None]
        return self.config.hidden_size * max(rows, default=0)

    def _setup_selective_recompute_and_offload(self, config):
        from ..recompute import ActivationOffloader, mark_recompute_modules
        n = len(self.layer_ids)
        sel = getattr(config, "select_recompute", False)
        patterns, count = [], 0
        if isinstance(sel, dict):                       # {pattern: layers per stage}
            patterns, count = list(sel.keys()), n
            counts = [self._resolve_recompute(v) for v in sel.values()]
            count = max(counts) if counts else 0
        elif isinstance(sel, (list, tuple)) and sel and all(isinstance(x, str) for x in sel):
            patterns, count = list(sel), n
        else:
            count = self._resolve_recompute(sel)
        self._select_layers = count
        extra = [p for p in patterns if p not in self._DEFAULT_SELECT]
        self._select_matched = []
        for layer in self.layers[:count]:
            self._select_matched += mark_recompute_modules(layer, extra)
        ignored = [k for k in ("recompute_slice_activation", "select_comm_recompute", "parallel_optimizer_comm_recompute")
                   if getattr(config, k, False)]
        if ignored:
            from ...tools.logger import logger
            logger.warning("recompute options without effect here: %s (the fused GEMM + collective kernels leave no "
                           "separate communication output to recompute, activations are not sliced)", ignored)
        # offload: ``swap: true`` with ``layer_swap`` = number of layers (or a list of {layers, backward_prefetch})
        self._offload = None
        self._offload_layers = set()
        if getattr(config, "cpu_offloading", False):
            spec = getattr(config, "cpu_offloading_num_layers", None)
            prefetch = int(getattr(config, "default_prefetch", 1) or 1)
            if isinstance(spec, (list, tuple)) and spec and isinstance(spec[0], dict):
                for entry in spec:
                    ids = entry.get("layers", True)
                    prefetch = int(entry.get("backward_prefetch", prefetch) or prefetch)
                    self._offload_layers |= set(range(n)) if ids is True else {int(i) for i in ids if int(i) < n}
            else:
                k = n if spec in (None, True) else min(int(spec), n)
                self._offload_layers = set(range(k))
            self._offload = ActivationOffloader(prefetch=prefetch)

    def _resolve_recompute(self, rc):
        n = len(self.layer_ids)
        if isinstance(rc, bool):
            return n if rc else 0
        if isinstance(rc, int):
            return min(rc, n)
        if isinstance(rc, (list, tuple)) and rc:
            pp_rank = ps.get_pipeline_model_parallel_rank()
            val = rc[pp_rank] if pp_rank < len(rc) else rc[-1]
            if isinstance(val, (list, tuple)):
                val = val[0]
            return n if val is True else int(val or 0)
        return 0

    def forward(self, hidden, rotary, meta: AttnMeta):
        pending, residual, layer = hidden, None, None
        aux_total = None
        training = self.training and torch.is_grad_enabled()
        if self.loop_in is not None:          # the embedding's part of every pass's first product
            W, w = self.config.hidden_size, self.loop_in
            x0 = stream.joint_step(hidden, (), None, None, None, 1, 0.0, w.dtype, keep=False)[0]
            meta.loop_entry = (w[:, :W], stream.linear(x0, w[:, W:], out_dtype=torch.float32))
        if training and self._offload is not None:
            self._offload.prune()
        for idx, at in enumerate(self.run_order):
            layer = run = self.layers[at]
            meta.layer_run = self.run_ids[idx]
            if self.loop_step is not None:
                meta.loop_step = None if self.run_steps[idx] is None else self.loop_step[self.run_steps[idx]]
            if self.params_ready_hook is not None:
                self.params_ready_hook(self.layers.layer_ids[at])
            if training and self.grads_final_hook is not None and pending.requires_grad:
                # the gradient of a layer's input is the last thing its backward pass produces
                def fire(_grad, _cb=self.grads_final_hook, _gid=self.layers.layer_ids[at]):
                    _cb(_gid)
                pending.register_hook(fire)
            if training and self._offload is not None and idx in self._offload_layers:
                def run(p, r, ro, m, _layer=layer, _idx=idx):     # saved tensors of this layer go to pinned host memory
                    with self._offload.layer(_idx):
                        return _layer(p, r, ro, m)
            if training and idx < self._recompute_layers:
                pending, residual, aux = checkpoint(run, pending, residual, rotary, meta, use_reentrant=False)
            elif training and idx < self._select_layers:
                from ..recompute import selective_checkpoint
                pending, residual, aux = selective_checkpoint(run, pending, residual, rotary, meta)
            else:
                pending, residual, aux = run(pending, residual, rotary, meta)
            if aux is not None:
                aux_total = aux if aux_total is None else aux_total + aux
        if getattr(layer, "residual_streams", False):
            norm, old = self.final_layernorm, residual.link
            if norm is None:
                raise NotImplementedError("residual streams stay on one pipeline stage")
            out, _ = stream.residual_streams(residual.x, old.read.numel(), pending, old.mix, old.write, None, norm.weight,
                                             norm.eps, keep=False)
        elif getattr(layer, "normed_residual", False):
            norm = self.final_layernorm
            if norm is None:
                raise NotImplementedError("an fp32 stream with a pending norm stays on one pipeline stage")
            out, _ = stream.normed_step(residual.x, pending, residual.norm.weight, None, norm.weight, norm.eps,
                                        self.config.layernorm_zero_centered_gamma, keep=False)
        elif getattr(layer, "joint_residual", False):
            norm = self.final_layernorm
            if norm is None:
                raise NotImplementedError("an fp32 stream with pending outputs stays on one pipeline stage")
            out = stream.joint_step(residual.x, (pending, residual.mixed), None, None, norm.weight, self.config.norm_groups, norm.eps,
                                    norm.weight.dtype, keep=False)[0]
        elif getattr(layer, "stream_in_residual", False):
            norm = self.final_layernorm
            out = residual if norm is None else stream.norm_stream(residual, norm.weight, getattr(norm, "bias", None), norm.eps,
                                                                   hasattr(norm, "bias"))
        elif self.final_layernorm is not None:
            if residual is None:
                out = self.final_layernorm(pending)
            else:
                out, _ = self.final_layernorm(pending, residual)
        else:
            out = pending if residual is None else pending + residual
        return out, aux_total
