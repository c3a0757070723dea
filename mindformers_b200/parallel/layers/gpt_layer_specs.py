"""Layer specs of the GPT family: which classes make up a transformer layer, a decoder stack and an MTP block.

Reference: ``training_graph/base_models/gpt/gpt_layer_specs.py`` (``get_gpt_layer_local_spec`` with its
``num_experts / moe_grouped_gemm / qk_layernorm / multi_latent_attention`` switches, ``get_gpt_decoder_block_spec``
:154-217 with the dense / MoE pattern from ``first_k_dense_replace`` or ``moe_layer_freq``,
``get_gpt_mtp_block_spec``) and ``moe_module_specs.py``. One implementation serves training and inference here, so
one set of specs does too: a model variant changes a spec entry (for instance a different attention class), not the
layer code. ``TransformerLayer`` and ``TransformerBlock`` build themselves from these specs.
"""
from __future__ import annotations

from typing import List, Optional

from ..spec_utils import ModuleSpec
from .attention import CrossAttention, MLASelfAttention, MLASelfAttentionMegatron, SelfAttention
from .delta_rule import GatedDeltaMixer, ParallelMixer
from .matrix_memory import MatrixMemoryMixer
from .mlp import MLP
from .moe import GroupedMLP, MoELayer, SharedExpertMLP, TopKRouter
from .mtp import MultiTokenPredictionBlock, MultiTokenPredictionLayer
from .norm import build_norm
from .ragged_attention import RaggedLatentAttention, RaggedSelfAttention
from .state_space import StateSpaceMixer
from .transformer_layer import (OutputNormTransformerLayer, ParallelTransformerLayer, SandwichTransformerLayer,
                                StreamTransformerLayer, TransformerLayer, TransformerLayerSubmodules)


def get_moe_module_spec(num_experts: Optional[int] = None, moe_grouped_gemm: bool = True) -> ModuleSpec:
    """Spec of the MoE sub-layer (router + grouped experts + optional shared experts). Experts are always the
    grouped-GEMM implementation; ``moe_grouped_gemm=False`` is accepted and means the same module."""
    if not num_experts:
        raise ValueError("an MoE spec needs num_experts")
    return ModuleSpec(module=MoELayer, submodules={"router": TopKRouter, "experts": GroupedMLP,
                                                   "shared_experts": SharedExpertMLP})


def get_mlp_module_spec(num_experts: Optional[int] = None, moe_grouped_gemm: bool = True) -> ModuleSpec:
    """Dense gated MLP, or the MoE sub-layer when ``num_experts`` is given."""
    return get_moe_module_spec(num_experts, moe_grouped_gemm) if num_experts else ModuleSpec(module=MLP)


def get_gpt_layer_local_spec(num_experts: Optional[int] = None, moe_grouped_gemm: bool = True,
                             qk_layernorm: bool = False, multi_latent_attention: bool = False,
                             sandwich_norm: bool = False, use_contiguous_weight_layout: bool = True,
                             mla_qkv_concat: bool = True) -> ModuleSpec:
    """Spec of one pre-LN transformer layer.

    ``qk_layernorm`` and the ``[Q|K|V]`` row layout live in the configuration that the attention reads, so those two
    switches select nothing here. ``mla_qkv_concat=False`` selects the multi-latent attention with one module per
    projection (``linear_q_down_proj`` / ``linear_q_up_proj`` / ``linear_kv_down_proj`` / ``linear_kv_up_proj``)
    instead of the concatenated down-projection."""
    norm = ModuleSpec(module=build_norm)
    mla = MLASelfAttention if mla_qkv_concat else MLASelfAttentionMegatron
    attn = ModuleSpec(module=mla if multi_latent_attention else SelfAttention)
    return ModuleSpec(module=TransformerLayer, submodules=TransformerLayerSubmodules(
        input_layernorm=norm, self_attention=attn, pre_mlp_layernorm=norm,
        mlp=get_mlp_module_spec(num_experts, moe_grouped_gemm),
        post_attn_layernorm=norm if sandwich_norm else None, post_mlp_layernorm=norm if sandwich_norm else None))


def get_output_norm_layer_spec(config) -> ModuleSpec:
    """Spec of one layer whose sub-layer outputs are normalised; a layer without a feed-forward has
    ``ffn_hidden_size == 0``."""
    norm = ModuleSpec(module=build_norm)
    ff = bool(config.ffn_hidden_size)
    return ModuleSpec(module=OutputNormTransformerLayer, submodules=TransformerLayerSubmodules(
        self_attention=ModuleSpec(module=RaggedSelfAttention), mlp=get_mlp_module_spec() if ff else None,
        post_attn_layernorm=norm, post_mlp_layernorm=norm if ff else None))


_MIXERS = {"attention": RaggedSelfAttention, "latent": RaggedLatentAttention, "delta": GatedDeltaMixer,
           "matrix_memory": MatrixMemoryMixer, "state_space": StateSpaceMixer, "parallel": ParallelMixer}


def get_stream_layer_spec(config, is_moe: bool) -> ModuleSpec:
    """Spec of one layer on several residual streams: ``config.mixer``, then an MoE or dense feed-forward (none with
    ``ffn_hidden_size == 0``)."""
    norm = ModuleSpec(module=build_norm)
    mlp = get_mlp_module_spec(config.num_moe_experts if is_moe else None) if is_moe or config.ffn_hidden_size else None
    return ModuleSpec(module=StreamTransformerLayer, submodules=TransformerLayerSubmodules(
        input_layernorm=norm, self_attention=ModuleSpec(module=_MIXERS[config.mixer]), mlp=mlp,
        pre_mlp_layernorm=norm if mlp is not None else None))


def get_sandwich_layer_spec(config, is_moe: bool) -> ModuleSpec:
    """Spec of one layer with norms on both sides of its sub-layers: ``config.mixer``, then an MoE or dense feed-forward
    (none with ``ffn_hidden_size == 0``)."""
    norm = ModuleSpec(module=build_norm)
    mlp = get_mlp_module_spec(config.num_moe_experts if is_moe else None) if is_moe or config.ffn_hidden_size else None
    after = norm if mlp is not None else None
    return ModuleSpec(module=SandwichTransformerLayer, submodules=TransformerLayerSubmodules(
        input_layernorm=norm, self_attention=ModuleSpec(module=_MIXERS[config.mixer]), post_attn_layernorm=norm, mlp=mlp,
        pre_mlp_layernorm=after, post_mlp_layernorm=after))


def get_parallel_layer_spec(config, is_moe: bool) -> ModuleSpec:
    """Spec of one layer whose sub-layers read one norm: ``config.mixer`` beside an MoE or dense feed-forward (none with
    ``ffn_hidden_size == 0``)."""
    mlp = get_mlp_module_spec(config.num_moe_experts if is_moe else None) if is_moe or config.ffn_hidden_size else None
    return ModuleSpec(module=ParallelTransformerLayer, submodules=TransformerLayerSubmodules(
        input_layernorm=ModuleSpec(module=build_norm), self_attention=ModuleSpec(module=_MIXERS[config.mixer]), mlp=mlp))


def get_gpt_layer_spec_for_config(config, is_moe: bool) -> ModuleSpec:
    """``get_gpt_layer_local_spec`` with the switches taken from a ``TransformerConfig``."""
    if config.residual_streams:
        if config.norm_placement != "input" or not config.ragged_attention or config.normalization != "RMSNorm":
            raise ValueError("layers on residual streams are pre-norm layers with RMS norms and ragged attention")
        return get_stream_layer_spec(config, is_moe)
    if config.norm_placement == "both":
        if not config.ragged_attention or config.normalization != "RMSNorm":
            raise ValueError("layers with norms on both sides are built with ragged attention and RMS norms")
        return get_sandwich_layer_spec(config, is_moe)
    if config.norm_placement == "parallel":
        if not config.ragged_attention or config.normalization != "RMSNorm" or config.layernorm_zero_centered_gamma:
            raise ValueError("layers whose sub-layers run side by side are built with ragged attention and plain RMS norms")
        return get_parallel_layer_spec(config, is_moe)
    if config.norm_placement == "output":
        if is_moe or not config.ragged_attention:
            raise ValueError("output-normalised layers are built with ragged attention and a dense feed-forward")
        return get_output_norm_layer_spec(config)
    return get_gpt_layer_local_spec(
        num_experts=config.num_moe_experts if is_moe else None, moe_grouped_gemm=True,
        qk_layernorm=bool(getattr(config, "qk_layernorm", False)),
        multi_latent_attention=bool(config.multi_latent_attention), sandwich_norm=bool(config.sandwich_norm),
        mla_qkv_concat=bool(getattr(config, "mla_qkv_concat", True)))


def get_gpt_decoder_block_spec(config) -> List[ModuleSpec]:
    """One layer spec per layer of the whole model: dense or MoE after ``config.moe_layer_pattern()``
    (``first_k_dense_replace`` wins over ``moe_layer_freq``). A pipeline stage picks its own layers from the list."""
    if config.layer_overrides:
        return [get_gpt_layer_spec_for_config(config.for_layer(i), bool(flag))
                for i, flag in enumerate(config.moe_layer_pattern())]
    dense = get_gpt_layer_spec_for_config(config, False)
    moe = get_gpt_layer_spec_for_config(config, True) if config.num_moe_experts else None
    return [moe if flag else dense for flag in config.moe_layer_pattern()]


def get_gpt_mtp_block_spec(config) -> Optional[ModuleSpec]:
    """Spec of the multi-token-prediction block (None without MTP layers): every MTP layer wraps one transformer layer
    of the kind the last decoder layer has."""
    if not getattr(config, "mtp_num_layers", 0):
        return None
    pattern = config.moe_layer_pattern()
    inner = get_gpt_layer_spec_for_config(config, bool(pattern[-1]) if pattern else False)
    return ModuleSpec(module=MultiTokenPredictionBlock,
                      submodules={"layer": ModuleSpec(module=MultiTokenPredictionLayer,
                                                      submodules={"transformer_layer": inner})})
