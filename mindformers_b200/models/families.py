"""Model families: configuration classes and ``…ForCausalLM`` classes, registered for YAML and Auto lookup.

Reference: ``models/llama`` (legacy), ``models/qwen2``, ``models/qwen3``, ``models/qwen3_moe``,
``models/deepseek3`` (mcore shims) and the research families (Llama-3.1, Qwen2.5, Mixtral, TeleChat2, GLM-4),
which here differ only in configuration defaults: all of them are instances of the same ``GPTModel``.
"""
from __future__ import annotations

import copy

from ..parallel.transformer_config_utils import ALIASES
from ..tools.register import MindFormerModuleType, MindFormerRegister
from .configuration_utils import PretrainedConfig
from .modeling_utils import PreTrainedModel

_BASE = dict(vocab_size=32000, hidden_size=4096, intermediate_size=11008, num_hidden_layers=32, num_attention_heads=32,
             num_key_value_heads=None, rms_norm_eps=1e-6, rope_theta=10000.0, max_position_embeddings=4096,
             tie_word_embeddings=False, pad_token_id=0, bos_token_id=1, eos_token_id=2)


def _config(name, model_type, defaults, is_mla=False):
    base = dict(_BASE)
    base.update(defaults)

    class _Cfg(PretrainedConfig):
        @classmethod
        def default_values(cls):
            return dict(base)

    _Cfg.__name__ = _Cfg.__qualname__ = name
    _Cfg.__doc__ = (f"Configuration of the ``{model_type}`` family with Hugging Face key names; defaults: "
                    + ", ".join(f"{k}={v!r}" for k, v in sorted(defaults.items())) + ".")
    _Cfg.model_type = model_type
    _Cfg.is_mla = is_mla
    MindFormerRegister.register_cls(_Cfg, MindFormerModuleType.CONFIG, alias=name)
    MindFormerRegister.register_cls(_Cfg, MindFormerModuleType.CONFIG, alias=name, legacy=False)
    return _Cfg


def _model(name, cfg_cls, family):
    class _M(PreTrainedModel):
        config_class = cfg_cls
        weight_family = family

    _M.__name__ = _M.__qualname__ = name
    _M.__doc__ = (f"Causal language model of the ``{family}`` family: ``{cfg_cls.__name__}`` → ``GPTModel``; Hugging Face "
                  f"checkpoints are mapped by the ``{family}`` name rules (``checkpoint/name_maps.py``).")
    MindFormerRegister.register_cls(_M, MindFormerModuleType.MODELS, alias=name)
    MindFormerRegister.register_cls(_M, MindFormerModuleType.MODELS, alias=name, legacy=False)
    return _M


LlamaConfig = _config("LlamaConfig", "llama", dict(rms_norm_eps=1e-5))
Qwen2Config = _config("Qwen2Config", "qwen2", dict(vocab_size=152064, attention_bias=True, rope_theta=1e6))
Qwen3Config = _config("Qwen3Config", "qwen3", dict(vocab_size=151936, qk_layernorm=True, head_dim=128, rope_theta=1e6))
Qwen3MoeConfig = _config("Qwen3MoeConfig", "qwen3_moe",
                         dict(vocab_size=151936, qk_layernorm=True, head_dim=128, rope_theta=1e6, num_experts=128,
                              num_experts_per_tok=8, moe_intermediate_size=768, norm_topk_prob=True,
                              first_k_dense_replace=0, moe_router_score_function="softmax"))
DeepseekV3Config = _config("DeepseekV3Config", "deepseek_v3",
                           dict(vocab_size=129280, hidden_size=7168, intermediate_size=18432, num_hidden_layers=61,
                                num_attention_heads=128, num_key_value_heads=128, n_routed_experts=256,
                                n_shared_experts=1, num_experts_per_tok=8, moe_intermediate_size=2048, n_group=8,
                                topk_group=4, routed_scaling_factor=2.5, norm_topk_prob=True, scoring_func="sigmoid",
                                first_k_dense_replace=3, q_lora_rank=1536, kv_lora_rank=512, qk_nope_head_dim=128,
                                qk_rope_head_dim=64, v_head_dim=128, moe_router_enable_expert_bias=True,
                                rope_interleave=True), is_mla=True)
DeepseekV2Config = _config("DeepseekV2Config", "deepseek_v2",
                           dict(vocab_size=102400, hidden_size=5120, intermediate_size=12288, num_hidden_layers=60,
                                num_attention_heads=128, num_key_value_heads=128, n_routed_experts=160,
                                n_shared_experts=2, num_experts_per_tok=6, moe_intermediate_size=1536, n_group=8,
                                topk_group=3, routed_scaling_factor=16.0, norm_topk_prob=False, scoring_func="softmax",
                                first_k_dense_replace=1, q_lora_rank=1536, kv_lora_rank=512, qk_nope_head_dim=128,
                                qk_rope_head_dim=64, v_head_dim=128, rope_interleave=True), is_mla=True)
Qwen2MoeConfig = _config("Qwen2MoeConfig", "qwen2_moe",
                         dict(vocab_size=151936, attention_bias=True, rope_theta=1e6, num_experts=60,
                              num_experts_per_tok=4, moe_intermediate_size=1408, shared_expert_intermediate_size=5632,
                              use_shared_expert_gating=True, norm_topk_prob=False, first_k_dense_replace=0,
                              moe_router_score_function="softmax"))
MixtralConfig = _config("MixtralConfig", "mixtral",
                        dict(num_experts=8, num_experts_per_tok=2, moe_intermediate_size=14336, norm_topk_prob=True,
                             first_k_dense_replace=0, num_key_value_heads=8, rope_theta=1e6))
TelechatConfig = _config("TelechatConfig", "telechat", dict(vocab_size=131072))


class ChatGLM2Config(PretrainedConfig):
    """ChatGLM2 / ChatGLM3 / GLM-4 configuration with the keys of the reference's class and of the published
    ``config.json`` files (``models/glm2/glm2_config.py:125-240``: ``padded_vocab_size``, ``num_layers``,
    ``ffn_hidden_size``, ``kv_channels``, ``multi_query_attention`` / ``multi_query_group_num``, ``rope_ratio``,
    ``rmsnorm``, ``add_qkv_bias`` …); defaults are GLM-4-9B.

    What makes the family differ from Llama is expressed in ``to_transformer_dict``: the rotary embedding covers the
    first half of every head and rotates adjacent pairs (``glm2_modules.py`` rotary: ``rope_cache`` over
    ``kv_channels // 2`` dims, pairs ``(2i, 2i+1)``), its base is ``10000 * rope_ratio``, Q/K/V carry a bias while the
    other projections do not, and there are ``multi_query_group_num`` KV heads."""

    model_type = "glm"

    @classmethod
    def default_values(cls):
        return dict(num_layers=40, padded_vocab_size=151552, hidden_size=4096, ffn_hidden_size=13696, kv_channels=128,
                    num_attention_heads=32, seq_length=8192, layernorm_epsilon=1.5625e-07, rope_ratio=1.0, rmsnorm=True,
                    post_layer_norm=True, add_bias_linear=False, add_qkv_bias=True, multi_query_attention=True,
                    multi_query_group_num=2, tie_word_embeddings=False, pad_token_id=151329, eos_token_id=151329,
                    max_position_embeddings=None)

    _PAIRS = (("num_layers", "num_hidden_layers"), ("padded_vocab_size", "vocab_size"),
              ("ffn_hidden_size", "intermediate_size"), ("kv_channels", "head_dim"),
              ("multi_query_group_num", "num_key_value_heads"), ("layernorm_epsilon", "rms_norm_eps"),
              ("add_qkv_bias", "attention_bias"), ("rope_ratio", "rope_theta"), ("rope_ratio", "rotary_base"))

    def __init__(self, **kwargs):
        self._explicit = set(kwargs)
        super().__init__(**kwargs)

    def to_transformer_dict(self) -> dict:
        d = self.to_dict()
        # a configuration written with Hugging Face keys (the GLM-4-0414 ``config.json`` spelling) wins over this
        # class's ChatGLM-keyed defaults
        for glm_key, hf_key in self._PAIRS:
            if d.get(hf_key) is not None and glm_key not in self._explicit:
                d.pop(glm_key, None)
        if "rope_ratio" not in d:
            d.pop("multi_query_attention", None)
            if "partial_rotary_factor" not in d:
                d.setdefault("rotary_percent", 0.5)
            d.setdefault("rotary_interleaved", True)
            d["normalization"] = "RMSNorm" if d.pop("rmsnorm", True) else "LayerNorm"
            return d
        if not d.pop("multi_query_attention", True):
            d["multi_query_group_num"] = d["num_attention_heads"]
        d["rotary_base"] = 10000.0 * float(d.pop("rope_ratio", 1.0) or 1.0)
        d.setdefault("rotary_percent", 0.5)
        d.setdefault("rotary_interleaved", True)
        d["normalization"] = "RMSNorm" if d.pop("rmsnorm", True) else "LayerNorm"
        if d.get("max_position_embeddings") is None:
            d["max_position_embeddings"] = d.get("seq_length")
        if "vocab_size" in d and "padded_vocab_size" in d:
            d.pop("vocab_size")
        return d


MindFormerRegister.register_cls(ChatGLM2Config, MindFormerModuleType.CONFIG, alias="ChatGLM2Config")
MindFormerRegister.register_cls(ChatGLM2Config, MindFormerModuleType.CONFIG, alias="ChatGLM2Config", legacy=False)
ChatGLM4Config = ChatGLM2Config



class MefesunConfig(PretrainedConfig):
    """Mefesun: a decoder described layer by layer, with norms on the sub-layer outputs only, layer scale, chunked
    grouped-query attention with a softmax sink, q / k norm, YaRN rotary positions, squared-relu feed-forwards, optional
    weight sharing between layers, a tied head and soft-capped logits.

    Keys of ``config.json``: ``vocab``, ``width``, ``norm.eps``, ``logit_softcap`` and ``layers``, a list of ``{"type":
    "attention", "mixer": {"heads", "kv_heads", "dim", "vdim", "scale", "mask": {"size"}, "rot": {"base", "dims",
    "scaling": {"factor", "original", "fast", "slow"}}}, "mlp": {"kind": "dense", "ff"} | null, "weights_of"}``. Framework
    keys (``seq_length``, ``block_size``, token ids) may stand beside them. ``to_transformer_dict`` translates."""

    model_type = "mefesun"

    @classmethod
    def default_values(cls):
        return dict(architecture="Mefesun", vocab=32000, width=1024, norm=dict(eps=1e-6), logit_softcap=30.0,
                    layers=MefesunConfig.uniform_layers(12, heads=8, kv_heads=2, dim=128, ff=4096, chunk=2048),
                    pad_token_id=0, bos_token_id=None, eos_token_id=None, block_size=64)

    @staticmethod
    def uniform_layers(n: int, heads: int, kv_heads: int, dim: int, ff: int, chunk: int, vdim=None, rot_dims=None,
                       base: float = 500000.0, factor: float = 8.0, original: int = 8192, fast: float = 32.0,
                       slow: float = 1.0, scale=None):
        """The ``layers`` list of a model whose ``n`` layers are alike."""
        mixer = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim or dim, scale=scale or dim ** -0.5,
                     mask=dict(size=chunk), rot=dict(base=base, dims=rot_dims or dim,
                                                     scaling=dict(factor=factor, original=original, fast=fast, slow=slow)))
        return [dict(type="attention", mixer=copy.deepcopy(mixer), mlp=dict(kind="dense", ff=ff)) for _ in range(n)]

    @staticmethod
    def _layer_fields(i: int, layer: dict) -> dict:
        if layer.get("type") != "attention":
            raise ValueError(f"layer {i}: unknown mixer type {layer.get('type')!r}")
        mix, mlp = layer["mixer"], layer.get("mlp")
        if mlp and mlp.get("kind", "dense") != "dense":
            raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
        rot = mix["rot"]
        scaling = rot.get("scaling")
        return dict(
            num_attention_heads=int(mix["heads"]), num_query_groups=int(mix["kv_heads"]), kv_channels=int(mix["dim"]),
            v_channels=int(mix["vdim"]), softmax_scale=float(mix["scale"]),
            attention_chunk_size=int((mix.get("mask") or {}).get("size") or 0),
            rotary_dim=int(rot["dims"]), rotary_base=float(rot["base"]),
            rope_scaling=None if not scaling else dict(
                type="yarn", factor=float(scaling["factor"]), original_max_position_embeddings=float(scaling["original"]),
                beta_fast=float(scaling["fast"]), beta_slow=float(scaling["slow"])),
            ffn_hidden_size=int(mlp["ff"]) if mlp else 0)

    def _owner(self, i: int) -> int:
        """The layer whose weights layer ``i`` runs with."""
        for _ in self.layers:
            j = self.layers[i].get("weights_of")
            if j is None:
                return i
            i = int(j)
        raise ValueError("weights_of: layers name one another in a circle")

    def to_transformer_dict(self) -> dict:
        d = {k: v for k, v in self.to_dict().items()
             if k not in ("architecture", "layers", "norm", "vocab", "width", "mlp", "mixer")}
        fields = [self._layer_fields(i, layer) for i, layer in enumerate(self.layers)]
        owners = [self._owner(i) for i in range(len(fields))]
        d.setdefault("seq_length", max(int(f["rope_scaling"]["factor"] * f["rope_scaling"]["original_max_position_embeddings"])
                                       if f["rope_scaling"] else 4096 for f in fields))
        d.setdefault("max_position_embeddings", d["seq_length"])
        own = {k: v for k, v in fields[0].items() if k != "rope_scaling"}
        own.update(vocab_size=int(self.vocab), hidden_size=int(self.width), num_layers=len(fields), layer_overrides=fields,
                 layer_sharing=owners, layernorm_epsilon=float(self.norm["eps"]), normalization="LayerNorm",
                 norm_placement="output", layer_scale=True, fp32_residual_connection=True, ragged_attention=True,
                 qk_layernorm=True, add_qkv_bias=True, add_attention_output_bias=True, attention_sink=True,
                 rotary_interleaved=True, gated_linear_unit=False, hidden_act="relu2", position_embedding_type="none",
                 tie_word_embeddings=True, logit_softcap=float(self.logit_softcap) if self.logit_softcap else None)
        # other spellings of what the design's own keys describe do not apply
        d = {k: v for k, v in d.items() if ALIASES.get(k, (k,))[0] not in own}
        return dict(d, **own)


class KukupelConfig(PretrainedConfig):
    """Kukupel: a decoder on several residual streams (hyper-connections) whose layers mix tokens with a gated delta rule,
    alone (``delta``: one decay per head, silu gate) or beside position-free, soft-capped grouped-query attention
    (``parallel``: decays per key channel and a sigmoid gate, both low-rank), pre-norm, with mixtures of clamped gated experts
    whose routing weight multiplies their input, and a tied head.

    Keys of ``config.json``: ``vocab``, ``width``, ``streams``, ``norm.eps`` and ``layers``, a list of ``{"type": "delta",
    "mixer": {"heads", "kv_heads", "dim", "vdim", "conv"}}`` or ``{"type": "parallel", "mixer": {"left": {"heads",
    "kv_heads", "dim", "vdim", "scale", "softcap"}, "right": {as delta}, "left_scale", "right_scale"}}``, each with ``"mlp":
    {"kind": "moe", "router": {"experts", "top"}, "expert": {"ff", "limit"}} | null``. The ranks of the low-rank factors are
    those of the checkpoint's tensors (``complete_from_checkpoint``), or ``right.decay_rank`` / ``right.gate_rank``, or the
    value size. Framework keys (``seq_length``, ``block_size``, token ids) may stand beside them."""

    model_type = "kukupel"

    @classmethod
    def default_values(cls):
        return dict(architecture="Kukupel", vocab=32000, width=1024, streams=4, norm=dict(eps=1e-6),
                    layers=KukupelConfig.layer_list("parallel delta delta delta", heads=8, kv_heads=2, dim=128, delta_heads=8,
                                                    delta_kv_heads=4, delta_dim=128, experts=16, top=2, ff=768),
                    pad_token_id=0, bos_token_id=None, eos_token_id=None, block_size=64)

    @staticmethod
    def layer_list(types: str, heads: int, kv_heads: int, dim: int, delta_heads: int, delta_kv_heads: int, delta_dim: int,
                   experts: int, top: int, ff: int, vdim=None, delta_vdim=None, conv: int = 4, softcap: float = 30.0,
                   scale=None, scales=(0.5, 0.5), limit: float = 7.0, rank=None):
        """The ``layers`` list of a model whose layers of one type (``types``, by name) are alike."""
        delta = dict(heads=delta_heads, kv_heads=delta_kv_heads, dim=delta_dim, vdim=delta_vdim or delta_dim, conv=conv)
        left = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim or dim, scale=scale or dim ** -0.5, softcap=softcap)
        right = dict(delta, **({} if rank is None else dict(decay_rank=rank, gate_rank=rank)))
        mixer = {"delta": delta, "parallel": dict(left=left, right=right, left_scale=scales[0], right_scale=scales[1])}
        mlp = dict(kind="moe", router=dict(experts=experts, top=top), expert=dict(ff=ff, limit=limit))
        return [dict(type=t, mixer=copy.deepcopy(mixer[t]), mlp=copy.deepcopy(mlp)) for t in types.split()]

    def complete_from_checkpoint(self, shape_of):
        """Sizes that only the checkpoint gives; ``shape_of(name)`` is a tensor's shape, None for one it does not hold."""
        for i, layer in enumerate(self.layers):
            if layer.get("type") == "parallel":
                for key, name in (("decay_rank", "a1"), ("gate_rank", "g1")):
                    shape = shape_of(f"l{i}.mix.right.{name}")
                    if shape is not None:
                        layer["mixer"]["right"][key] = int(shape[0])

    @staticmethod
    def _delta_fields(mix: dict, channel: bool) -> dict:
        rank = int(mix["vdim"])
        return dict(delta_heads=int(mix["heads"]), delta_kv_heads=int(mix["kv_heads"]), delta_key_dim=int(mix["dim"]),
                    delta_value_dim=int(mix["vdim"]), delta_conv_taps=int(mix["conv"]),
                    delta_decay="channel" if channel else "head", delta_gate="sigmoid" if channel else "silu",
                    delta_decay_rank=int(mix.get("decay_rank") or rank) if channel else 0,
                    delta_gate_rank=int(mix.get("gate_rank") or rank) if channel else 0)

    @classmethod
    def _layer_fields(cls, i: int, layer: dict) -> dict:
        kind, mix, mlp = layer.get("type"), layer["mixer"], layer.get("mlp")
        if kind == "delta":
            out = dict(mixer="delta", **cls._delta_fields(mix, False))
        elif kind == "parallel":
            a = mix["left"]
            out = dict(mixer="parallel", parallel_scales=(float(mix["left_scale"]), float(mix["right_scale"])),
                       num_attention_heads=int(a["heads"]), num_query_groups=int(a["kv_heads"]), kv_channels=int(a["dim"]),
                       v_channels=int(a["vdim"]), softmax_scale=float(a["scale"]),
                       attention_softcap=float(a["softcap"]) if a.get("softcap") else None,
                       **cls._delta_fields(mix["right"], True))
        else:
            raise ValueError(f"layer {i}: unknown mixer type {kind!r}")
        if mlp and mlp.get("kind", "moe") != "moe":
            raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
        out.update(ffn_hidden_size=0)
        if mlp:
            r, e = mlp["router"], mlp["expert"]
            if not 1 <= int(r["top"]) <= int(r["experts"]):
                raise ValueError(f"layer {i}: {r['top']} of {r['experts']} experts")
            out.update(num_moe_experts=int(r["experts"]), moe_router_topk=int(r["top"]), moe_ffn_hidden_size=int(e["ff"]),
                       moe_activation_limit=float(e["limit"]))
        return out

    def to_transformer_dict(self) -> dict:
        d = {k: v for k, v in self.to_dict().items()
             if k not in ("architecture", "layers", "norm", "vocab", "width", "streams", "mlp", "mixer")}
        fields = [self._layer_fields(i, layer) for i, layer in enumerate(self.layers)]
        d.setdefault("seq_length", 32768)                      # no positions enter the model: a bound for buffers alone
        d.setdefault("max_position_embeddings", d["seq_length"])
        moe = [1 if f.get("num_moe_experts") else 0 for f in fields]
        own = dict(num_attention_heads=1, num_query_groups=1, kv_channels=1, ffn_hidden_size=0)       # layers without attention
        for f in fields:                                       # the stack's own view of what its layers override
            own.update({k: v for k, v in f.items() if k in own and k != "ffn_hidden_size"})
        if any(moe):
            own.update({k: v for k, v in fields[moe.index(1)].items() if k.startswith(("num_moe", "moe_"))}, moe_layer_freq=moe)
        own.update(vocab_size=int(self.vocab), hidden_size=int(self.width), num_layers=len(fields), layer_overrides=fields,
                   residual_streams=int(self.streams), layernorm_epsilon=float(self.norm["eps"]), normalization="RMSNorm",
                   fp32_residual_connection=True, ragged_attention=True, rotary_dim=0, position_embedding_type="none",
                   moe_activation="clamped_glu", moe_activation_alpha=1.702, moe_apply_probs_on_input=True, norm_topk_prob=False,
                   moe_router_score_function="sigmoid", moe_router_topk_scaling_factor=1.0, tie_word_embeddings=True)
        d = {k: v for k, v in d.items() if ALIASES.get(k, (k,))[0] not in own}
        return dict(d, **own)


class GavatarConfig(PretrainedConfig):
    """Gavatar: a decoder on one fp32 stream with norms (weights around zero) on both sides of every sub-layer, a token shift in
    front of every mixer, scaled embeddings plus sinusoidal position vectors, and a block of layers that runs several times. Its
    mixers are sliding-window grouped-query attention with unit-norm queries, keys and values whose softmax weights are mixed over
    heads (``attention``), sliding-window latent attention with a softmax sink (``latent_attention``), both position-free and
    gated, and a matrix memory (``mlstm``); its feed-forwards are mixtures of SwiGLU experts with biased router logits.

    Keys of ``config.json``: ``vocab``, ``width``, ``norm.eps``, ``embedding.scale``, ``loop`` (``{"start", "stop", "times"}`` or
    null) and ``layers``, a list of ``{"type": "attention", "mixer": {"heads", "kv_heads", "dim", "vdim", "scale", "mask":
    {"size"}}}``, ``{"type": "latent_attention", "mixer": {"heads", "dim", "vdim", "q_rank", "kv_rank", "scale", "mask":
    {"size"}}}`` or ``{"type": "mlstm", "mixer": {"heads", "dim", "vdim", "gate_cap"}}``, each with ``"mlp": {"kind": "moe",
    "router": {"experts", "top"}, "expert": {"ff"}} | null``. Framework keys (``seq_length``, ``block_size``, token ids) may
    stand beside them."""

    model_type = "gavatar"

    @classmethod
    def default_values(cls):
        return dict(architecture="Gavatar", vocab=32000, width=1024, norm=dict(eps=1e-6), embedding=dict(scale=1.0), loop=None,
                    layers=GavatarConfig.layer_list("latent_attention mlstm attention", heads=8, kv_heads=2, dim=128, rank=256,
                                                    window=1024, memory_heads=4, memory_dim=128, experts=16, top=2, ff=768),
                    pad_token_id=0, bos_token_id=None, eos_token_id=None, block_size=64)

    @staticmethod
    def layer_list(types: str, heads: int, kv_heads: int, dim: int, rank: int, window: int, memory_heads: int, memory_dim: int,
                   experts: int, top: int, ff: int, vdim=None, q_rank=None, memory_vdim=None, scale=None, gate_cap: float = 15.0):
        """The ``layers`` list of a model whose layers of one type (``types``, by name) are alike."""
        common = dict(heads=heads, dim=dim, vdim=vdim or dim, scale=scale or dim ** -0.5, mask=dict(size=window))
        mixer = {"attention": dict(common, kv_heads=kv_heads),
                 "latent_attention": dict(common, q_rank=q_rank or rank, kv_rank=rank),
                 "mlstm": dict(heads=memory_heads, dim=memory_dim, vdim=memory_vdim or memory_dim, gate_cap=gate_cap)}
        mlp = dict(kind="moe", router=dict(experts=experts, top=top), expert=dict(ff=ff))
        return [dict(type=t, mixer=copy.deepcopy(mixer[t]), mlp=copy.deepcopy(mlp)) for t in types.split()]

    @staticmethod
    def _layer_fields(i: int, layer: dict) -> dict:
        kind, mix, mlp = layer.get("type"), layer["mixer"], layer.get("mlp")
        if kind in ("attention", "latent_attention"):
            out = dict(num_attention_heads=int(mix["heads"]), kv_channels=int(mix["dim"]), v_channels=int(mix["vdim"]),
                       softmax_scale=float(mix["scale"]), attention_window=int((mix.get("mask") or {}).get("size") or 0))
            if kind == "attention":
                out.update(mixer="attention", num_query_groups=int(mix["kv_heads"]), add_qkv_bias=True, qk_unit_norm=True,
                           value_unit_norm=True, attention_talk=True, attention_output_gate="channel")
            else:
                out.update(mixer="latent", num_query_groups=int(mix["heads"]), q_lora_rank=int(mix["q_rank"]),
                           kv_lora_rank=int(mix["kv_rank"]), attention_sink=True, attention_output_gate="head")
        elif kind == "mlstm":
            out = dict(mixer="matrix_memory", memory_heads=int(mix["heads"]), memory_key_dim=int(mix["dim"]),
                       memory_value_dim=int(mix["vdim"]), memory_gate_cap=float(mix["gate_cap"]))
        else:
            raise ValueError(f"layer {i}: unknown mixer type {kind!r}")
        if mlp and mlp.get("kind", "moe") != "moe":
            raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
        out.update(ffn_hidden_size=0)
        if mlp:
            r, e = mlp["router"], mlp["expert"]
            if not 1 <= int(r["top"]) <= int(r["experts"]):
                raise ValueError(f"layer {i}: {r['top']} of {r['experts']} experts")
            out.update(num_moe_experts=int(r["experts"]), moe_router_topk=int(r["top"]), moe_ffn_hidden_size=int(e["ff"]))
        return out

    def to_transformer_dict(self) -> dict:
        d = {k: v for k, v in self.to_dict().items()
             if k not in ("architecture", "layers", "norm", "vocab", "width", "embedding", "loop", "mlp", "mixer")}
        fields = [self._layer_fields(i, layer) for i, layer in enumerate(self.layers)]
        d.setdefault("seq_length", 32768)                      # position vectors have no longest position: a bound for buffers
        d.setdefault("max_position_embeddings", d["seq_length"])
        moe = [1 if f.get("num_moe_experts") else 0 for f in fields]
        own = dict(num_attention_heads=1, num_query_groups=1, kv_channels=1, ffn_hidden_size=0)       # layers without attention
        for f in fields:                                       # the stack's own view of what its layers override
            own.update({k: v for k, v in f.items() if k in own and k != "ffn_hidden_size"})
        if any(moe):
            own.update({k: v for k, v in fields[moe.index(1)].items() if k.startswith(("num_moe", "moe_"))}, moe_layer_freq=moe)
        loop = self.loop
        own.update(vocab_size=int(self.vocab), hidden_size=int(self.width), num_layers=len(fields), layer_overrides=fields,
                   layer_loop=(int(loop["start"]), int(loop["stop"]), int(loop["times"])) if loop else None,
                   layernorm_epsilon=float(self.norm["eps"]), normalization="RMSNorm", layernorm_zero_centered_gamma=True,
                   norm_placement="both", token_shift=True, fp32_residual_connection=True, ragged_attention=True, rotary_dim=0,
                   position_embedding_type="sinusoidal", embedding_scale=float(self.embedding["scale"]),
                   moe_router_score_function="softmax", norm_topk_prob=True, moe_router_logit_bias=True, moe_router_dtype="params",
                   moe_router_topk_scaling_factor=1.0, tie_word_embeddings=False)
        d = {k: v for k, v in d.items() if ALIASES.get(k, (k,))[0] not in own}
        return dict(d, **own)


class TogalornConfig(PretrainedConfig):
    """Togalorn: a decoder on one fp32 stream whose layers read one norm, in parts of the width, and run their mixer and their
    feed-forward side by side, the mixer behind a causal convolution of its input. A block of layers may run several times, each pass
    starting from a product of the stream and the embedding output. Its mixers are latent attention with a rotated key part for all
    heads and a gate per channel (``latent_attention``) and a state space with a scalar decay per head (``mamba2``); its
    feed-forwards are mixtures of clamped gated experts with identity experts and a shared one; the head is untied.

    Keys of ``config.json``: ``vocab``, ``width``, ``norm`` (``{"eps", "groups"}``), ``canon.taps``, ``embedding.scale``, ``loop``
    (``{"start", "stop", "times"}`` or null) and ``layers``, a list of ``{"type": "latent_attention", "mixer": {"heads", "dim",
    "rot_dim", "vdim", "q_rank", "kv_rank", "scale", "rot": {"base", "dims"}}}`` or ``{"type": "mamba2", "mixer": {"heads",
    "vdim", "state", "groups", "conv", "norm_groups"}}``, each with ``"mlp": {"kind": "moe", "router": {"experts", "identity",
    "top"}, "expert": {"ff", "limit"}, "shared": {"ff", "limit"}} | null``. Framework keys (``seq_length``, ``block_size``, token
    ids) may stand beside them."""

    model_type = "togalorn"

    @classmethod
    def default_values(cls):
        return dict(architecture="Togalorn", vocab=32000, width=1024, norm=dict(eps=1e-6, groups=1), canon=dict(taps=4),
                    embedding=dict(scale=1.0), loop=None,
                    layers=TogalornConfig.layer_list("mamba2 mamba2 latent_attention", heads=8, dim=96, rot_dim=32, vdim=128, rank=256,
                                                     ssm_heads=32, ssm_dim=64, state=128, experts=16, top=2, ff=768),
                    pad_token_id=0, bos_token_id=None, eos_token_id=None, block_size=64)

    @staticmethod
    def layer_list(types: str, heads: int, dim: int, rot_dim: int, vdim: int, rank: int, ssm_heads: int, ssm_dim: int, state: int,
                   experts: int, top: int, ff: int, q_rank=None, base: float = 500000.0, scale=None, ssm_groups: int = 1, conv: int = 4,
                   norm_groups: int = 1, identity: int = 0, limit: float = 7.0, shared_ff=None, shared_limit=None):
        """The ``layers`` list of a model whose layers of one type (``types``, by name) are alike."""
        mixer = {"latent_attention": dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, q_rank=q_rank or rank, kv_rank=rank,
                                          scale=scale or (dim + rot_dim) ** -0.5, rot=dict(base=base, dims=rot_dim)),
                 "mamba2": dict(heads=ssm_heads, vdim=ssm_dim, state=state, groups=ssm_groups, conv=conv, norm_groups=norm_groups)}
        mlp = dict(kind="moe", router=dict(experts=experts, identity=identity, top=top), expert=dict(ff=ff, limit=limit),
                   shared=dict(ff=shared_ff or ff, limit=shared_limit or limit))
        return [dict(type=t, mixer=copy.deepcopy(mixer[t]), mlp=copy.deepcopy(mlp)) for t in types.split()]

    @staticmethod
    def _layer_fields(i: int, layer: dict) -> dict:
        kind, mix, mlp = layer.get("type"), layer["mixer"], layer.get("mlp")
        if kind == "latent_attention":
            rot = int(mix["rot_dim"])
            if int(mix["rot"]["dims"]) != rot:
                raise ValueError(f"layer {i}: {mix['rot']['dims']} rotated dimensions of a rotated part of {rot}")
            out = dict(mixer="latent", num_attention_heads=int(mix["heads"]), num_query_groups=int(mix["heads"]),
                       kv_channels=int(mix["dim"]), v_channels=int(mix["vdim"]), softmax_scale=float(mix["scale"]),
                       q_lora_rank=int(mix["q_rank"]), kv_lora_rank=int(mix["kv_rank"]), rotary_dim=rot,
                       rotary_base=float(mix["rot"]["base"]), attention_output_gate="channel")
        elif kind == "mamba2":
            out = dict(mixer="state_space", ssm_heads=int(mix["heads"]), ssm_head_dim=int(mix["vdim"]), ssm_state=int(mix["state"]),
                       ssm_groups=int(mix["groups"]), ssm_conv_taps=int(mix["conv"]), ssm_norm_groups=int(mix["norm_groups"]))
        else:
            raise ValueError(f"layer {i}: unknown mixer type {kind!r}")
        if mlp and mlp.get("kind", "moe") != "moe":
            raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
        out.update(ffn_hidden_size=0)
        if mlp:
            r, e, s = mlp["router"], mlp["expert"], mlp["shared"]
            identity = int(r.get("identity") or 0)
            if not 1 <= int(r["top"]) <= int(r["experts"]) + identity:
                raise ValueError(f"layer {i}: {r['top']} of {r['experts']} + {identity} experts")
            out.update(num_moe_experts=int(r["experts"]), moe_identity_experts=identity, moe_router_topk=int(r["top"]),
                       moe_ffn_hidden_size=int(e["ff"]), moe_activation_limit=float(e["limit"]),
                       moe_shared_expert_intermediate_size=int(s["ff"]), moe_shared_expert_activation_limit=float(s["limit"]))
        return out

    def to_transformer_dict(self) -> dict:
        d = {k: v for k, v in self.to_dict().items()
             if k not in ("architecture", "layers", "norm", "vocab", "width", "embedding", "canon", "loop", "mlp", "mixer")}
        fields = [self._layer_fields(i, layer) for i, layer in enumerate(self.layers)]
        d.setdefault("seq_length", 32768)                      # angles are evaluated: a bound for buffers alone
        d.setdefault("max_position_embeddings", d["seq_length"])
        moe = [1 if f.get("num_moe_experts") else 0 for f in fields]
        own = dict(num_attention_heads=1, num_query_groups=1, kv_channels=1, ffn_hidden_size=0)       # layers without attention
        for f in fields:                                       # the stack's own view of what its layers override
            own.update({k: v for k, v in f.items() if k in own and k != "ffn_hidden_size"})
        if any(moe):
            own.update({k: v for k, v in fields[moe.index(1)].items() if k.startswith(("num_moe", "moe_"))}, moe_layer_freq=moe)
        loop = self.loop
        own.update(vocab_size=int(self.vocab), hidden_size=int(self.width), num_layers=len(fields), layer_overrides=fields,
                   layer_loop=(int(loop["start"]), int(loop["stop"]), int(loop["times"])) if loop else None, loop_input=bool(loop),
                   layernorm_epsilon=float(self.norm["eps"]), norm_groups=int(self.norm["groups"]), normalization="RMSNorm",
                   norm_placement="parallel", input_conv_taps=int(self.canon["taps"]), fp32_residual_connection=True,
                   ragged_attention=True, rotary_interleaved=True, position_embedding_type="none",
                   embedding_scale=float(self.embedding["scale"]), moe_activation="clamped_glu", moe_activation_alpha=1.702,
                   moe_router_score_function="softmax", norm_topk_prob=True, moe_router_enable_expert_bias=True,
                   moe_router_dtype="params", moe_router_topk_scaling_factor=1.0, tie_word_embeddings=False)
        d = {k: v for k, v in d.items() if ALIASES.get(k, (k,))[0] not in own}
        return dict(d, **own)


for _legacy in (True, False):
    MindFormerRegister.register_cls(TogalornConfig, MindFormerModuleType.CONFIG, alias="TogalornConfig", legacy=_legacy)
    MindFormerRegister.register_cls(GavatarConfig, MindFormerModuleType.CONFIG, alias="GavatarConfig", legacy=_legacy)
    MindFormerRegister.register_cls(KukupelConfig, MindFormerModuleType.CONFIG, alias="KukupelConfig", legacy=_legacy)
    MindFormerRegister.register_cls(MefesunConfig, MindFormerModuleType.CONFIG, alias="MefesunConfig", legacy=_legacy)

LlamaForCausalLM = _model("LlamaForCausalLM", LlamaConfig, "llama")
Qwen2ForCausalLM = _model("Qwen2ForCausalLM", Qwen2Config, "qwen2")
Qwen3ForCausalLM = _model("Qwen3ForCausalLM", Qwen3Config, "qwen3")
Qwen3MoeForCausalLM = _model("Qwen3MoeForCausalLM", Qwen3MoeConfig, "qwen3_moe")
DeepseekV3ForCausalLM = _model("DeepseekV3ForCausalLM", DeepseekV3Config, "deepseek_v3")
DeepseekV2ForCausalLM = _model("DeepseekV2ForCausalLM", DeepseekV2Config, "deepseek_v2")
Qwen2MoeForCausalLM = _model("Qwen2MoeForCausalLM", Qwen2MoeConfig, "qwen2_moe")
MixtralForCausalLM = _model("MixtralForCausalLM", MixtralConfig, "mixtral")
TelechatForCausalLM = _model("TelechatForCausalLM", TelechatConfig, "telechat")
MefesunForCausalLM = _model("MefesunForCausalLM", MefesunConfig, "mefesun")
MefesunForCausalLM.kernel_sources = ("host_util", "elementwise", "gemm_tcgen05", "gemm_tcgen05_2cta", "gemm_bf16_decode",
                                     "output_norm", "qkv_rope_cache", "paged_prefill_tc", "paged_decode_tc",
                                     "paged_attention", "paged_attention_any", "decode_loop")
KukupelForCausalLM = _model("KukupelForCausalLM", KukupelConfig, "kukupel")
KukupelForCausalLM.kernel_sources = ("host_util", "elementwise", "gemm_tcgen05", "gemm_tcgen05_2cta", "gemm_bf16_decode",
                                     "residual_streams", "delta_rule", "qkv_rope_cache", "paged_prefill_tc", "paged_decode_tc",
                                     "paged_attention", "paged_attention_any", "router", "moe_ep", "moe_any", "decode_loop")
GavatarForCausalLM = _model("GavatarForCausalLM", GavatarConfig, "gavatar")
GavatarForCausalLM.kernel_sources = ("host_util", "elementwise", "gemm_tcgen05", "gemm_tcgen05_2cta", "gemm_bf16_decode",
                                     "sandwich_norm", "head_mix", "matrix_memory", "qkv_rope_cache", "paged_prefill_tc",
                                     "paged_decode_tc", "paged_attention", "paged_attention_any", "paged_talk_decode",
                                     "latent_decode", "router", "moe_ep",
                                     "moe_any", "decode_loop")
TogalornForCausalLM = _model("TogalornForCausalLM", TogalornConfig, "togalorn")
TogalornForCausalLM.kernel_sources = ("host_util", "elementwise", "gemm_tcgen05", "gemm_tcgen05_2cta", "gemm_bf16_decode",
                                      "sandwich_norm", "joint_norm", "head_mix", "state_space", "paged_prefill_tc",
                                      "paged_attention", "paged_attention_any", "paged_decode_tc", "latent_decode", "router", "moe_ep",
                                      "moe_any", "decode_loop")
ChatGLM2ForConditionalGeneration = _model("ChatGLM2ForConditionalGeneration", ChatGLM4Config, "glm")

def _backbone(name, causal_cls):
    class _B(causal_cls):
        def forward(self, input_ids, position_ids=None, attn_meta=None, **kw):
            return self.model(input_ids, None, None, position_ids, attn_meta, return_hidden=True,
                              input_embeds=kw.get("input_embeds"))

    _B.__name__ = _B.__qualname__ = name
    _B.__doc__ = (f"The ``{causal_cls.__name__}`` network without its language-model head: ``forward(input_ids)`` returns the "
                  f"final-norm hidden states ``[B * S, hidden]`` (reference ``models/llama/llama.py`` ``LlamaModel``, "
                  f"``models/glm2/glm2.py`` ``ChatGLM2Model``). The head's weights are still built so that a causal-LM "
                  f"checkpoint loads without missing keys.")
    return _B


LlamaModel = _backbone("LlamaModel", LlamaForCausalLM)
ChatGLM2Model = _backbone("ChatGLM2Model", ChatGLM2ForConditionalGeneration)


class ChatGLM2WithPtuning2(ChatGLM2ForConditionalGeneration):
    """ChatGLM2 with P-Tuning v2 (reference ``models/glm2/glm2.py`` ``ChatGLM2WithPtuning2``): the base weights are frozen
    and a per-layer key / value prefix of ``config.pet_config.pre_seq_len`` virtual tokens is trained."""

    def __init__(self, config, **kwargs):
        super().__init__(config, **kwargs)
        from ..pet.pet_config import Ptuning2Config
        from ..pet.prompt import PrefixTuningModel
        pet = getattr(config, "pet_config", None) or {}
        if not isinstance(pet, Ptuning2Config):
            pet = dict(pet)
            pet.pop("pet_type", None)
            pet = Ptuning2Config(**pet)
        tuned = PrefixTuningModel(pet, self)
        object.__setattr__(self, "_tuned", tuned)           # not a sub-module: it holds this module already
        self.prefix_encoder = tuned.prefix_encoder

    def forward(self, *args, **kwargs):
        self._tuned.current = self.prefix_encoder()
        return super().forward(*args, **kwargs)


# Names that configurations written for the reference use for the same models: its mcore shims pick a
# ``Training...`` or ``Inference...`` class by run mode (``qwen3/modeling_qwen3.py:27-54``,
# ``deepseek3/modeling_deepseek_v3.py:25-42``) and its research directories ship explicit tensor-parallel inference
# models (``research/llama3_1/llama.py:48`` ``ParallelLlamaForCausalLM``, ``research/qwen2_5`` ``ParallelQwenForCausalLM``,
# ``research/deepseek3`` ``DeepseekV3ForCausalLM`` / ``InferenceDeepseekV3ForCausalLM``). One class serves training and
# inference here, so these are aliases.
_ALIASES = {
    "ParallelLlamaForCausalLM": LlamaForCausalLM, "ParallelQwenForCausalLM": Qwen2ForCausalLM,
    "TrainingQwen3ForCausalLM": Qwen3ForCausalLM, "InferenceQwen3ForCausalLM": Qwen3ForCausalLM,
    "TrainingQwen3MoeForCausalLM": Qwen3MoeForCausalLM, "InferenceQwen3MoeForCausalLM": Qwen3MoeForCausalLM,
    "TrainingDeepseekV3ForCausalLM": DeepseekV3ForCausalLM, "InferenceDeepseekV3ForCausalLM": DeepseekV3ForCausalLM,
    "InferenceQwen2ForCausalLM": Qwen2ForCausalLM, "DeepseekV2ForCausalLM_legacy": DeepseekV2ForCausalLM,
    "TelechatForCausalLM_MoE": TelechatForCausalLM,
}
globals().update(_ALIASES)
for _alias, _cls in _ALIASES.items():
    for _legacy in (True, False):
        MindFormerRegister.register_cls(_cls, MindFormerModuleType.MODELS, alias=_alias, legacy=_legacy)

MODEL_TYPE_TO_CLASSES = {
    "llama": (LlamaConfig, LlamaForCausalLM), "qwen2": (Qwen2Config, Qwen2ForCausalLM),
    "qwen2_5": (Qwen2Config, Qwen2ForCausalLM), "qwen3": (Qwen3Config, Qwen3ForCausalLM),
    "qwen3_moe": (Qwen3MoeConfig, Qwen3MoeForCausalLM), "deepseek_v3": (DeepseekV3Config, DeepseekV3ForCausalLM),
    "deepseekv3": (DeepseekV3Config, DeepseekV3ForCausalLM), "mixtral": (MixtralConfig, MixtralForCausalLM),
    "deepseek_v2": (DeepseekV2Config, DeepseekV2ForCausalLM), "deepseek2": (DeepseekV2Config, DeepseekV2ForCausalLM),
    "qwen2_moe": (Qwen2MoeConfig, Qwen2MoeForCausalLM),
    "telechat": (TelechatConfig, TelechatForCausalLM), "glm": (ChatGLM4Config, ChatGLM2ForConditionalGeneration),
    "mefesun": (MefesunConfig, MefesunForCausalLM), "kukupel": (KukupelConfig, KukupelForCausalLM),
    "gavatar": (GavatarConfig, GavatarForCausalLM), "togalorn": (TogalornConfig, TogalornForCausalLM),
    "chatglm": (ChatGLM4Config, ChatGLM2ForConditionalGeneration),
}
