"""Prefill and decode throughput of Kukupel beside Qwen3-MoE at equal size, and the roofline fraction of every kernel of the
two (random-init weights, synthetic tokens, one GPU). ``bench.py --config kukupel_serving`` runs it.

Equal size: same width, attention heads, head size, experts, experts per token, expert width, layers and vocabulary; every
second Kukupel layer is a ``parallel`` one (attention beside a gated delta rule), the others have the delta rule alone. Model
figures are device-timed (CUDA events): prefill is one call over whole prompts, decode the captured step of the device-side
loop. L2 is flushed before every timed kernel; the working set of the model runs exceeds it. Roofline denominators are the
measured peaks of ``MEASURED_PEAKS.json``; the recurrence, which runs in fp32 on the FMA pipes, is put against their nominal
rate (148 SMs x 128 lanes at 1965 MHz).
"""
from __future__ import annotations

import json
import os
import sys

import torch

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
if ROOT not in sys.path:
    sys.path.insert(0, ROOT)

from benchmarks.bench_ragged_serving import LAYERS, VOCAB, Table, decode_rate, prefill_rate, step_meta  # noqa: E402

SIZES = {
    "w4096_h32_kv8_d128_e32_top4": dict(width=4096, heads=32, kv=8, dim=128, delta=32, delta_kv=16, experts=32, top=4, ff=1536),
    "w2048_h16_kv4_d128_e64_top8": dict(width=2048, heads=16, kv=4, dim=128, delta=16, delta_kv=8, experts=64, top=8, ff=768),
    "w2048_h32_kv8_d64_e64_top8": dict(width=2048, heads=32, kv=8, dim=64, delta=32, delta_kv=16, experts=64, top=8, ff=768),
}
STREAMS, RANK, TAPS, SOFTCAP = 4, 128, 4, 30.0
FMA_PEAK = 148 * 128 * 2 * 1.965e9


def kukupel(size, max_len):
    from mindformers_b200.models import AutoModel, KukupelConfig
    layers = KukupelConfig.layer_list(" ".join(["parallel delta"] * (LAYERS // 2)), size["heads"], size["kv"], size["dim"],
                                      size["delta"], size["delta_kv"], size["dim"], size["experts"], size["top"], size["ff"],
                                      conv=TAPS, softcap=SOFTCAP, rank=RANK)
    cfg = KukupelConfig(vocab=VOCAB, width=size["width"], streams=STREAMS, norm=dict(eps=1e-6), layers=layers, seq_length=max_len)
    return AutoModel.from_config(cfg, device="cuda").eval()


def qwen3_moe(size, max_len):
    from mindformers_b200.models import AutoModel
    cfg = dict(model_type="qwen3_moe", num_hidden_layers=LAYERS, hidden_size=size["width"], num_attention_heads=size["heads"],
               num_key_value_heads=size["kv"], head_dim=size["dim"], intermediate_size=size["ff"] * size["top"],
               moe_intermediate_size=size["ff"], num_experts=size["experts"], num_experts_per_tok=size["top"], vocab_size=VOCAB,
               rms_norm_eps=1e-6, rope_theta=1e6, max_position_embeddings=max_len, qk_layernorm=True, tie_word_embeddings=True)
    return AutoModel.from_config(cfg, device="cuda", block_size=64, seq_length=max_len).eval()


@torch.no_grad()
def kernel_table(size, prompt_batch=4, prompt=4096, decode_batch=64, context=4096):
    """Every kernel of a layer of the two models, prefill (``prompt_batch`` prompts) and decode shapes."""
    from mindformers_b200.inference.paged_attention import paged_attention_forward, _write_cache
    from mindformers_b200.inference.ragged_attention import ragged_attention
    from mindformers_b200.ops import functional as Fn
    from mindformers_b200.ops import recurrent, stream
    from mindformers_b200.parallel.layers.attention import AttnMeta
    W, H, G, D, DH, DG, E, K, FF = (size[k] for k in ("width", "heads", "kv", "dim", "delta", "delta_kv", "experts", "top", "ff"))
    dev, bf = "cuda", torch.bfloat16
    new = lambda *shape, dt=bf: torch.randn(*shape, device=dev, dtype=dt)
    out = Table()
    m, q3 = kukupel(size, 8192), qwen3_moe(size, 8192)
    par, dl, ql = m.model.decoder.layers[0], m.model.decoder.layers[1], q3.model.decoder.layers[0]
    n_str = STREAMS
    for phase, B, n, ctx_len in (("prefill", prompt_batch, prompt, prompt), ("decode", decode_batch, 1, context)):
        T = B * n
        cm, tm = m._set_kv_cache(B, ctx_len)
        step_meta(cm, tm, B, n, ctx_len)
        cq, tq = q3._set_kv_cache(B, ctx_len)
        step_meta(cq, tq, B, n, ctx_len)
        pos = torch.arange(ctx_len - n, ctx_len, device=dev).repeat(B)
        x, y = new(T, W), new(T, W)
        # ---- norm + residual
        xs, link, norm = new(T, n_str, W, dt=torch.float32), par.mlp_connection, par.pre_mlp_layernorm
        out.add(f"{phase} streams: mix + read + norm", "kukupel", lambda: stream.residual_streams(
            xs, n_str, y, link.mix, link.write, link.read, norm.weight, 1e-6), T * W * (8 * n_str + 4))
        out.add(f"{phase} norm + residual", "qwen3_moe", lambda: Fn.rmsnorm(x, ql.input_layernorm.weight, 1e-6, y), T * W * 8)
        del xs
        # ---- attention
        width = (H + 2 * G) * D
        qkv = new(T, width)
        core = par.self_attention.left
        nb = T * width * 4
        out.add(f"{phase} q copy + cache write", "kukupel", lambda: stream.qkv_rope_cache(
            qkv, None, None, None, 1e-6, core.rotary.freqs, 1.0, True, pos, cm.slot_mapping, cm.key_cache[0], cm.value_cache[0], H, G,
            D, D), nb)
        cos, sin = q3.model.rotary_pos_emb()
        qa = ql.self_attention

        def qwen_rope():
            packed, q, k, v = qa._split(qkv)
            packed = torch.cat((qa.q_layernorm(q), qa.k_layernorm(k), v), dim=1)
            packed = Fn.rope(packed, cos, sin, pos, H + G, D, False)
            _write_cache(cq, 0, packed[:, H:H + G], packed[:, H + G:])
        out.add(f"{phase} qk norm + rotation + cache", "qwen3_moe", qwen_rope, nb)
        q = new(T, H, D)
        attend = lambda cap: ragged_attention(q, cm, 0, D ** -0.5, softcap=cap)
        if n > 1:
            pairs = B * n * (n + 1) // 2
            io, fl = T * (H + G) * D * 4, pairs * H * D * 4
            out.add("prefill attention", f"kukupel softcap {SOFTCAP:g}", lambda: attend(SOFTCAP), io, fl)
            out.add("prefill attention", "kukupel kernel, no softcap", lambda: attend(0.0), io, fl)
            k, v = new(B, n, G, D), new(B, n, G, D)
            out.add("prefill attention", "qwen3_moe", lambda: Fn.attention(q.view(B, n, H, D), k, v, True, D ** -0.5), io, fl)
        else:
            io = B * ctx_len * G * D * 4
            out.add("decode attention", f"kukupel softcap {SOFTCAP:g}", lambda: attend(SOFTCAP), io)
            k, v = new(T, G, D), new(T, G, D)
            meta = AttnMeta(batch=1, seq_len=T, positions=pos, cache=cq)
            out.add("decode attention", "qwen3_moe", lambda: paged_attention_forward(q, k, v, meta, 1, D ** -0.5), io)
        del q, k, v, qkv
        # ---- gated delta rule: per head, and per channel with its low-rank factors
        for label, layer, run in (("per head", dl.self_attention.core, 1), ("per channel", par.self_attention.right, 0)):
            s = layer.shape
            proj = new(T, sum(layer.sections))
            meta = AttnMeta(batch=1, seq_len=T, positions=pos, cache=cm, layer_run=run)
            res = torch.empty(T, layer.width, device=dev, dtype=bf)
            state = 2 * B * s.heads * s.dim * s.v_dim * 4
            io = T * (sum(layer.sections) + layer.width) * 2 + state
            row = out.add(f"{phase} delta rule, decays {label}", "kukupel", lambda: layer(proj, meta, res), io)
            flop = 8.0 * T * s.heads * s.dim * s.v_dim           # decay, two products with S, update: two operations each (decay one)
            if n > 1:
                row["of_fma_pipes"] = round(flop / FMA_PEAK * 1e3 / row["ms"], 3)
        # ---- experts
        mlp, qm = par.mlp, ql.mlp
        used = min(E, T * K)
        fl, wb = 6 * T * K * W * FF, 3 * used * W * FF * 2
        io = wb + T * W * 4 + T * K * (W * 4 + FF * 6)
        out.add(f"{phase} experts", "kukupel", lambda: mlp(x), io, fl)
        out.add(f"{phase} experts", "qwen3_moe", lambda: qm(x), io, fl)
        if n > 1:
            h2 = new(T * K, 2 * FF)
            out.add("prefill expert activation", "kukupel", lambda: Fn.clamped_glu(h2, 7.0, 1.702), T * K * FF * 6)
            out.add("prefill expert activation", "qwen3_moe", lambda: Fn.swiglu(h2), T * K * FF * 6)
            del h2
        # ---- projections
        for label, lin, ref in (("parallel in", par.self_attention.linear_in, None), ("delta in", dl.self_attention.linear_in, None),
                                ("parallel out", par.self_attention.linear_proj, None), ("delta out", dl.self_attention.linear_proj, None),
                                ("qkv", None, qa.linear_qkv), ("out", None, qa.linear_proj)):
            mod = lin or ref
            N, Kd = mod.weight.shape
            a = new(T, Kd)
            out.add(f"{phase} projection {label} ({N} x {Kd})", "kukupel" if lin else "qwen3_moe", lambda: mod(a),
                    N * Kd * 2 + T * (N + Kd) * 2, 2 * T * N * Kd)
        r = x[:B].contiguous()
        out.add(f"{phase} head ({B} rows)", "kukupel", lambda: m.model.logits(r).float(), VOCAB * W * 2 + B * VOCAB * 4, 2 * B * W * VOCAB)
        out.add(f"{phase} head ({B} rows)", "qwen3_moe", lambda: q3.model.logits(r).float(), VOCAB * W * 2 + B * VOCAB * 4, 2 * B * W * VOCAB)
        del cm, cq
    return out.rows


def main(sizes=None, kernels=True):
    from mindformers_b200.ops import _lib
    results = {}
    for name in sizes or SIZES:
        size = SIZES[name]
        res = {"size": dict(size, layers=LAYERS, vocab=VOCAB, streams=STREAMS, low_rank=RANK, conv=TAPS)}
        for label, make in (("kukupel", kukupel), ("qwen3_moe", qwen3_moe)):
            torch.manual_seed(0)
            model = make(size, 8192)
            rate, ms = prefill_rate(model, 4, 4096)
            res[label] = {"prefill_tokens_per_s (4 x 4096)": round(rate), "prefill_ms": round(ms, 3)}
            for batch, context in ((1, 4096), (16, 4096), (64, 4096)):
                rate, ms = decode_rate(model, batch, context - 124)
                res[label][f"decode_tokens_per_s (batch {batch}, context ~{context})"] = round(rate)
                res[label][f"decode_ms (batch {batch})"] = round(ms, 4)
            res[label]["parameters"] = model.num_parameters()
            del model
            torch.cuda.empty_cache()
        if kernels:
            res["kernels"] = kernel_table(size)
        torch.cuda.empty_cache()
        results[name] = res
    return {"metric": "prefill and decode tokens/s of Kukupel beside Qwen3-MoE at equal size", "unit": "tokens/s", "n_gpus": 1,
            "dtype": "bf16", "data": "synthetic token ids, random-init weights", "results": results,
            "kernel_status_word": _lib.read_status()}


if __name__ == "__main__":
    print(json.dumps(main(sys.argv[1:] or None)))
