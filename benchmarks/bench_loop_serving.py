"""Prefill and decode throughput of Gavatar beside Kukupel at equal size, and the roofline fraction of every kernel of the two
(random-init weights, synthetic tokens, one GPU). ``bench.py --config gavatar_serving`` runs it.

Equal size: same width, attention heads, head size, recurrent heads and state size, experts, experts per token, expert width,
layers and vocabulary. Half of Gavatar's layers are latent attention, a quarter each matrix memory and attention; every second
Kukupel layer is attention beside a gated delta rule, the others have the delta rule alone. Gavatar's attention has a window.
Model figures are device-timed (CUDA events): prefill is one call over whole prompts, decode the captured step of the device-side
loop. Kernels of a decode step and element-wise kernels are replayed from a graph, so that the host's launches are not part of
their time. L2 is flushed before every timed kernel; the working set of the model runs exceeds it. Roofline denominators are the
measured peaks of ``MEASURED_PEAKS.json``; the recurrences are also put against the nominal rate of the FMA pipes (148 SMs x 128
lanes at 1965 MHz).
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
from benchmarks.bench_recurrent_serving import FMA_PEAK, SIZES as KUKUPEL_SIZES, STREAMS, kukupel  # noqa: E402

EXTRA = {
    "w4096_h32_kv8_d128_e32_top4": dict(rank=512, q_rank=1536, window=2048),
    "w2048_h16_kv4_d128_e64_top8": dict(rank=256, q_rank=768, window=1024),
    "w2048_h32_kv8_d64_e64_top8": dict(rank=256, q_rank=768, window=1024),
}
SIZES = {name: dict(size, **EXTRA[name]) for name, size in KUKUPEL_SIZES.items()}
TYPES = "latent_attention mlstm latent_attention attention"


def gavatar(size, max_len):
    from mindformers_b200.models import AutoModel, GavatarConfig
    layers = GavatarConfig.layer_list(" ".join([TYPES] * (LAYERS // 4)), size["heads"], size["kv"], size["dim"], size["rank"],
                                      size["window"], size["delta"], size["dim"], size["experts"], size["top"], size["ff"],
                                      q_rank=size["q_rank"])
    cfg = GavatarConfig(vocab=VOCAB, width=size["width"], norm=dict(eps=1e-6), layers=layers, seq_length=max_len,
                        embedding=dict(scale=size["width"] ** 0.5), loop=dict(start=0, stop=LAYERS, times=1))
    return AutoModel.from_config(cfg, device="cuda").eval()


def captured(fn):
    """``fn`` as a CUDA graph: the host's launches are not part of what is timed."""
    side = torch.cuda.Stream()
    side.wait_stream(torch.cuda.current_stream())
    with torch.cuda.stream(side):
        fn()
        fn()
    torch.cuda.current_stream().wait_stream(side)
    torch.cuda.synchronize()
    graph = torch.cuda.CUDAGraph()
    with torch.cuda.graph(graph):
        fn()
    return graph.replay


@torch.no_grad()
def kernel_table(size, prompt_batch=4, prompt=4096, decode_batch=64, context=4096, only=None):
    """Every kernel of a layer of the two models, prefill (``prompt_batch`` prompts) and decode shapes; ``only``: a part of the
    kernels' names."""
    from mindformers_b200.inference.paged_attention import mla_decode_attention
    from mindformers_b200.inference.ragged_attention import latent_attention, ragged_attention, talking_attention
    from mindformers_b200.ops import functional as Fn
    from mindformers_b200.ops import recurrent, stream
    from mindformers_b200.parallel.layers.attention import AttnMeta
    W, H, G, D, MH, E, K, FF, R, Q, WIN = (size[k] for k in ("width", "heads", "kv", "dim", "delta", "experts", "top", "ff", "rank",
                                                             "q_rank", "window"))
    dev, bf = "cuda", torch.bfloat16
    new = lambda *shape, dt=bf: torch.randn(*shape, device=dev, dtype=dt)
    out = Table()

    def add(what, model, fn, *a):
        if only and only not in what:
            return {"ms": 1.0}
        small = what.startswith("decode") or any(w in what for w in ("embedding", "norms", "streams", "cache", "gates"))
        return out.add(what, model, captured(fn) if small else fn, *a)

    m, ku = gavatar(size, 8192), kukupel(size, 8192)
    latl, mem, att = (m.model.decoder.layers[i] for i in (0, 1, 3))
    kpar, kdl = ku.model.decoder.layers[0], ku.model.decoder.layers[1]
    for phase, B, n, ctx_len in (("prefill", prompt_batch, prompt, prompt), ("decode", decode_batch, 1, context)):
        T = B * n
        cm, tm = m._set_kv_cache(B, ctx_len)
        step_meta(cm, tm, B, n, ctx_len)
        ck, tk = ku._set_kv_cache(B, ctx_len)
        step_meta(ck, tk, B, n, ctx_len)
        pos = torch.arange(ctx_len - n, ctx_len, device=dev).repeat(B)
        seen = sum(min(i + 1, WIN) for i in range(ctx_len - n, ctx_len)) * B          # (query, key) pairs inside the window
        x, y, xs = new(T, W), new(T, W), new(T, W, dt=torch.float32)
        # ---- embedding, norms, shift
        ids = torch.randint(0, VOCAB, (T,), device=dev)
        emb = m.model.embedding
        add(f"{phase} embedding + positions", "gavatar", lambda: emb(ids[None], pos), T * W * 6)
        norms = (latl.post_mlp_layernorm.weight, latl.input_layernorm, m.model.decoder.loop_step[0])
        carry = stream.Carry(latl.token_shift, cm, 0)
        add(f"{phase} norms + residual + shift", "gavatar", lambda: stream.normed_step(
            xs, y, norms[0], None, norms[1].weight, 1e-6, True, carry), T * W * 12)
        add(f"{phase} norms + residual", "gavatar", lambda: stream.normed_step(
            xs, y, norms[0], None, norms[1].weight, 1e-6, True), T * W * 12)
        st, link, norm = new(T, STREAMS, W, dt=torch.float32), kpar.mlp_connection, kpar.pre_mlp_layernorm
        add(f"{phase} streams: mix + read + norm", "kukupel", lambda: stream.residual_streams(
            st, STREAMS, y, link.mix, link.write, link.read, norm.weight, 1e-6), T * W * (8 * STREAMS + 4))
        del st
        # ---- attention
        width = (H + 2 * G) * D
        qkv, gate = new(T, width), new(T, H * D)
        sa, left = att.self_attention, kpar.self_attention.left
        for label, core, ctx, layer, unit in (("gavatar", sa, cm, 3, True), ("kukupel", left, ck, 0, False)):
            add(f"{phase} q, k, v + cache write", label, lambda: stream.qkv_rope_cache(
                qkv, sa.qkv_bias if unit else None, None, None, 1e-6, core.rotary.freqs, 1.0, True, pos, ctx.slot_mapping,
                ctx.key_cache[layer], ctx.value_cache[layer], H, G, D, D, unit, unit), T * width * 4)
        q = new(T, H, D)
        kv_bytes = B * min(WIN, ctx_len) * G * D * 4 if n == 1 else 0
        talk_flop = seen * H * (4 * D + 2 * H)
        mixed = lambda: talking_attention(q, cm, 3, sa.scale, sa.talk, gate, WIN)
        add(f"{phase} attention", "gavatar window, mixed weights, gate", mixed, kv_bytes or T * (3 * H + 2 * G) * D * 2,
            talk_flop if n > 1 else 0)
        add(f"{phase} attention", "gavatar kernel, window alone", lambda: ragged_attention(q, cm, 3, sa.scale, window=WIN),
            kv_bytes or T * (2 * H + 2 * G) * D * 2, seen * H * 4 * D if n > 1 else 0)
        full = B * n * (n + 1) // 2
        add(f"{phase} attention", "kukupel kernel", lambda: ragged_attention(q, ck, 0, D ** -0.5, softcap=30.0),
            T * (2 * H + 2 * G) * D * 2 if n > 1 else B * ctx_len * G * D * 4, full * H * 4 * D if n > 1 else 0)
        # ---- latent attention
        la = latl.self_attention
        proj = new(T, Q + R + H)
        add(f"{phase} latent norms + cache write", "gavatar", lambda: stream.latent_norm_cache(
            proj[:, :Q + R], la.q_latent_norm.weight, la.kv_latent_norm.weight, 1e-6, cm.slot_mapping, cm.key_cache[0]),
            T * (Q + R) * 4)
        lat = lambda: latent_attention(q, cm, 0, la.linear_kv_up.weight, D, la.scale, WIN, la.sink)
        if n > 1:
            add("prefill latent attention", "gavatar expanded", lat, 0, seen * H * 4 * D + 2 * T * R * H * 2 * D)
        else:
            io = B * min(WIN, ctx_len) * R * 2
            add("decode latent attention", "gavatar absorbed", lat, io + 2 * H * D * R * 2)
            if R == 512:
                cache = torch.zeros(B * WIN // 64, 64, 576, dtype=bf, device=dev)
                table = torch.arange(B * WIN // 64, dtype=torch.int32, device=dev).view(B, -1)
                lens, q576 = torch.full((B,), WIN, dtype=torch.int32, device=dev), new(B, H, 576)
                holder = AttnMeta()
                add("decode latent attention", "deepseek kernel, 512 + 64 columns", lambda: mla_decode_attention(
                    q576, cache, table, lens, 64, 0.1, holder), B * WIN * 576 * 2)
        add(f"{phase} gates per head", "gavatar", lambda: stream.gate_heads_(x[:, :H * D], proj[:, Q + R:]), T * H * D * 4)
        # ---- recurrences
        state = 2 * B * MH * D * D * 4
        mm = mem.self_attention
        mp = new(T, sum(mm.sections))
        row = add(f"{phase} matrix memory", "gavatar", lambda: recurrent.matrix_memory(
            mp, mm.input_bias, mm.forget_bias, mm.norm, mm.shape, cm.recurrent[1], cm, 1e-6),
            T * (sum(mm.sections) + MH * D) * 2 + state)
        core = kdl.self_attention.core
        dp = new(T, sum(core.sections))
        meta = AttnMeta(batch=1, seq_len=T, positions=pos, cache=ck, layer_run=1)
        res = torch.empty(T, core.width, device=dev, dtype=bf)
        krow = add(f"{phase} delta rule", "kukupel", lambda: core(dp, meta, res), T * (sum(core.sections) + core.width) * 2 + state)
        if n > 1:             # operations per token, head and element of the state: decay, update, read-out; delta: another product
            row["of_fma_pipes"] = round(5.0 * T * MH * D * D / FMA_PEAK * 1e3 / row["ms"], 3)
            krow["of_fma_pipes"] = round(8.0 * T * MH * D * D / FMA_PEAK * 1e3 / krow["ms"], 3)
        # ---- experts
        used = min(E, T * K)
        io, fl = 3 * used * W * FF * 2 + T * W * 4 + T * K * (W * 4 + FF * 6), 6 * T * K * W * FF
        add(f"{phase} experts", "gavatar", lambda: latl.mlp(x), io, fl)
        add(f"{phase} experts", "kukupel", lambda: kpar.mlp(x), io, fl)
        # ---- projections
        for label, lin in (("latent in", la.linear_in), ("latent q up", la.linear_q_up), ("memory in", mm.linear_in),
                           ("attention in", sa.linear_qkv), ("out", la.linear_proj)):
            N, Kd = lin.weight.shape
            a = new(T, Kd)
            add(f"{phase} projection {label} ({N} x {Kd})", "gavatar", lambda: lin(a), N * Kd * 2 + T * (N + Kd) * 2, 2 * T * N * Kd)
        for label, lin in (("parallel in", kpar.self_attention.linear_in), ("parallel out", kpar.self_attention.linear_proj)):
            N, Kd = lin.weight.shape
            a = new(T, Kd)
            add(f"{phase} projection {label} ({N} x {Kd})", "kukupel", lambda: lin(a), N * Kd * 2 + T * (N + Kd) * 2, 2 * T * N * Kd)
        r = x[:B].contiguous()
        for label, model in (("gavatar", m), ("kukupel", ku)):
            add(f"{phase} head ({B} rows)", label, lambda: model.model.logits(r).float(), VOCAB * W * 2 + B * VOCAB * 4,
                2 * B * W * VOCAB)
        del cm, ck, xs, x, y, qkv, gate, q, mp, dp
    return out.rows


def main(sizes=None, kernels=True):
    from mindformers_b200.ops import _lib
    results = {}
    for name in sizes or SIZES:
        size = SIZES[name]
        res = {"size": dict(size, layers=LAYERS, vocab=VOCAB, types=TYPES)}
        for label, make in (("gavatar", gavatar), ("kukupel", kukupel)):
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
    return {"metric": "prefill and decode tokens/s of Gavatar beside Kukupel at equal size", "unit": "tokens/s", "n_gpus": 1,
            "dtype": "bf16", "data": "synthetic token ids, random-init weights", "results": results,
            "kernel_status_word": _lib.read_status()}


if __name__ == "__main__":
    print(json.dumps(main(sys.argv[1:] or None)))
