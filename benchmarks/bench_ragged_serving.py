"""Prefill and decode throughput of Mefesun beside Qwen3 at equal size, and the roofline fraction of every kernel of the
two (random-init weights, synthetic tokens, one GPU). ``bench.py --config mefesun_serving`` runs it.

Equal size: same width, heads, head size, layers and vocabulary, and a feed-forward with as many weights (Mefesun's has
two matrices, Qwen3's three). Model figures are device-timed (CUDA events): prefill is one call over whole prompts,
decode the captured step of the device-side loop. The working set of every timed region exceeds the 126 MB L2 or L2 is
flushed between iterations. Roofline denominators are the measured peaks of ``MEASURED_PEAKS.json``.
"""
from __future__ import annotations

import json
import os
import sys

import torch

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
if ROOT not in sys.path:
    sys.path.insert(0, ROOT)

SIZES = {
    "w4096_h32_kv8_d128": dict(width=4096, heads=32, kv=8, dim=128, ff=12288, chunk=2048),
    "w2048_h16_kv4_d128": dict(width=2048, heads=16, kv=4, dim=128, ff=6144, chunk=1024),
    "w2048_h32_kv8_d64": dict(width=2048, heads=32, kv=8, dim=64, ff=6144, chunk=1024),
}
VOCAB, LAYERS = 32768, 8


def peaks():
    path = os.path.join(ROOT, "MEASURED_PEAKS.json")
    if os.path.exists(path):
        with open(path) as f:
            d = json.load(f)
        return d["hbm_gbs"] * 1e9, d["bf16_tflops"] * 1e12, "measured"
    return 6.65e12, 1.59e15, "fallback"


def mefesun(size, max_len):
    from mindformers_b200.models import AutoModel, MefesunConfig
    cfg = MefesunConfig(vocab=VOCAB, width=size["width"], norm=dict(eps=1e-6), logit_softcap=30.0, seq_length=max_len,
                        layers=MefesunConfig.uniform_layers(LAYERS, size["heads"], size["kv"], size["dim"], size["ff"] * 3 // 2,
                                                            size["chunk"]))
    return AutoModel.from_config(cfg, device="cuda").eval()


def qwen3(size, max_len):
    from mindformers_b200.models import AutoModel
    cfg = dict(model_type="qwen3", num_hidden_layers=LAYERS, hidden_size=size["width"], num_attention_heads=size["heads"],
               num_key_value_heads=size["kv"], head_dim=size["dim"], intermediate_size=size["ff"], vocab_size=VOCAB,
               rms_norm_eps=1e-6, rope_theta=1e6, max_position_embeddings=max_len, qk_layernorm=True,
               tie_word_embeddings=True)
    return AutoModel.from_config(cfg, device="cuda", block_size=64, seq_length=max_len).eval()


def timed(fn, iters, warmup=3, flush=None):
    """Median milliseconds of ``fn`` (device events around each call; ``flush`` runs before every call)."""
    for _ in range(warmup):
        fn()
    ev = [(torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)) for _ in range(iters)]
    for a, b in ev:
        if flush is not None:
            flush.zero_()
        a.record()
        fn()
        b.record()
    torch.cuda.synchronize()
    return sorted(a.elapsed_time(b) for a, b in ev)[iters // 2]


def prefill_rate(model, batch, prompt):
    g = torch.Generator().manual_seed(1)
    toks = torch.randint(3, VOCAB, (batch, prompt), generator=g).tolist()
    ctx, tables = model._set_kv_cache(batch, prompt + 64)

    def step():
        tables.init_cache_engine(batch)
        model._forward_step(toks, [0] * batch, ctx, tables, True)
    ms = timed(step, 5)
    tables.clear_cache()
    return batch * prompt / ms * 1e3, ms


def decode_rate(model, batch, context, steps=48):
    ctx, tables = model._set_kv_cache(batch, context + 128)
    tables.init_cache_engine(batch)
    for e in tables.engines:
        e.reserve(context + 128)
        e.num_tokens = context
    table, slots = tables.assemble_pa_inc_inputs([True] * batch, 1)
    entry = {"ctx": ctx, "captures": 0}
    loop = model._build_device_loop(entry, batch, tables.max_blocks_per_seq, tables.block_size, 128)
    st = loop["state"]
    st.load([5] * batch, [context] * batch, table, slots, [False] * batch, [context + 120] * batch)
    st.set_sampling((), 0.0, 0)
    with torch.no_grad():
        graph = loop["capture"]()
        for _ in range(3):
            graph.replay()
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        for _ in range(steps):
            graph.replay()
        b.record()
    torch.cuda.synchronize()
    ms = a.elapsed_time(b) / steps
    del graph
    loop.clear()
    return batch / ms * 1e3, ms


class Table:
    """Rows ``(what, model, milliseconds, fraction of the measured peak, bound)``."""

    def __init__(self):
        self.hbm, self.flops, self.source = peaks()
        self.rows, self.flush = [], torch.empty(64 << 20, dtype=torch.float32, device="cuda")      # 256 MB, above L2

    def add(self, what, model, fn, nbytes=0, flop=0):
        ms = timed(fn, 9, flush=self.flush)
        t_mem, t_math = nbytes / self.hbm * 1e3, flop / self.flops * 1e3
        self.rows.append({"kernel": what, "model": model, "ms": round(ms, 4),
                          "of_" + self.source: round(max(t_mem, t_math) / ms, 3), "bound": "hbm" if t_mem >= t_math else "tensor"})
        return self.rows[-1]


def step_meta(ctx, tables, batch, new, context):
    """Cache context of a step with ``new`` tokens per sequence that ends at ``context``."""
    tables.init_cache_engine(batch)
    for e in tables.engines:
        e.reserve(context)
        e.num_tokens = context - new
    table, slots = (tables.assemble_pa_full_inputs([new] * batch) if new > 1 else tables.assemble_pa_inc_inputs(None, 1))
    ctx.set_step(is_prefill=new > 1, block_tables=table, slot_mapping=slots, context_lens=[context] * batch,
                 q_seq_lens=[new] * batch, device="cuda")


@torch.no_grad()
def kernel_table(size, prompt_batch=4, prompt=4096, decode_batch=64, context=4096):
    """Every kernel of a layer of the two models, prefill (``prompt_batch`` prompts) and decode shapes."""
    from mindformers_b200.inference.paged_attention import paged_attention_forward, _write_cache
    from mindformers_b200.inference.ragged_attention import ragged_attention
    from mindformers_b200.ops import functional as Fn
    from mindformers_b200.ops import stream
    from mindformers_b200.parallel.layers.attention import AttnMeta
    from mindformers_b200.parallel.layers.norm import RMSNorm
    W, H, G, D, C = (size[k] for k in ("width", "heads", "kv", "dim", "chunk"))
    dev, bf = "cuda", torch.bfloat16
    new = lambda *shape, dt=bf: torch.randn(*shape, device=dev, dtype=dt)
    out = Table()
    m, q3 = mefesun(size, 8192), qwen3(size, 8192)
    ml, ql = m.model.decoder.layers[0], q3.model.decoder.layers[0]
    for phase, B, n, ctx_len in (("prefill", prompt_batch, prompt, prompt), ("decode", decode_batch, 1, context)):
        T = B * n
        cm, tm = m._set_kv_cache(B, ctx_len)
        step_meta(cm, tm, B, n, ctx_len)
        cq, tq = q3._set_kv_cache(B, ctx_len)
        step_meta(cq, tq, B, n, ctx_len)
        pos = torch.arange(ctx_len - n, ctx_len, device=dev).repeat(B)
        x, y, xf = new(T, W), new(T, W), new(T, W, dt=torch.float32)
        qkv = new(T, (H + 2 * G) * D)
        # ---- norm + residual: bf16 y and embedding-type copy, fp32 stream read and written / bf16 stream
        norm, ln = ml.post_attn_layernorm, (ml.self_attention.linear_proj.bias, ml.attn_layer_scale)
        out.add(f"{phase} norm + residual", "mefesun",
                lambda: stream.add_normed(xf, y, ln[0], norm.weight, norm.bias, ln[1], 1e-6, True, inplace=True), T * W * 12)
        out.add(f"{phase} norm + residual", "qwen3", lambda: Fn.rmsnorm(x, ql.input_layernorm.weight, 1e-6, y), T * W * 8)
        # ---- q / k norm, rotation, cache write
        a = ml.self_attention
        nb = T * (H + 2 * G) * D * 4
        out.add(f"{phase} qk norm + rotation + cache", "mefesun", lambda: stream.qkv_rope_cache(
            qkv, a.linear_qkv.bias, a.q_layernorm.weight, a.k_layernorm.weight, 1e-6, a.rotary.freqs, a.rotary.amplitude, True, pos,
            cm.slot_mapping, cm.key_cache[0], cm.value_cache[0], H, G, D, D), nb)
        cos, sin = q3.model.rotary_pos_emb()
        qa = ql.self_attention

        def qwen_rope():
            packed, q, k, v = qa._split(qkv)
            packed = torch.cat((qa.q_layernorm(q), qa.k_layernorm(k), v), dim=1)
            packed = Fn.rope(packed, cos, sin, pos, H + G, D, False)
            _write_cache(cq, 0, packed[:, H:H + G], packed[:, H + G:])
        out.add(f"{phase} qk norm + rotation + cache", "qwen3", qwen_rope, nb)
        # ---- attention
        q = new(T, H, D)
        if n > 1:
            seen = sum(min(i % C, i) + 1 for i in range(n)) * B            # (query, key) pairs under the chunk mask
            out.add("prefill attention", f"mefesun chunk {C}",
                    lambda: ragged_attention(q, cm, 0, D ** -0.5, C, a.sink), T * (H + G) * D * 4, seen * H * D * 4)
            full = B * n * (n + 1) // 2
            out.add("prefill attention", "mefesun kernel, no chunks",
                    lambda: ragged_attention(q, cm, 0, D ** -0.5, 0, a.sink), T * (H + G) * D * 4, full * H * D * 4)
            k, v = new(B, n, G, D), new(B, n, G, D)
            out.add("prefill attention", "qwen3", lambda: Fn.attention(q.view(B, n, H, D), k, v, True, D ** -0.5),
                    T * (H + G) * D * 4, full * H * D * 4)
        else:
            last = (ctx_len - 1) % C + 1                                   # keys of the chunk that ends at the last position
            out.add("decode attention", f"mefesun chunk {C}", lambda: ragged_attention(q, cm, 0, D ** -0.5, C, a.sink),
                    B * last * G * D * 4)
            out.add("decode attention", "mefesun kernel, no chunks", lambda: ragged_attention(q, cm, 0, D ** -0.5, 0, a.sink),
                    B * ctx_len * G * D * 4)
            k, v = new(T, G, D), new(T, G, D)
            meta = AttnMeta(batch=1, seq_len=T, positions=pos, cache=cq)
            out.add("decode attention", "qwen3", lambda: paged_attention_forward(q, k, v, meta, 1, D ** -0.5),
                    B * ctx_len * G * D * 4)
        # ---- feed-forward: projections with their activation
        fm, fq = size["ff"] * 3 // 2, size["ff"]
        wbytes = 2 * W * fm * 2
        out.add(f"{phase} feed-forward", "mefesun", lambda: ml.mlp(x), wbytes + T * (2 * W + (2 if n > 1 else 0) * fm) * 2, 4 * T * W * fm)
        out.add(f"{phase} feed-forward", "qwen3", lambda: ql.mlp(x), wbytes + T * (2 * W + (3 if n > 1 else 0) * fq) * 2, 4 * T * W * fm)
        if n > 1:
            h, g2 = new(T, fm), new(T, 2 * fq)
            out.add("prefill activation", "mefesun", lambda: stream.relu2(h), T * fm * 4)
            out.add("prefill activation", "qwen3", lambda: Fn.swiglu(g2), T * fq * 6)
        # ---- attention projections
        out.add(f"{phase} qkv projection", "mefesun", lambda: a.linear_qkv(x), W * (H + 2 * G) * D * 2 + T * (W + (H + 2 * G) * D) * 2,
                2 * T * W * (H + 2 * G) * D)
        out.add(f"{phase} qkv projection", "qwen3", lambda: qa.linear_qkv(x), W * (H + 2 * G) * D * 2 + T * (W + (H + 2 * G) * D) * 2,
                2 * T * W * (H + 2 * G) * D)
        # ---- head on one row per sequence
        r = x[:B].contiguous()
        out.add(f"{phase} head ({B} rows)", "mefesun", lambda: m.model.logits(r).float(), VOCAB * W * 2 + B * VOCAB * 4, 2 * B * W * VOCAB)
        out.add(f"{phase} head ({B} rows)", "qwen3", lambda: q3.model.logits(r).float(), VOCAB * W * 2 + B * VOCAB * 4, 2 * B * W * VOCAB)
        xs = new(T, W, dt=torch.float32)
        fl = m.model.decoder.final_layernorm
        out.add(f"{phase} final norm", "mefesun", lambda: stream.norm_stream(xs, fl.weight, fl.bias, 1e-6, True), T * W * 6)
        out.add(f"{phase} final norm", "qwen3", lambda: Fn.rmsnorm(x, ql.input_layernorm.weight, 1e-6), T * W * 4)
        del cm, cq
    return out.rows


def main(sizes=None, kernels=True):
    from mindformers_b200.ops import _lib
    results = {}
    for name in sizes or SIZES:
        size = SIZES[name]
        res = {"size": dict(size, layers=LAYERS, vocab=VOCAB, mefesun_ff=size["ff"] * 3 // 2)}
        for label, make in (("mefesun", mefesun), ("qwen3", qwen3)):
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
    return {"metric": "prefill and decode tokens/s of Mefesun beside Qwen3 at equal size", "unit": "tokens/s", "n_gpus": 1,
            "dtype": "bf16", "data": "synthetic token ids, random-init weights", "results": results,
            "kernel_status_word": _lib.read_status()}


if __name__ == "__main__":
    print(json.dumps(main(sys.argv[1:] or None)))
