"""Prefill and decode throughput of Togalorn beside Gavatar at equal size, and the roofline fraction of every kernel of the two
(random-init weights, synthetic tokens, one GPU). ``bench.py --config togalorn_serving`` runs it.

Equal size: same width, attention heads, query / key size (Togalorn's with its rotated part), value size, latents, experts,
experts per token, expert width, layers and vocabulary, and the same numbers of state per recurrent layer and of channels that read
it. Half of the layers of each are latent attention, Togalorn's over all earlier tokens, Gavatar's in a window; Togalorn's others have
the state space, Gavatar's the matrix memory and attention by turns. Togalorn's experts have a shared one and identity experts (a
quarter of the real ones) beside them. Model figures are device-timed (CUDA events): prefill is one call over whole prompts, decode
the captured step of the device-side loop. Kernels of a decode step and element-wise kernels are replayed from a graph, so that the
host's launches are not part of their time. L2 is flushed before every timed kernel; the working set of the model runs exceeds it.
Roofline denominators are the measured peaks of ``MEASURED_PEAKS.json``; the recurrences are also put against the nominal rate of
the FMA pipes (148 SMs x 128 lanes at 1965 MHz).
"""
from __future__ import annotations

import json
import os
import sys

import torch

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
if ROOT not in sys.path:
    sys.path.insert(0, ROOT)

from benchmarks.bench_loop_serving import SIZES, captured, gavatar  # noqa: E402
from benchmarks.bench_ragged_serving import LAYERS, VOCAB, Table, decode_rate, prefill_rate, step_meta  # noqa: E402
from benchmarks.bench_recurrent_serving import FMA_PEAK  # noqa: E402

TYPES = "latent_attention mamba2"
HEAD = 64                      # channels per head of the state space
TAPS, NORM_GROUPS, SSM_GROUPS = 4, 4, 1


def togalorn(size, max_len):
    from mindformers_b200.models import AutoModel, TogalornConfig
    D = size["dim"]
    layers = TogalornConfig.layer_list(" ".join([TYPES] * (LAYERS // 2)), size["heads"], D - D // 4, D // 4, D, size["rank"],
                                       size["delta"] * D // HEAD, HEAD, D, size["experts"], size["top"], size["ff"],
                                       q_rank=size["q_rank"], ssm_groups=SSM_GROUPS, norm_groups=NORM_GROUPS,
                                       identity=size["experts"] // 4)
    cfg = TogalornConfig(vocab=VOCAB, width=size["width"], norm=dict(eps=1e-6, groups=NORM_GROUPS), canon=dict(taps=TAPS), layers=layers,
                         seq_length=max_len, embedding=dict(scale=size["width"] ** 0.5), loop=dict(start=0, stop=LAYERS, times=1))
    return AutoModel.from_config(cfg, device="cuda").eval()


@torch.no_grad()
def kernel_table(size, prompt_batch=4, prompt=4096, decode_batch=64, context=4096, only=None):
    """Every kernel of a layer of the two models, prefill (``prompt_batch`` prompts) and decode shapes; ``only``: a part of the
    kernels' names."""
    from mindformers_b200.inference.ragged_attention import latent_attention
    from mindformers_b200.ops import recurrent, stream
    W, H, D, MH, E, K, FF, R, Q, WIN = (size[k] for k in ("width", "heads", "dim", "delta", "experts", "top", "ff", "rank", "q_rank",
                                                          "window"))
    P, I = D // 4, E // 4
    dev, bf = "cuda", torch.bfloat16
    new = lambda *shape, dt=bf: torch.randn(*shape, device=dev, dtype=dt)
    out = Table()

    def add(what, model, fn, *a):
        if only and only not in what:
            return {"ms": 1.0}
        small = what.startswith("decode") or any(w in what for w in ("embedding", "norm", "rotation", "cache", "gates"))
        return out.add(what, model, captured(fn) if small else fn, *a)

    m, ga = togalorn(size, 8192), gavatar(size, 8192)
    lat, ssm = m.model.decoder.layers[0], m.model.decoder.layers[1]
    glat, gmem = ga.model.decoder.layers[0], ga.model.decoder.layers[1]
    for phase, B, n, ctx_len in (("prefill", prompt_batch, prompt, prompt), ("decode", decode_batch, 1, context)):
        T = B * n
        cm, tm = m._set_kv_cache(B, ctx_len)
        step_meta(cm, tm, B, n, ctx_len)
        cg, tg = ga._set_kv_cache(B, ctx_len)
        step_meta(cg, tg, B, n, ctx_len)
        pos = torch.arange(ctx_len - n, ctx_len, device=dev).repeat(B)
        pairs = sum(range(ctx_len - n + 1, ctx_len + 1)) * B                          # (query, key) pairs
        seen = sum(min(i + 1, WIN) for i in range(ctx_len - n, ctx_len)) * B          # ... inside Gavatar's window
        x, y, y2, xs, base = new(T, W), new(T, W), new(T, W), new(T, W, dt=torch.float32), new(T, W, dt=torch.float32)
        # ---- embedding, norms, convolution
        ids = torch.randint(0, VOCAB, (T,), device=dev)
        emb = m.model.embedding
        add(f"{phase} embedding", "togalorn", lambda: emb(ids[None], pos), T * W * 6)
        norm, conv, step = lat.input_layernorm.weight, stream.InputConv(lat.input_conv, cm, 0), m.model.decoder.loop_step[0]
        add(f"{phase} residual + norm + convolution", "togalorn", lambda: stream.joint_step(
            xs, (y, y2), None, None, norm, NORM_GROUPS, 1e-6, bf, conv), T * W * 16)
        add(f"{phase} residual + norm", "togalorn", lambda: stream.joint_step(
            xs, (y, y2), None, None, norm, NORM_GROUPS, 1e-6, bf), T * W * 14)
        add(f"{phase} start of a pass: operand", "togalorn", lambda: stream.joint_step(
            xs, (y, y2), None, None, None, 1, 0.0, bf, keep=False), T * W * 10)
        w_in = m.model.decoder.loop_in[:, :W]
        add(f"{phase} start of a pass: product", "togalorn", lambda: stream.linear(x, w_in, out_dtype=torch.float32),
            W * W * 2 + T * W * 6, 2 * T * W * W)
        gnorms = (glat.post_mlp_layernorm.weight, glat.input_layernorm.weight)
        carry = stream.Carry(glat.token_shift, cg, 0)
        add(f"{phase} norms + residual + shift", "gavatar", lambda: stream.normed_step(xs, y, gnorms[0], None, gnorms[1], 1e-6, True, carry),
            T * W * 12)
        add(f"{phase} norms + residual", "gavatar", lambda: stream.normed_step(xs, y, gnorms[0], None, gnorms[1], 1e-6, True), T * W * 12)
        # ---- latent attention
        la, gl = lat.self_attention, glat.self_attention
        proj, gproj, q, gate = new(T, Q + R + P), new(T, Q + R + H), new(T, H, D), new(T, H * D)
        add(f"{phase} latent norms + rotation + cache write", "togalorn", lambda: stream.latent_norm_cache(
            proj, la.q_latent_norm.weight, la.kv_latent_norm.weight, 1e-6, cm.slot_mapping, cm.key_cache[0], la.rotary.freqs, pos),
            T * (Q + R + P) * 4)
        add(f"{phase} latent norms + cache write", "gavatar", lambda: stream.latent_norm_cache(
            gproj[:, :Q + R], gl.q_latent_norm.weight, gl.kv_latent_norm.weight, 1e-6, cg.slot_mapping, cg.key_cache[0]),
            T * (Q + R) * 4)
        add(f"{phase} rotation of the queries", "togalorn", lambda: stream.rotate_tail_(q, la.rotary.freqs, pos), T * H * P * 4)
        attend = lambda: latent_attention(q, cm, 0, la.linear_kv_up.weight, D, la.scale, v_rank=R)
        gattend = lambda: latent_attention(q, cg, 0, gl.linear_kv_up.weight, D, gl.scale, WIN, gl.sink)
        if n > 1:
            add("prefill latent attention", "togalorn expanded", attend, 0, pairs * H * 4 * D + 2 * T * R * H * (2 * D - P))
            add("prefill latent attention", "gavatar expanded", gattend, 0, seen * H * 4 * D + 2 * T * R * H * 2 * D)
        else:
            add("decode latent attention", "togalorn absorbed", attend, B * ctx_len * (R + P) * 2 + 2 * H * D * R * 2)
            add("decode latent attention", "gavatar absorbed", gattend, B * min(WIN, ctx_len) * R * 2 + 2 * H * D * R * 2)
        o = new(T, H * D)
        add(f"{phase} gates per channel", "togalorn", lambda: stream.gate_heads_(o, gate), T * H * D * 6)
        add(f"{phase} gates per head", "gavatar", lambda: stream.gate_heads_(o, gproj[:, Q + R:]), T * H * D * 4)
        # ---- recurrences
        sm, mm = ssm.self_attention, gmem.self_attention
        s = sm.shape
        state = 2 * B * s.heads * s.state * s.head_dim * 4
        sp, mp = new(T, s.columns), new(T, sum(mm.sections))
        sw = recurrent.StateSpaceWeights(sm.conv, sm.conv_bias, sm.dt_bias, sm.a_log, sm.skip, sm.norm)
        row = add(f"{phase} state space", "togalorn", lambda: recurrent.state_space(sp, sw, s, cm.recurrent[1], cm, 1e-6),
                  T * (s.columns + s.inner) * 2 + state)
        grow = add(f"{phase} matrix memory", "gavatar", lambda: recurrent.matrix_memory(
            mp, mm.input_bias, mm.forget_bias, mm.norm, mm.shape, cg.recurrent[1], cg, 1e-6),
            T * (sum(mm.sections) + MH * D) * 2 + 2 * B * MH * D * D * 4)
        if n > 1:             # operations per token and number of state: decay, update, read-out
            row["of_fma_pipes"] = round(5.0 * T * s.heads * s.state * s.head_dim / FMA_PEAK * 1e3 / row["ms"], 3)
            grow["of_fma_pipes"] = round(5.0 * T * MH * D * D / FMA_PEAK * 1e3 / grow["ms"], 3)
        # ---- experts
        real = K * E / (E + I)
        used = min(E, T * real)
        add(f"{phase} experts", "togalorn", lambda: lat.mlp(x), 3 * (used + 1) * W * FF * 2 + T * W * 4 + T * (real + 1) * (W * 4 + FF * 6),
            6 * T * (real + 1) * W * FF)
        used = min(E, T * K)
        add(f"{phase} experts", "gavatar", lambda: glat.mlp(x), 3 * used * W * FF * 2 + T * W * 4 + T * K * (W * 4 + FF * 6),
            6 * T * K * W * FF)
        # ---- projections
        for label, lin in (("latent in", la.linear_in), ("latent q up", la.linear_q_up), ("latent out", la.linear_proj),
                           ("state space in", sm.linear_in), ("state space out", sm.linear_proj)):
            N, Kd = lin.weight.shape
            a = new(T, Kd)
            add(f"{phase} projection {label} ({N} x {Kd})", "togalorn", lambda: lin(a), N * Kd * 2 + T * (N + Kd) * 2, 2 * T * N * Kd)
        for label, lin in (("latent in", gl.linear_in), ("memory in", mm.linear_in)):
            N, Kd = lin.weight.shape
            a = new(T, Kd)
            add(f"{phase} projection {label} ({N} x {Kd})", "gavatar", lambda: lin(a), N * Kd * 2 + T * (N + Kd) * 2, 2 * T * N * Kd)
        r = x[:B].contiguous()
        for label, model in (("togalorn", m), ("gavatar", ga)):
            add(f"{phase} head ({B} rows)", label, lambda: model.model.logits(r).float(), VOCAB * W * 2 + B * VOCAB * 4,
                2 * B * W * VOCAB)
        del cm, cg, xs, x, y, y2, base, q, o, gate, proj, gproj, sp, mp
    return out.rows


def main(sizes=None, kernels=True):
    from mindformers_b200.ops import _lib
    results = {}
    for name in sizes or SIZES:
        size = SIZES[name]
        res = {"size": dict(size, layers=LAYERS, vocab=VOCAB, types=TYPES, rotated=size["dim"] // 4, head=HEAD, state=size["dim"],
                            identity=size["experts"] // 4)}
        for label, make in (("togalorn", togalorn), ("gavatar", gavatar)):
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
    return {"metric": "prefill and decode tokens/s of Togalorn beside Gavatar at equal size", "unit": "tokens/s", "n_gpus": 1,
            "dtype": "bf16", "data": "synthetic token ids, random-init weights", "results": results,
            "kernel_status_word": _lib.read_status()}


if __name__ == "__main__":
    print(json.dumps(main(sys.argv[1:] or None)))
