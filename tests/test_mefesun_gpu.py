"""The Mefesun design on the CUDA kernels, against the plain implementation of ``oracles/mefesun.py``: every kernel alone,
whole prompts, portions, decoding, mixed batches with pages and slots used again, generation through the engine."""
import pytest
import torch

from mindformers_b200.inference import ragged_attention as ragged
from mindformers_b200.inference.ragged_attention import ragged_attention
from mindformers_b200.ops import _lib, stream
from mindformers_b200.serving import SamplingParams, ServingEngine
from mindformers_b200.serving.trace import build_engine

from oracles import cases, mefesun
from oracles.paged import attention_case

pytestmark = pytest.mark.gpu
DEV = "cuda"
DTYPES = [torch.float32, torch.bfloat16]
# error of the logits relative to their spread: rounding alone gives about 1e-6 (fp32 kernels) and 1e-2 (bf16)
LIMIT = {"float32": 2e-5, "bfloat16": 4e-2}


def rand(*shape, seed=0, dtype=torch.float32, scale=1.0):
    return (torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * scale).to(dtype)


def rel(got, want):
    return float((got.double().cpu() - want.double()).norm() / want.double().norm())


def tol(dtype, f32=2e-6, bf16=5e-3):
    return f32 if dtype == torch.float32 else bf16


# ---- single mechanisms ---------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,W", [(1, 8), (3, 100), (5, 192), (2, 4096), (7, 5000), (2, 6152)])
@pytest.mark.parametrize("layer_norm", [True, False])
def test_add_normed(dtype, T, W, layer_norm):
    y = rand(T, W, seed=1, dtype=dtype) + 0.5
    bias, w, b, ls = (rand(W, seed=s, dtype=dtype) for s in (2, 3, 4, 5))
    x = rand(T, W, seed=6)

    def want(x, bias, b, ls):
        v = y.double() + (bias.double() if bias is not None else 0)
        n = mefesun.layer_norm(v, w.double(), 0, 1e-4) if layer_norm else mefesun.rms_norm(v, w.double(), 1e-4)
        n = n + (b.double() if b is not None else 0)
        return x.double() + n * (ls.double() if ls is not None else 1)
    c = lambda t: None if t is None else t.to(DEV)
    for args in ((bias, b, ls), (None, None, ls), (bias, b, None)):
        xd = x.to(DEV)
        copy, s = stream.add_normed(xd, y.to(DEV), c(args[0]), c(w), c(args[1]), c(args[2]), 1e-4, layer_norm, inplace=True)
        assert s.data_ptr() == xd.data_ptr() and s.dtype == torch.float32 and copy.dtype == dtype
        assert rel(s, want(x, *args)) < 2e-6 and rel(copy, want(x, *args)) < tol(dtype)
    # first sub-layer: the residual is the embedding in the activation dtype and is left alone
    e = rand(T, W, seed=8, dtype=dtype)
    ed = e.to(DEV)
    _, s = stream.add_normed(ed, y.to(DEV), c(bias), c(w), c(b), c(ls), 1e-4, layer_norm)
    assert torch.equal(ed.cpu(), e) and rel(s, want(e, bias, b, ls)) < 2e-6
    z = stream.norm_stream(x.to(DEV), c(w), c(b), 1e-4, layer_norm)
    n = mefesun.layer_norm(x.double(), w.double(), 0, 1e-4) if layer_norm else mefesun.rms_norm(x.double(), w.double(), 1e-4)
    assert z.dtype == dtype and rel(z, n + b.double()) < tol(dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", [(1, 7), (3, 64), (130, 1000)])
def test_relu2_and_softcap(dtype, shape):
    x = rand(*shape, seed=1, dtype=dtype)
    want = torch.relu(x.double()) ** 2
    assert rel(stream.relu2(x.to(DEV)), want) < tol(dtype)
    wide = torch.zeros(shape[0], shape[1] + 5, dtype=dtype, device=DEV)
    wide[:, :shape[1]] = x.to(DEV)
    assert rel(stream.relu2(wide[:, :shape[1]]), want) < tol(dtype)
    z = rand(*shape, seed=2, scale=30.0)
    wide = torch.zeros(shape[0], shape[1] + 3, device=DEV)
    view = wide[:, :shape[1]]
    view.copy_(z)
    assert rel(stream.softcap_(view, 12.5), mefesun.softcap(z.double(), 12.5)) < 2e-6
    assert float(wide[:, shape[1]:].abs().max()) == 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("M,N,K", [(1, 77, 100), (4, 301, 176), (64, 96, 40), (3, 515, 128), (65, 77, 90), (130, 301, 176), (300, 512, 256)])
@pytest.mark.parametrize("act", [None, "relu2", "softcap"])
def test_linear_with_activation(dtype, M, N, K, act):
    x, w = rand(M, K, seed=1, dtype=dtype), rand(N, K, seed=2, dtype=dtype)
    want = x.double() @ w.double().t()
    want = {None: want, "relu2": torch.relu(want) ** 2, "softcap": mefesun.softcap(want, 8.0)}[act]
    got = stream.linear(x.to(DEV), w.to(DEV), act=act, cap=8.0)
    assert got.shape == (M, N) and got.dtype == (torch.float32 if act == "softcap" else dtype)
    # the capped logits come from unrounded accumulators
    assert rel(got, want) < (2e-6 if dtype == torch.float32 or act == "softcap" else 6e-3)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,DV,rot", [(4, 2, 64, 64, 64), (6, 2, 40, 24, 16), (5, 1, 128, 128, 96), (3, 3, 20, 36, 12),
                                          (2, 1, 144, 12, 144), (34, 9, 64, 32, 40), (17, 1, 256, 8, 256), (70, 2, 32, 4, 6), (8, 8, 16, 16, 0), (2, 2, 7, 5, 4)])
@pytest.mark.parametrize("interleaved", [True, False])
def test_qkv_rope_cache(dtype, H, G, D, DV, rot, interleaved):
    T, bs, blocks, eps = 9, 16, 5, 1e-3
    nq, nk, nv = H * D, G * D, G * DV
    qkv, bias = rand(T, nq + nk + nv, seed=1, dtype=dtype), rand(nq + nk + nv, seed=2, dtype=dtype)
    qn, kn = rand(D, seed=3, dtype=dtype), rand(D, seed=4, dtype=dtype)
    pos = torch.tensor([0, 1, 2, 500, 501, 9000, 70000, 3, 4])
    slots = torch.tensor([5, 79, 0, 17, -1, 33, 34, -1, 48], dtype=torch.int32)
    if rot:
        freqs, amp = mefesun.yarn_frequencies(rot, 5000.0, dict(factor=4.0, original=64, fast=16.0, slow=1.0))
    else:
        freqs, amp = [], 1.0
    fr = torch.tensor(freqs, dtype=torch.float32)
    kc = torch.full((blocks, bs, G, D), 7.0, dtype=dtype, device=DEV)
    vc = torch.full((blocks, bs, G, DV), 7.0, dtype=dtype, device=DEV)
    d = lambda t: t.to(DEV)
    wide = torch.zeros(T, nq + nk + nv + 8, dtype=dtype, device=DEV)          # a padded pitch, as a GEMM may return it
    wide[:, :nq + nk + nv] = d(qkv)
    for src in (d(qkv), wide[:, :nq + nk + nv]):
        q = stream.qkv_rope_cache(src, d(bias), d(qn), d(kn), eps, d(fr), amp, interleaved, d(pos), d(slots), kc, vc, H, G, D, DV)
    x = qkv.double() + bias.double()

    def side(a, n, w):
        a = mefesun.rms_norm(a.view(T, n, D), w.double(), eps)
        if not rot:
            return a
        if not interleaved:           # bring the halves into pairs, rotate, and back
            perm = [i // 2 + (i % 2) * (rot // 2) for i in range(rot)]
            b = a.clone()
            b[..., :rot] = a[..., perm]
            b = mefesun.rotate_pairs(b, pos, [float(f) for f in fr], amp)
            a = b.clone()
            a[..., perm] = b[..., :rot]
            return a
        return mefesun.rotate_pairs(a, pos, [float(f) for f in fr], amp)
    wq, wk, wv = side(x[:, :nq], H, qn), side(x[:, nq:nq + nk], G, kn), x[:, nq + nk:].view(T, G, DV)
    # fp32 angles: position 70000 times a frequency is good to about 4e-3 radians
    near = pos < 10000
    assert rel(q[d(near)], wq[near]) < tol(dtype, 3e-4) and rel(q, wq) < tol(dtype, 5e-3)
    assert rel(q[:3], wq[:3]) < tol(dtype)
    kf, vf = kc.view(-1, G, D).cpu(), vc.view(-1, G, DV).cpu()
    for t in range(T):
        if slots[t] >= 0:
            assert rel(kf[slots[t]], wk[t]) < tol(dtype, 5e-3) and rel(vf[slots[t]], wv[t]) < tol(dtype)
    untouched = [s for s in range(blocks * bs) if s not in slots.tolist()]
    assert bool((kf[untouched] == 7).all()) and bool((vf[untouched] == 7).all())


ATTENTION = [(4, 2, 64, 64), (8, 2, 128, 128), (6, 2, 40, 24), (5, 5, 128, 64), (3, 1, 64, 128), (20, 1, 24, 40), (3, 1, 20, 36),
             (2, 1, 144, 12)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,DV", ATTENTION)
@pytest.mark.parametrize("bs,persistent", [(16, 0), (64, 0), (64, 1000)])
def test_ragged_attention(dtype, H, G, D, DV, bs, persistent, monkeypatch):
    """Mixed batch: whole prompts, later portions, single rows, a sequence left out; chunks smaller than a key tile, at its
    size and above, that do not divide it, and no chunks at all."""
    monkeypatch.setattr(ragged, "_PERSISTENT_UP_TO", persistent)
    lens, news = [1, 300, 129, 517, 64, 130, 40], [1, 300, 2, 260, 1, 1, 0]
    for chunk in (0, 21, 64, 128, 200):
        ctx, table, qs, sink, scale, want = attention_case(dtype, H, G, D, DV, bs, chunk, lens, news, seed=chunk)
        ctx.set_step(is_prefill=True, block_tables=table, slot_mapping=[0] * sum(news), context_lens=lens, q_seq_lens=news, device=DEV)
        got = ragged_attention(torch.cat(qs).to(DEV), ctx, 0, scale, chunk, sink.to(DEV))
        assert torch.isfinite(got).all() and rel(got, want) < tol(dtype, 2e-6, 8e-3), chunk
        rows = (got.double().cpu() - want).norm(dim=1) / want.norm(dim=1)
        assert float(rows.max()) < tol(dtype, 1e-5, 3e-2), (chunk, int(rows.argmax()))
    assert _lib.read_status() == 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,DV", ATTENTION)
@pytest.mark.parametrize("bs", [16, 128])
def test_decode_attention(dtype, H, G, D, DV, bs):
    lens = [1, 63, 64, 65, 128, 129, 700, 256]
    for chunk in (0, 50, 64, 257):
        ctx, table, qs, sink, scale, want = attention_case(dtype, H, G, D, DV, bs, chunk, lens, [1] * 8, seed=chunk)
        ctx.set_step(is_prefill=False, block_tables=table, slot_mapping=[0] * 8, context_lens=lens, q_seq_lens=[1] * 8, device=DEV)
        got = ragged_attention(torch.cat(qs).to(DEV), ctx, 0, scale, chunk, sink.to(DEV))
        rows = (got.double().cpu() - want).norm(dim=1) / want.norm(dim=1)
        assert float(rows.max()) < tol(dtype, 1e-5, 3e-2), (chunk, int(rows.argmax()))
        plain = ragged_attention(torch.cat(qs).to(DEV), ctx, 0, scale, chunk, None)
        assert rel(plain, want) > 1e-2                                             # the sink shows
    assert _lib.read_status() == 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,DV", [(8, 2, 128, 128), (4, 2, 64, 64), (3, 1, 20, 36)])
@pytest.mark.parametrize("chunk", [0, 48, 64, 192])
def test_attention_at_edges(dtype, H, G, D, DV, chunk):
    """One key that would decide the row, just inside and just outside the visible range: the first key of the chunk, the
    last of the chunk before, the token itself, keys at page borders, the first token; in a prompt, in a portion of two
    tokens, and decoded."""
    n, bs = 400, 16
    c = chunk or n
    spots = []
    for qp in (399, 385, 384, 383, 200, 193, 192, 191, 65, 64, 63, 48, 47, 1, 0):
        first = qp - qp % c
        spots += [(qp, kp) for kp in {first, first - 1, qp, qp - 1, qp + 1, first + 15, first + 16, 0} if 0 <= kp < n]
    for qp, kp in spots:
        for lens, news in ((n, n), (qp + 2, 2), (qp + 1, 1)):
            if lens > n or kp >= lens or (news == n and (qp + kp) % 3):
                continue
            ctx, table, qs, sink, scale, want = attention_case(dtype, H, G, D, DV, bs, chunk, [lens], [news], seed=qp * n + kp,
                                                               spots=[(0, qp, kp)])
            ctx.set_step(is_prefill=news > 1, block_tables=table, slot_mapping=[0] * news, context_lens=[lens], q_seq_lens=[news],
                         device=DEV)
            got = ragged_attention(qs[0].to(DEV), ctx, 0, scale, chunk, sink.to(DEV))
            row = qp - (lens - news)
            err = (got[row].double().cpu() - want[row]).norm() / want[row].norm()
            assert float(err) < tol(dtype, 1e-5, 3e-2), (qp, kp, lens, news)
    assert _lib.read_status() == 0


# ---- the whole model -------------------------------------------------------------------------------------------------------
@pytest.fixture(scope="module")
def checkpoints(tmp_path_factory):
    made = {}

    def get(name, dtype):
        if name not in made:
            cfg = cases.CASES[name]
            w = mefesun.random_weights(cfg, seed=len(name))
            made[name] = (cases.write_checkpoint(tmp_path_factory.mktemp(name), cfg, w), cfg, w, {})
        path, cfg, w, models = made[name]
        if dtype not in models:
            models[dtype] = cases.load(path, dtype, DEV)
        return models[dtype], cfg, w
    return get


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(cases.CASES))
def test_logits_do_not_depend_on_the_schedule(checkpoints, name, dtype):
    model, cfg, w = checkpoints(name, dtype)
    toks = {f"r{i}": cases.tokens(n, cfg["vocab"], seed=i) for i, n in enumerate((283, 1, 70, 131, 40))}
    want = {r: cases.expected(cfg, w, t) for r, t in toks.items()}
    lim = LIMIT[dtype]
    whole = [{r: len(t)} for r, t in toks.items()]
    one_by_one = [{"r2": 30}] + [{"r2": 1}] * 40
    cut = [{r: c} for r, t in toks.items() for c in cases.portions(len(t), (2, 37, 1, 64, 3, 65))]
    # at most four live: r4 takes the slot and pages that r1 and r2 gave back
    p0, p3 = cases.portions(283, (100, 2, 29, 64)), cases.portions(131, (33, 1, 1, 50, 2))
    mixed = [{"r0": p0[0], "r1": 1, "r2": 29, "r3": p3[0]}, {"r0": p0[1], "r2": 2}, {"r0": p0[2], "r2": 38, "r3": p3[1]}]
    mixed += [{"r2": 1, "r3": p3[2], "r4": 33}] + [{"r4": 1, "r0": c} for c in p0[3:]]
    mixed += [{"r3": c} for c in p3[3:]]
    left = 40 - 33 - len(p0[3:])
    mixed += [{"r4": 1}] * left
    for schedule, pool in ((whole, 320), (cut, 320), (mixed, 640)):
        got = cases.run_schedule(build_engine(model, pool), toks, schedule)
        for r in toks:
            assert cases.worst(got[r], want[r]) < lim, (r, schedule[:2])
    got = cases.run_schedule(build_engine(model, 128), {"r2": toks["r2"]}, one_by_one)
    assert cases.worst(got["r2"], want["r2"]) < lim
    assert _lib.read_status() == 0


@pytest.mark.parametrize("name", ["mixed_layers", "wide_heads"])
def test_long_decoding(checkpoints, name):
    model, cfg, w = checkpoints(name, "bfloat16")
    toks = cases.tokens(330, cfg["vocab"], seed=9)
    got = cases.run_schedule(build_engine(model, 384), {"a": toks}, [{"a": 3}] + [{"a": 1}] * 327)
    assert cases.worst(got["a"], cases.expected(cfg, w, toks)) < LIMIT["bfloat16"]


def greedy_is_right(cfg, w, prompt, out, slack):
    """Every generated token is the plain implementation's best one, up to rounding."""
    logits = cases.expected(cfg, w, prompt + out)[len(prompt) - 1:-1]
    best = logits.max(-1).values
    took = logits[torch.arange(len(out)), torch.tensor(out)]
    return float((best - took).max()) <= slack * float(logits.std())


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["mixed_layers", "wide_heads"])
def test_greedy_generation(checkpoints, name, dtype):
    """``generate`` (host loop, captured step, device loop) and the engine's scheduler with mixed steps, bursts, and a pool
    small enough to preempt."""
    model, cfg, w = checkpoints(name, dtype)
    prompts = [cases.tokens(n, cfg["vocab"], seed=20 + i) for i, n in enumerate((50, 3, 130, 65, 1))]
    slack = 1e-4 if dtype == "float32" else 0.15
    for kw in (dict(), dict(use_cuda_graph=True, device_loop=False), dict(use_cuda_graph=True), dict(chunk_prefill_size=48)):
        out = model.generate(prompts, max_new_tokens=20, do_sample=False, eos_token_id=None, **kw)
        for p, o in zip(prompts, out):
            assert o[:len(p)] == p and len(o) == len(p) + 20 and greedy_is_right(cfg, w, p, o[len(p):], slack), kw
    for burst, blocks in ((0, None), (8, None), (8, 5)):
        engine = ServingEngine(model, max_num_seqs=3, max_model_len=192, num_blocks=blocks, max_prefill_tokens=40, eos_token_id=None,
                               decode_burst=burst)
        reqs = [engine.add_request(f"q{i}", p, SamplingParams(max_tokens=20, temperature=0.0)) for i, p in enumerate(prompts)]
        engine.run_until_idle()
        for p, r in zip(prompts, reqs):
            assert len(r.output) == 20 and greedy_is_right(cfg, w, p, r.output, slack), (burst, blocks, len(p))
        assert engine.counters["mixed_steps"] > 3 and engine.stats()["free_blocks"] == engine.stats()["total_blocks"]
        if blocks:
            assert engine.counters["preempted"] > 0
    assert _lib.read_status() == 0
