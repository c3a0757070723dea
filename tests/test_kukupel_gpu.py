"""Kukupel on the CUDA kernels, against the plain implementation of ``oracles/kukupel.py``: every kernel alone, whole
prompts, portions, decoding, mixed batches with pages and slots used again, generation through the engine."""
import numpy as np
import pytest
import torch

from mindformers_b200.inference import ragged_attention as ragged
from mindformers_b200.inference.paged_attention import KVCacheContext
from mindformers_b200.inference.ragged_attention import ragged_attention
from mindformers_b200.ops import _lib, recurrent, stream
from mindformers_b200.ops import functional as Fn
from mindformers_b200.parallel.layers.moe import PermutePlan
from mindformers_b200.serving import SamplingParams, ServingEngine
from mindformers_b200.serving.trace import build_engine

from oracles import cases, kukupel
from oracles import kukupel_cases as kc
from oracles.paged import attention_case

pytestmark = pytest.mark.gpu
DEV = "cuda"
DTYPES = [torch.float32, torch.bfloat16]
# least limits of the logits' error relative to their spread; where rounding alone gives more, three times that
LIMIT = {"float32": 2e-5, "bfloat16": 4e-2}


def rand(*shape, seed=0, dtype=torch.float32, scale=1.0):
    return (torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * scale).to(dtype)


def rel(got, want):
    return float((got.double().cpu() - want.double()).norm() / want.double().norm())


def tol(dtype, f32=3e-6, bf16=6e-3):
    return f32 if dtype == torch.float32 else bf16


# ---- residual streams ----------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,W", [(1, 8), (3, 101), (5, 192), (2, 4096), (4, 1150), (2, 6152)])
@pytest.mark.parametrize("n", [1, 2, 3, 4, 5, 8, 11])
def test_residual_streams(dtype, T, W, n):
    e, y, w = rand(T, W, seed=1, dtype=dtype), rand(T, W + 8, seed=2, dtype=dtype), rand(W, seed=3, dtype=dtype) + 1
    mix, write, read = rand(n, n, seed=4), rand(n, seed=5), rand(n, seed=6)
    d = lambda t: t.to(DEV)
    h, x = stream.residual_streams(d(e), n, None, None, None, d(read), d(w), 1e-4)
    assert x.dtype == dtype and rel(h, kukupel.rms_norm(read.double().sum() * e.double(), w.double(), 1e-4)) < tol(dtype, 2e-5)
    xs = torch.stack([e.double()] * n)
    ed = d(e)
    for step, (keep, src) in enumerate(((True, ed), (True, None), (False, None))):
        xs = kukupel.write_streams(xs, mix.double(), write.double(), y[:, :W].double())
        h, new = stream.residual_streams(ed if step == 0 else x, n, d(y)[:, :W], d(mix), d(write), d(read) if keep else None, d(w),
                                         1e-4, keep)
        u = kukupel.read_streams(xs, read.double()) if keep else xs.sum(0)
        assert h.dtype == dtype and rel(h, kukupel.rms_norm(u, w.double(), 1e-4)) < tol(dtype, 2e-5), step
        if keep:
            assert new.dtype == torch.float32 and rel(new.transpose(0, 1), xs) < 3e-6
            x = new
        else:
            assert new is None and rel(x.transpose(0, 1), before) < 3e-6          # the streams were not written
        before = xs
    assert torch.equal(ed.cpu(), e)


# ---- soft-capped attention ----------------------------------------------------------------------------------------------
SHAPES = [(4, 2, 64, 64), (8, 2, 128, 128), (6, 2, 40, 24), (6, 3, 48, 96), (20, 1, 24, 40), (3, 1, 20, 36), (2, 1, 144, 12)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,DV", SHAPES)
@pytest.mark.parametrize("softcap,score_scale,persistent", [(30.0, 1.3, 0), (2.0, 1.3, 1000), (20.0, 12.0, 0)])
def test_softcapped_attention(dtype, H, G, D, DV, softcap, score_scale, persistent, monkeypatch):
    """Scores that the cap hardly touches, flattens, and clips here and there; portions and decoded rows; a result that lies
    in a wider matrix and is scaled."""
    monkeypatch.setattr(ragged, "_PERSISTENT_UP_TO", persistent)
    lens, news = [1, 300, 129, 517, 64, 130, 40], [1, 300, 2, 260, 1, 1, 0]
    case = dict(softcap=softcap, score_scale=score_scale)
    ctx, table, qs, _, scale, want = attention_case(dtype, H, G, D, DV, 64, 0, lens, news, seed=D, **case)
    ctx.set_step(is_prefill=True, block_tables=table, slot_mapping=[0] * sum(news), context_lens=lens, q_seq_lens=news, device=DEV)
    wide = torch.full((sum(news), H * DV + 24), 7.0, dtype=dtype, device=DEV)
    got = ragged_attention(torch.cat(qs).to(DEV), ctx, 0, scale, softcap=softcap, out=wide[:, :H * DV], out_scale=0.6)
    assert got.data_ptr() == wide.data_ptr() and bool((wide[:, H * DV:] == 7).all())
    rows = (got.double().cpu() - 0.6 * want).norm(dim=1) / (0.6 * want).norm(dim=1)
    assert float(rows.max()) < tol(dtype, 2e-5, 3e-2), int(rows.argmax())
    lens = [1, 63, 64, 129, 700]
    ctx, table, qs, _, scale, want = attention_case(dtype, H, G, D, DV, 16, 0, lens, [1] * 5, seed=D + 1, **case)
    ctx.set_step(is_prefill=False, block_tables=table, slot_mapping=[0] * 5, context_lens=lens, q_seq_lens=[1] * 5, device=DEV)
    got = ragged_attention(torch.cat(qs).to(DEV), ctx, 0, scale, softcap=softcap, out_scale=1.7)
    rows = (got.double().cpu() - 1.7 * want).norm(dim=1) / (1.7 * want).norm(dim=1)
    assert float(rows.max()) < tol(dtype, 2e-5, 3e-2), int(rows.argmax())
    if softcap == 2.0:
        plain = ragged_attention(torch.cat(qs).to(DEV), ctx, 0, scale)
        assert rel(plain * 1.7, 1.7 * want) > 1e-2                         # the cap shows
    assert _lib.read_status() == 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,DV", [(8, 2, 128, 128), (3, 1, 20, 36)])
def test_softcapped_attention_finds_far_keys(dtype, H, G, D, DV):
    """One key that stands out as far as the cap allows: the first token, keys at page and tile borders, the row itself, and
    the key just after it, which is hidden."""
    n, bs = 400, 16
    for qp, kp in ((399, 0), (399, 15), (399, 16), (398, 127), (399, 128), (300, 300), (300, 301), (257, 255), (2, 3), (2, 1), (0, 0)):
        for lens, news in ((n, n), (max(qp + 2, kp + 1), 2), (qp + 1, 1)):
            if lens > n or kp >= lens:
                continue
            ctx, table, qs, _, scale, want = attention_case(dtype, H, G, D, DV, bs, 0, [lens], [news], seed=qp + kp, spots=[(0, qp, kp)],
                                                            softcap=12.0)
            ctx.set_step(is_prefill=news > 1, block_tables=table, slot_mapping=[0] * news, context_lens=[lens], q_seq_lens=[news],
                         device=DEV)
            got = ragged_attention(qs[0].to(DEV), ctx, 0, scale, softcap=12.0)
            row = qp - (lens - news)
            err = (got[row].double().cpu() - want[row]).norm() / want[row].norm()
            assert float(err) < tol(dtype, 2e-5, 3e-2), (qp, kp, lens, news)
    assert _lib.read_status() == 0


# ---- gated delta rule ------------------------------------------------------------------------------------------------------
DELTA = [(4, 2, 32, 32, 4), (6, 3, 64, 40, 3), (4, 2, 128, 128, 4), (3, 1, 20, 36, 2), (2, 1, 7, 5, 1), (2, 2, 256, 128, 4),
         (2, 2, 256, 256, 4), (2, 1, 160, 72, 5), (1, 1, 300, 40, 4), (5, 5, 48, 96, 6), (34, 2, 16, 16, 4), (2, 1, 96, 200, 3)]


def delta_case(H, G, D, DV, taps, by_channel, seed, dt=(-2.0, 1.0)):
    s = recurrent.DeltaShape(H, G, D, DV, taps, by_channel, not by_channel)
    w = recurrent.DeltaWeights(rand(taps, s.channels, seed=seed, scale=0.5), rand(H, seed=seed + 1, scale=0.7),
                               dt[0] + dt[1] * rand(H * D if by_channel else H, seed=seed + 2), 1 + 0.2 * rand(DV, seed=seed + 3))
    return s, w


def delta_oracle(x, b, a, gate, w, s, eps):
    """Read-out of one whole sequence in float64."""
    x, b, a, gate = (t.double() for t in (x, b, a, gate))
    T, H, G, D, DV = x.shape[0], s.heads, s.kv_heads, s.dim, s.v_dim
    y = kukupel.silu(kukupel.short_conv(x, w.conv.double().t()))
    reps = torch.arange(H) // (H // G)
    q = (kukupel.unit(y[:, :G * D].view(T, G, D)) * D ** -0.5)[:, reps]
    k = kukupel.unit(y[:, G * D:2 * G * D].view(T, G, D))[:, reps]
    raw = kukupel.softplus(a + w.dt_bias.double()).view(T, H, -1)
    g = torch.exp(-torch.exp(w.a_log.double())[None, :, None] * raw).expand(T, H, D)
    o = kukupel.delta_scan(q, k, y[:, 2 * G * D:].view(T, H, DV), torch.sigmoid(b), g)
    z = kukupel.silu(gate) if s.gate_silu else torch.sigmoid(gate)
    return (kukupel.rms_norm(o, w.norm.double(), eps) * z.view(T, H, DV)).reshape(T, H * DV)


class Slots:
    """Sequences on state slots that are full of old values, fed in portions of a common projection matrix."""

    def __init__(self, s, w, dtype, slots=4, eps=1e-4):
        self.s, self.w, self.eps, self.n, self.dtype = s, w, eps, slots, dtype
        self.ctx = KVCacheContext(1, 1, 64, 0, 0, dtype, DEV, layer_shapes=[None], slots=slots,
                                  state_shapes=[(s.heads, s.dim, s.v_dim, s.channels, s.taps)])
        for t in self.ctx.recurrent[0]:
            t.normal_(0, 9)
        self.at = [0] * slots
        self.dw = recurrent.DeltaWeights(*(t.to(DEV).contiguous() for t in (w.conv, w.a_log, w.dt_bias, w.norm)))

    def step(self, rows, prefill=True):
        """``rows``: {slot: (x, b, a, gate) of its next rows}; returns {slot: read-out}."""
        n = [len(rows[i][0]) if i in rows else 0 for i in range(self.n)]
        lens = [self.at[i] + n[i] if prefill or n[i] else 5 for i in range(self.n)]
        if not prefill:                       # every slot has a row; idle ones hold garbage
            some = next(iter(rows.values()))
            rows = {i: rows.get(i) or tuple(torch.full_like(t[:1], 3.0) for t in some) for i in range(self.n)}
        parts = [torch.cat([rows[i][j] for i in sorted(rows)]) for j in range(4)]
        s = self.s
        proj = torch.zeros(parts[0].shape[0], s.channels + 8 + s.heads, dtype=self.dtype, device=DEV)      # x and b share a pitch
        proj[:, :s.channels], proj[:, -s.heads:] = parts[0].to(DEV), parts[1].to(DEV)
        self.ctx.set_step(is_prefill=prefill, block_tables=np.zeros((self.n, 1)),
                          slot_mapping=[0] * sum(n) if prefill else [0 if c else -1 for c in n], context_lens=lens,
                          q_seq_lens=n if prefill else [1] * self.n, device=DEV)
        wide = torch.full((proj.shape[0], s.heads * s.v_dim + 16), 7.0, dtype=self.dtype, device=DEV)
        out = recurrent.delta_rule(proj[:, :s.channels], proj[:, -s.heads:], parts[2].to(DEV), parts[3].to(DEV), self.dw, s,
                                   self.ctx.recurrent[0], self.ctx, self.eps, wide[:, 8:8 + s.heads * s.v_dim], 0.5)
        assert bool((wide[:, :8] == 7).all()) and bool((wide[:, 8 + s.heads * s.v_dim:] == 7).all())
        got, at = {}, 0
        for i in sorted(rows):
            m = len(rows[i][0])
            if n[i]:
                got[i] = out[at:at + m].float().cpu() * 2
            at += m
        self.at = [self.at[i] + n[i] for i in range(self.n)]
        return got


def sequences(s, lens, dtype, seed):
    cols = (s.channels, s.heads, s.heads * s.dim if s.by_channel else s.heads, s.heads * s.v_dim)
    return [tuple(rand(n, c, seed=seed + 10 * i + j, dtype=dtype) for j, c in enumerate(cols)) for i, n in enumerate(lens)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("by_channel", [False, True])
@pytest.mark.parametrize("H,G,D,DV,taps", DELTA)
def test_delta_rule(dtype, by_channel, H, G, D, DV, taps):
    """Unequal sequences in portions down to one row, idle slots, decoded rows, slots taken over by new sequences."""
    s, w = delta_case(H, G, D, DV, taps, by_channel, seed=D)
    seqs = sequences(s, (70, 9, 41, 30), dtype, seed=100 + DV)
    want = [delta_oracle(*q, w, s, 1e-4) for q in seqs]
    run = Slots(s, w, dtype)
    got = [[] for _ in seqs]
    at = [0] * 4

    def go(plan, prefill=True, slot=lambda i: i):
        rows = {slot(i): tuple(t[at[i]:at[i] + c] for t in seqs[i]) for i, c in plan.items()}
        for k, v in run.step(rows, prefill).items():
            i = next(i for i in plan if slot(i) == k)
            got[i].append(v)
        for i, c in plan.items():
            at[i] += c
    go({0: 33, 2: 2})
    go({0: 1, 1: 5, 2: 16})
    go({1: 2, 0: 2})
    go({0: 1, 2: 1}, prefill=False)
    go({2: 18, 0: 3, 1: 1})
    go({1: 1}, prefill=False)
    go({2: 1, 0: 1}, prefill=False)
    go({0: 24, 2: 3})
    for _ in range(5):
        go({0: 1}, prefill=False)
    # sequence 1 is over: sequence 3 starts on its slot, from decoded rows alone and then in a portion
    run.at[1] = 0
    one = lambda i: {3: 1}.get(i, i)
    go({3: 1}, prefill=False, slot=one)
    go({3: 1}, prefill=False, slot=one)
    go({3: 28}, slot=one)
    assert at == [70, 8 + 1, 41, 30]
    for i in range(4):
        rows = torch.cat(got[i]).double()
        err = (rows - want[i]).norm(dim=1) / want[i].norm(dim=1)
        assert float(err.max()) < tol(dtype, 2e-5, 6e-3), (i, int(err.argmax()))


@pytest.mark.parametrize("by_channel", [False, True])
@pytest.mark.parametrize("D,DV", [(128, 128), (20, 36), (256, 256)])
def test_delta_rule_far_writes(by_channel, D, DV):
    """A state that forgets nothing: what the first token wrote is read by rows hundreds of tokens later, with the same unit
    key again, in a prompt, a portion of two tokens and decoded."""
    s, w = delta_case(2, 1, D, DV, 1, by_channel, seed=5, dt=(-40.0, 0.0))
    n = 600
    x, b, a, gate = sequences(s, (n,), torch.float32, seed=3)[0]
    w.conv[:] = 1.0
    a.zero_()
    for t in (n - 3, n - 2, n - 1):
        x[t, :D] = x[0, D:2 * D] * 3                             # the query is the first token's key
    b[1:, :] -= 6.0                                              # later tokens write little
    want = delta_oracle(x, b, a, gate, w, s, 1e-4)
    other = x.clone()
    other[0, 2 * D:] += 1.0
    assert rel(delta_oracle(other, b, a, gate, w, s, 1e-4)[n - 1], want[n - 1]) > 0.05
    for cuts in ((n,), (n - 2, 2), (130, n - 133, 2, 1)):
        run, at, got = Slots(s, w, torch.float32), 0, []
        for c in cuts:
            got.append(run.step({2: tuple(t[at:at + c] for t in (x, b, a, gate))}, prefill=c > 1)[2])
            at += c
        err = (torch.cat(got).double() - want).norm(dim=1) / want.norm(dim=1)
        assert float(err.max()) < 2e-5, (cuts, int(err.argmax()))


def test_delta_rule_does_not_depend_on_the_cut_or_the_slot():
    """fp32 recurrence: portions of any size give the same numbers up to rounding, whatever shares the batch."""
    s, w = delta_case(4, 2, 64, 64, 4, True, seed=7)
    seqs = sequences(s, (150, 77), torch.bfloat16, seed=9)
    ref = None
    for slot, sizes, mate in ((0, (150,), False), (3, (2,) * 75, False), (1, (64, 1, 2, 50, 33), True)):
        run, at, got = Slots(s, w, torch.bfloat16), 0, []
        for c in sizes:
            rows = {slot: tuple(t[at:at + c] for t in seqs[0])}
            if mate and run.at[2] + c <= 77:
                rows[2] = tuple(t[run.at[2]:run.at[2] + c] for t in seqs[1])
            got.append(run.step(rows)[slot])
            at += c
        got = torch.cat(got)
        ref = got if ref is None else ref
        assert float((got - ref).abs().max()) <= 2 ** -7 * float(ref.abs().max())


def test_delta_rule_refuses_wrong_arguments():
    s, w = delta_case(2, 1, 16, 16, 4, False, seed=1)
    run = Slots(s, w, torch.float32)
    x, b, a, gate = (t.to(DEV) for t in sequences(s, (3,), torch.float32, seed=1)[0])
    run.ctx.set_step(is_prefill=True, block_tables=np.zeros((4, 1)), slot_mapping=[0] * 3, context_lens=[3, 0, 0, 0],
                     q_seq_lens=[3, 0, 0, 0], device=DEV)
    with pytest.raises(ValueError, match="pitch"):
        recurrent.delta_rule(x, b, a, gate, run.dw, s, run.ctx.recurrent[0], run.ctx, 1e-4)
    with pytest.raises(TypeError):
        recurrent.delta_rule(x.bfloat16(), b, a, gate, run.dw, s, run.ctx.recurrent[0], run.ctx, 1e-4)


# ---- experts ---------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("R,F", [(128, 64), (300, 50), (1, 8), (640, 200)])
def test_clamped_glu(dtype, R, F):
    x = rand(R, 2 * F, seed=1, dtype=dtype, scale=2.0)
    g, u = x.double().chunk(2, dim=1)
    g, u = g.clamp(max=0.9), u.clamp(-0.9, 0.9)
    want = g * torch.sigmoid(1.702 * g) * (u + 1)
    assert rel(Fn.clamped_glu(x.to(DEV), 0.9, 1.702), want) < tol(dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("N,K", [(64, 192), (50, 33), (200, 96), (7, 100)])
def test_grouped_gemm_of_any_size(dtype, N, K):
    ids = torch.tensor([0, 3, 3, 1, 3] * 40 + [1] * 70, device=DEV)
    plan = PermutePlan(ids, 4)
    x = torch.zeros(plan.rows, K, dtype=dtype, device=DEV)
    rows = rand(ids.numel(), K, seed=2, dtype=dtype)
    x[plan.dest] = rows.to(DEV)
    w = rand(4, K, N, seed=3, dtype=dtype)
    y = Fn.grouped_gemm(x, w.to(DEV), plan.block_group, plan.num_blocks, b_mn=True)
    want = torch.einsum("rk,rkn->rn", rows.double(), w.double()[ids.cpu()])
    assert rel(y[plan.dest], want) < tol(dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["mixed_layers", "chosen_experts", "odd_sizes"])
def test_feed_forward(checkpoints, name, dtype):
    """One decode-sized and one prompt-sized call; the routing weight is on the experts' input."""
    model, cfg, w = checkpoints(name, dtype)
    for T in (1, 5, 300):
        h = rand(T, cfg["width"], seed=T, dtype=torch.bfloat16)
        for i, layer in enumerate(cfg["layers"]):
            if layer["mlp"]:
                with torch.no_grad():
                    got, _ = model.model.decoder.layers[i].mlp(h.to(DEV, getattr(torch, dtype)))
                m = layer["mlp"]
                get = lambda n: w[f"l{i}.mlp.{n}"].double()
                s = torch.sigmoid(h.double() @ get("router").t()).sort(dim=-1, descending=True).values
                top = m["router"]["top"]
                sure = torch.ones(T, dtype=torch.bool) if top == m["router"]["experts"] else s[:, top - 1] - s[:, top] > 1e-4
                want = kukupel.feed_forward(h.double(), get, m)
                assert rel(got[sure.to(DEV)], want[sure]) < tol(getattr(torch, dtype), 3e-6, 1e-2), (T, i)


# ---- the whole model ------------------------------------------------------------------------------------------------------------
@pytest.fixture(scope="module")
def checkpoints(tmp_path_factory):
    made = {}

    def get(name, dtype):
        if name not in made:
            cfg, w = kc.CASES[name], kc.weights(name, seed=len(name))
            made[name] = (cases.write_checkpoint(tmp_path_factory.mktemp(name), cfg, w), cfg, w, {})
        path, cfg, w, models = made[name]
        if dtype not in models:
            models[dtype] = cases.load(path, dtype, DEV)
        return models[dtype], cfg, w
    return get


def sure_rows(name, cfg, w, toks, dtype):
    """Positions that no close choice of experts reaches."""
    if dtype == "float32" or name != "chosen_experts":
        return torch.ones(len(toks), dtype=torch.bool)
    return ~kc.close_calls(cfg, w, toks, 0.02)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(kc.CASES))
def test_logits_do_not_depend_on_the_schedule(checkpoints, name, dtype):
    model, cfg, w = checkpoints(name, dtype)
    toks = {f"r{i}": cases.tokens(n, cfg["vocab"], seed=i) for i, n in enumerate((283, 1, 70, 131, 40))}
    want = {r: kc.expected(cfg, w, t) for r, t in toks.items()}
    sure = {r: sure_rows(name, cfg, w, t, dtype) for r, t in toks.items()}
    noise = {r: kc.rounding(cfg, w, t, dtype) for r, t in toks.items()}

    def check(r, logits, what):
        ok = sure[r]
        if ok.any():
            err, ref = kc.errors(logits, want[r])[ok], noise[r][ok]
            assert float(err.max()) < max(LIMIT[dtype], 3 * float(ref.max())), (r, what, int(err.argmax()))
            assert float(err.median()) < max(LIMIT[dtype] / 10, 3 * float(ref.median())), (r, what)
    whole = [{r: len(t)} for r, t in toks.items()]
    one_by_one = [{"r2": 30}] + [{"r2": 1}] * 40
    cut = [{r: c} for r, t in toks.items() for c in cases.portions(len(t), (2, 37, 1, 64, 3, 65, 2, 2))]
    # at most four live: r4 takes the slot and pages that r1 and r2 gave back
    p0, p3 = cases.portions(283, (100, 2, 29, 64)), cases.portions(131, (33, 1, 1, 50, 2))
    mixed = [{"r0": p0[0], "r1": 1, "r2": 29, "r3": p3[0]}, {"r0": p0[1], "r2": 2}, {"r0": p0[2], "r2": 38, "r3": p3[1]}]
    mixed += [{"r2": 1, "r3": p3[2], "r4": 33}] + [{"r4": 1, "r0": c} for c in p0[3:]]
    mixed += [{"r3": c} for c in p3[3:]]
    mixed += [{"r4": 1}] * (40 - 33 - len(p0[3:]))
    for schedule, pool in ((whole, 320), (cut, 320), (mixed, 640)):
        got = cases.run_schedule(build_engine(model, pool), toks, schedule)
        for r in toks:
            check(r, got[r], schedule[:2])
    got = cases.run_schedule(build_engine(model, 128), {"r2": toks["r2"]}, one_by_one)
    check("r2", got["r2"], "decoded")
    assert _lib.read_status() == 0


@pytest.mark.parametrize("name", ["mixed_layers", "wide_heads"])
def test_long_decoding(checkpoints, name):
    model, cfg, w = checkpoints(name, "bfloat16")
    toks = cases.tokens(330, cfg["vocab"], seed=9)
    got = cases.run_schedule(build_engine(model, 384), {"a": toks}, [{"a": 3}] + [{"a": 1}] * 327)
    err, noise = kc.errors(got["a"], kc.expected(cfg, w, toks)), kc.rounding(cfg, w, toks, "bfloat16")
    assert float(err.max()) < max(LIMIT["bfloat16"], 3 * float(noise.max())) and float(err.median()) < 3 * float(noise.median())


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["mixed_layers", "odd_sizes", "wide_heads"])
def test_greedy_generation(checkpoints, name, dtype):
    """``generate`` (host loop, captured step, device loop: twice, the second time on states that the first call left) and the
    engine's scheduler with mixed steps, bursts, and a pool small enough to preempt."""
    model, cfg, w = checkpoints(name, dtype)
    prompts = [cases.tokens(n, cfg["vocab"], seed=20 + i) for i, n in enumerate((50, 3, 130, 65, 1))]
    slack = 1e-4 if dtype == "float32" else 0.15
    for kw in (dict(), dict(use_cuda_graph=True, device_loop=False), dict(use_cuda_graph=True), dict(use_cuda_graph=True),
               dict(chunk_prefill_size=48)):
        out = model.generate(prompts, max_new_tokens=20, do_sample=False, eos_token_id=None, **kw)
        for p, o in zip(prompts, out):
            assert o[:len(p)] == p and len(o) == len(p) + 20 and kc.greedy_is_right(cfg, w, p, o[len(p):], slack), kw
    model.release_device_loops()
    for burst, blocks in ((0, None), (8, None), (8, 5)):
        engine = ServingEngine(model, max_num_seqs=3, max_model_len=192, num_blocks=blocks, max_prefill_tokens=40, eos_token_id=None,
                               decode_burst=burst)
        reqs = [engine.add_request(f"q{i}", p, SamplingParams(max_tokens=20, temperature=0.0)) for i, p in enumerate(prompts)]
        engine.run_until_idle()
        for p, r in zip(prompts, reqs):
            assert len(r.output) == 20 and kc.greedy_is_right(cfg, w, p, r.output, slack), (burst, blocks, len(p))
        assert engine.counters["mixed_steps"] > 3 and engine.stats()["free_blocks"] == engine.stats()["total_blocks"]
        if burst and not blocks:
            assert engine.counters["bursts"] > 0
        if blocks:
            assert engine.counters["preempted"] > 0
    assert _lib.read_status() == 0


def test_half_precision_and_single_precision_agree_on_the_stream_types(checkpoints):
    """The streams and the states are fp32 in 16-bit models too."""
    model, cfg, _ = checkpoints("mixed_layers", "bfloat16")
    seen = []
    hooks = [layer.register_forward_hook(lambda mod, args, out: seen.append(out[1].x.dtype)) for layer in model.model.decoder.layers]
    with torch.no_grad():
        model(torch.tensor([cases.tokens(12, cfg["vocab"])]))
    for h in hooks:
        h.remove()
    assert seen[-1] == torch.float32
    ctx, _ = model._set_kv_cache(2, 64)
    assert all(r[0].dtype == torch.float32 and r[1].dtype == torch.bfloat16 for r in ctx.recurrent if r is not None)
    assert all(c is None for c, m in zip(ctx.key_cache, cfg["layers"]) if m["type"] == "delta")
