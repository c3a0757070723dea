"""Togalorn on the CUDA kernels, against the plain implementation of ``oracles/togalorn.py``: every kernel alone, whole prompts,
portions, decoding, mixed batches with pages and slots used again, generation through the engine."""
import numpy as np
import pytest
import torch

from mindformers_b200.inference.paged_attention import KVCacheContext
from mindformers_b200.inference.ragged_attention import latent_attention
from mindformers_b200.ops import _lib, recurrent, stream
from mindformers_b200.parallel.layers.ragged_attention import expand_kv_up
from mindformers_b200.serving import SamplingParams, ServingEngine
from mindformers_b200.serving.trace import build_engine

from oracles import cases, togalorn
from oracles import togalorn_cases as tc

pytestmark = pytest.mark.gpu
DEV = "cuda"
DTYPES = [torch.float32, torch.bfloat16]
# least limits of the logits' error relative to their spread; where rounding alone gives more, three times that
LIMIT = {"float32": 2e-5, "bfloat16": 4e-2}


def rand(*shape, seed=0, dtype=torch.float32, scale=1.0):
    return (torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * scale).to(dtype)


def rel(got, want):
    return float((got.double().cpu() - want.double()).norm() / want.double().norm())


def rows_rel(got, want):
    return (got.double().cpu() - want.double()).norm(dim=1) / want.double().norm(dim=1)


def tol(dtype, f32=3e-6, bf16=6e-3):
    return f32 if dtype == torch.float32 else bf16


class Slots:
    """Sequences on state slots that are full of old values, fed in portions. ``states``: the tensors of ``run`` (layer 1 of two),
    slots first; ``call(rows)``: the op on the step's rows."""

    def __init__(self, dtype, call, states, slots=4, **kw):
        self.ctx = KVCacheContext(2, 1, 64, 0, 0, dtype, DEV, layer_shapes=[None] * 2, slots=slots, **kw)
        self.call, self.states, self.n, self.dtype = call, states(self.ctx), slots, dtype
        for t in self.states:
            t.normal_(0, 9)
        self.at = [0] * slots

    def step(self, rows, prefill=True):
        """``rows``: {slot: its next rows}; returns {slot: result}."""
        n = [len(rows[i]) if i in rows else 0 for i in range(self.n)]
        lens = [self.at[i] + n[i] if prefill or n[i] else 5 for i in range(self.n)]
        some = next(iter(rows.values()))
        if not prefill:                       # every slot has a row; idle ones hold garbage
            rows = {i: rows.get(i, torch.full((1, some.shape[1]), 3.0, dtype=some.dtype)) for i in range(self.n)}
        x = torch.cat([rows[i] for i in sorted(rows)])
        self.ctx.set_step(is_prefill=prefill, block_tables=np.zeros((self.n, 1)),
                          slot_mapping=[0] * sum(n) if prefill else [0 if c else -1 for c in n], context_lens=lens,
                          q_seq_lens=n if prefill else [1] * self.n, device=DEV)
        idle = [i for i in range(self.n) if not n[i]]
        kept = [t[idle].clone() for t in self.states]
        out = self.call(self.ctx, x)
        assert all(torch.equal(t[idle], k) for t, k in zip(self.states, kept))
        got, at = {}, 0
        for i in sorted(rows):
            m = len(rows[i])
            if n[i]:
                got[i] = out[at:at + m].float().cpu()
                assert torch.isfinite(got[i]).all()
            at += m
        self.at = [self.at[i] + n[i] for i in range(self.n)]
        return got

    def visit(self, seqs):
        """Unequal sequences (270, 9, 141 and 30 rows) in portions down to one row, idle slots, decoded rows, a slot taken over by a
        new sequence. Returns the result of every sequence."""
        got, at = [[] for _ in seqs], [0] * 4

        def go(plan, prefill=True, slot=lambda i: i):
            rows = {slot(i): seqs[i][at[i]:at[i] + c] for i, c in plan.items()}
            for k, v in self.step(rows, prefill).items():
                got[next(i for i in plan if slot(i) == k)].append(v)
            for i, c in plan.items():
                at[i] += c
        go({0: 33, 2: 2})
        go({0: 1, 1: 5, 2: 66})
        go({1: 2, 0: 2})
        go({0: 1, 2: 1}, prefill=False)
        go({2: 64, 0: 3, 1: 1})
        go({1: 1}, prefill=False)
        go({2: 1, 0: 1}, prefill=False)
        go({0: 224, 2: 7})
        for _ in range(5):
            go({0: 1}, prefill=False)
        # sequence 1 is over: sequence 3 starts on its slot, from decoded rows alone and then in a portion
        self.at[1] = 0
        one = lambda i: {3: 1}.get(i, i)
        go({3: 1}, prefill=False, slot=one)
        go({3: 1}, prefill=False, slot=one)
        go({3: 28}, slot=one)
        assert at == [270, 9, 141, 30]
        return [torch.cat(g) for g in got]


VISIT = (270, 9, 141, 30)


# ---- the stream -----------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,W,groups", [(1, 8, 1), (3, 105, 3), (5, 192, 6), (2, 4096, 4), (4, 1150, 5), (3, 8192, 1), (2, 9000, 2), (2, 4100, 1)])
def test_joint_step(dtype, T, W, groups):
    x, y0, y1, base = rand(T, W, seed=1), rand(T, W + 8, seed=2, dtype=dtype), rand(T, W, seed=3, dtype=dtype), rand(T, W, seed=4)
    w, vec = rand(W, seed=5, dtype=dtype) + 1, rand(W, seed=6, dtype=dtype)
    d = lambda t: None if t is None else t.to(DEV)
    for ys, b, s, keep in (((y0[:, :W], y1), base, vec, True), ((None, y1), None, None, False), ((y0[:, :W], None), None, vec, True),
                           ((), base, None, True)):
        x2 = x.double() + sum(t.double() for t in ys if t is not None) + sum(t.double() for t in (b, s) if t is not None)
        xd = d(x)
        wide = d(y0)
        yd = tuple(wide[:, :W] if t is not None and t.data_ptr() == y0.data_ptr() else d(t) for t in ys)
        h, hc, new = stream.joint_step(xd, yd, d(b), d(s), d(w), groups, 1e-3, dtype, keep=keep)
        assert hc is None and h.dtype == dtype and rel(h, togalorn.grouped_norm(x2, w.double(), groups, 1e-3)) < tol(dtype, 2e-6)
        assert torch.equal(xd.cpu(), x) and (new is None if not keep else rel(new, x2) < 2e-6)
    h, _, new = stream.joint_step(d(x), (), None, None, None, 1, 0.0, dtype)
    assert torch.equal(h.cpu(), x.to(dtype)) and torch.equal(new.cpu(), x)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("W,groups,taps,scale", [(96, 2, 3, 1), (105, 3, 4, 1), (2048, 4, 4, 1), (64, 1, 2, 400), (320, 5, 3, 300), (48, 2, 1, 1),
                                                 (64, 2, 9, 1), (33, 1, 16, 1), (128, 2, 8, 100)])
def test_input_convolution(dtype, W, groups, taps, scale):
    """With ``scale`` portions long enough for CTAs of several rows; portions shorter than the convolution."""
    w, conv = rand(W, seed=1, dtype=dtype) + 1, rand(W, taps, seed=2)
    seqs = [rand(n * scale, W, seed=10 + i) for i, n in enumerate((20, 9, 13))] if scale > 1 else [rand(n, W, seed=i) for i, n in enumerate(VISIT)]
    want = []
    for s in seqs:
        h = togalorn.grouped_norm(s.double(), w.double(), groups, 1e-5)
        k = conv.double()
        pad = torch.cat((h.new_zeros(taps - 1, W), h))
        want.append(h + sum(k[:, j] * pad[j:j + len(h)] for j in range(taps)))
    assert rel(want[1], togalorn.grouped_norm(seqs[1].double(), w.double(), groups, 1e-5)) > 0.1
    kd, wd = conv.t().contiguous().to(DEV), w.to(DEV)
    run = Slots(dtype, lambda ctx, x: stream.joint_step(x.to(DEV), (), None, None, wd, groups, 1e-5, dtype, stream.InputConv(kd, ctx, 1),
                                                        want_h=False)[1],
                lambda ctx: [] if taps == 1 else [ctx.carry[1]], carry_width=(taps - 1) * W)
    if scale == 1:
        got = run.visit(seqs)
    else:
        got, at = [[], [], []], [0, 0, 0]
        for plan in ({0: 7 * scale, 1: 1}, {0: 2, 2: 5 * scale, 1: 4 * scale}, {1: 2, 2: 1}, None):
            plan = plan or {i: len(seqs[i]) - at[i] for i in range(3)}
            for i, v in run.step({i: seqs[i][at[i]:at[i] + c] for i, c in plan.items()}).items():
                got[i].append(v)
                at[i] += plan[i]
        got = [torch.cat(g) for g in got]
    for g, x in zip(got, want):
        assert float(rows_rel(g, x).max()) < tol(dtype, 3e-6)


# ---- latent attention -------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("Q,R,P,more", [(64, 128, 32, 9), (33, 7, 2, 9), (1536, 512, 64, 8), (264, 72, 8, 16), (8, 2048, 16, 0), (40, 24, 6, 2)])
def test_latent_norm_rotation_and_cache_write(dtype, Q, R, P, more):
    T = 5
    x, qn, kn = rand(T, Q + R + P + more, seed=1, dtype=dtype), rand(Q, seed=2, dtype=dtype) + 1, rand(R, seed=3, dtype=dtype) + 1
    cache = torch.zeros(6, 1, 1, R + P, dtype=dtype, device=DEV)
    slots, pos = torch.tensor([5, 0, -1, 2, 3], dtype=torch.int32, device=DEV), torch.tensor([0, 1, 5, 130, 1000])
    freqs = (500.0 ** (-torch.arange(0, P, 2, dtype=torch.float64) / P)).float()
    q = stream.latent_norm_cache(x.to(DEV)[:, :Q + R + P], qn.to(DEV), kn.to(DEV), 1e-3, slots, cache, freqs.to(DEV), pos.to(DEV))
    xd = x.double()
    assert rel(q, togalorn.rms(xd[:, :Q], 1e-3) * qn.double()) < tol(dtype)
    c = togalorn.rms(xd[:, Q:Q + R], 1e-3) * kn.double()
    keep = [0, 1, 3, 4]
    got = cache[[5, 0, 2, 3], 0, 0]
    assert rel(got[:, :R], c[keep]) < tol(dtype)
    k = togalorn.rotate(xd[:, Q + R:Q + R + P], 500.0, pos)
    assert rel(got[:, R:], k[keep]) < tol(dtype, 1e-4) and rel(got[:2, R:], k[:2]) < tol(dtype, 1e-6)
    assert float(cache[[1, 4]].abs().max()) == 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,D,P", [(4, 24, 8), (3, 13, 6), (8, 96, 32), (5, 64, 64), (40, 32, 16), (1, 0, 2), (300, 8, 8)])
def test_rotation_of_the_last_dimensions(dtype, H, D, P):
    x, pos = rand(4, H, D + P, seed=1, dtype=dtype), torch.tensor([0, 3, 64, 900])
    freqs = (1e4 ** (-torch.arange(0, P, 2, dtype=torch.float64) / P)).float()
    got = stream.rotate_tail_(x.to(DEV), freqs.to(DEV), pos.to(DEV)).cpu()
    assert torch.equal(got[..., :D], x[..., :D])
    want = togalorn.rotate(x[..., D:].double(), 1e4, pos)
    assert rel(got[..., D:], want) < tol(dtype, 1e-4) and rel(got[:2, :, D:], want[:2]) < tol(dtype, 1e-6)


def latent_case(dtype, H, D, P, DV, R, bs, lens, news, seed=0, spots=()):
    """Cached latents with a rotated key part in shuffled pages full of old rows, queries, and the expected attention. ``spots``:
    (sequence, query position, key position) whose score, through the rotated part alone, is made to stand out."""
    g = torch.Generator().manual_seed(seed)
    per = [-(-n // bs) for n in lens]
    perm = torch.randperm(sum(per) + 3, generator=g).tolist()
    ctx = KVCacheContext(1, sum(per) + 3, bs, 0, 0, dtype, DEV, layer_shapes=[(1, R + P, 0)])
    ctx.key_cache[0].copy_((torch.randn(ctx.key_cache[0].shape, generator=g) * 5).to(dtype))
    table = torch.full((len(lens), max(per) + 2), -1, dtype=torch.int32)
    uk, uv = (torch.randn(H * n, R, generator=g) * R ** -0.5 for n in (D, DV))
    uk, uv = uk.to(dtype), uv.to(dtype)
    scale, qs, want = 1.3 * (D + P) ** -0.5, [], []
    for b, (n, m) in enumerate(zip(lens, news)):
        for i in range(per[b]):
            table[b, i] = perm.pop()
        c, q = torch.randn(n, R + P, generator=g), torch.randn(m, H, D + P, generator=g)
        for sb, qp, kp in spots:
            if sb == b:
                c[kp, R:] = q[qp - (n - m), :, D:].mean(0) * 12 * H ** 0.5
        c, q = c.to(dtype), q.to(dtype)
        for t in range(n):
            ctx.key_cache[0][int(table[b, t // bs]), t % bs, 0] = c[t].to(DEV)
        cd, qd = c.double(), q.double()
        k = (cd[:, :R] @ uk.double().t()).view(n, H, D)
        v = (cd[:, :R] @ uv.double().t()).view(n, H, DV)
        s = (torch.einsum("qhd,khd->hqk", qd[..., :D], k) + torch.einsum("qhp,kp->hqk", qd[..., D:], cd[:, R:])) * scale
        hide = torch.arange(n)[None] > torch.arange(n - m, n)[:, None]
        p = torch.softmax(s.masked_fill(hide, float("-inf")), dim=-1)
        want.append(torch.einsum("hqk,khv->qhv", p, v).reshape(m, H * DV))
        qs.append(q)
    return ctx, table, torch.cat(qs), expand_kv_up(uk, uv, H, D, P).to(DEV), scale, torch.cat(want)


LATENT = [(4, 48, 16, 64, 128), (8, 96, 32, 128, 512), (16, 128, 64, 128, 512), (20, 24, 8, 40, 200), (3, 13, 4, 11, 29), (2, 32, 64, 96, 64),
          (40, 64, 64, 64, 256), (33, 16, 8, 8, 320), (5, 8, 24, 32, 104), (4, 128, 64, 64, 192), (2, 72, 72, 136, 64)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,D,P,DV,R", LATENT)
def test_latent_attention(dtype, H, D, P, DV, R):
    """Expanded portions, absorbed rows and both in one batch."""
    for lens, news, bs, ragged_step in (([1, 300, 129, 517, 64, 130, 40], [1, 300, 2, 260, 1, 1, 0], 64, True),
                                        ([70, 3], [1, 1], 64, True), ([200], [90], 16, True), ([1, 63, 64, 129, 700], [1] * 5, 16, False)):
        ctx, table, q, w, scale, want = latent_case(dtype, H, D, P, DV, R, bs, lens, news, seed=R)
        ctx.set_step(is_prefill=ragged_step, block_tables=table, slot_mapping=[0] * sum(news), context_lens=lens, q_seq_lens=news,
                     device=DEV)
        got = latent_attention(q.to(DEV), ctx, 0, w, DV, scale, v_rank=R)
        err = rows_rel(got, want)
        assert float(err.max()) < tol(dtype, 2e-5, 4e-2), (ragged_step, lens, int(err.argmax()))
        assert float(err.median()) < tol(dtype, 1e-5, 1e-2), (ragged_step, lens)
    assert _lib.read_status() == 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,D,P,DV,R", [(8, 96, 32, 128, 256), (3, 13, 4, 11, 29), (4, 128, 64, 128, 512)])
def test_a_far_rotated_key_is_found(dtype, H, D, P, DV, R):
    """One key whose rotated part stands out, at page and tile borders; in a prompt, in a portion of two rows and decoded."""
    n, bs = 400, 16
    for qp in (399, 256, 128, 127, 16):
        for kp in (0, 1, 15, 16, 127, 128, qp, qp + 1):
            for lens, news in ((n, n), (qp + 2, 2), (qp + 1, 1)):
                if lens > n or kp >= lens:
                    continue
                ctx, table, q, w, scale, want = latent_case(dtype, H, D, P, DV, R, bs, [lens], [news], seed=qp + kp, spots=[(0, qp, kp)])
                ctx.set_step(is_prefill=news > 1, block_tables=table, slot_mapping=[0] * news, context_lens=[lens], q_seq_lens=[news],
                             device=DEV)
                got = latent_attention(q.to(DEV), ctx, 0, w, DV, scale, v_rank=R)
                row = qp - (lens - news)
                err = (got[row].double().cpu() - want[row]).norm() / want[row].norm()
                assert float(err) < tol(dtype, 2e-5, 4e-2), (qp, kp, lens, news)
    assert _lib.read_status() == 0


# ---- state space ------------------------------------------------------------------------------------------------------------
# heads, channels per head, state, groups, taps, parts of the norm
SPACE = [(8, 64, 128, 1, 4, 8), (6, 48, 32, 2, 3, 2), (4, 64, 64, 4, 4, 1), (3, 20, 36, 1, 2, 3), (2, 7, 5, 2, 6, 1), (2, 128, 256, 1, 4, 4),
         (5, 16, 16, 5, 1, 5), (2, 72, 160, 2, 4, 2), (1, 200, 24, 1, 3, 1), (16, 8, 8, 4, 16, 2), (1, 24, 300, 1, 4, 1), (40, 32, 128, 8, 4, 1),
         (2, 136, 512, 1, 2, 2), (3, 40, 88, 3, 4, 6)]


def space_weights(s, seed, decay=(-1.0, 1.0), step=(-2.0, 1.0)):
    conv = rand(s.channels, s.taps, seed=seed, scale=0.6)
    return {"conv": conv, "conv.b": rand(s.channels, seed=seed + 1, scale=0.2), "dt_bias": step[0] + step[1] * rand(s.heads, seed=seed + 2),
            "A_log": decay[0] + decay[1] * rand(s.heads, seed=seed + 3), "D": 1 + 0.5 * rand(s.heads, seed=seed + 4),
            "norm": 1 + 0.2 * rand(s.inner, seed=seed + 5)}


def space_oracle(proj, w, s, eps, dtype, arith=torch.float64):
    """Result of one whole sequence, the convolution's activations rounded to ``dtype``."""
    w = {n: t.to(arith) for n, t in w.items()}
    T, p = proj.shape[0], proj.to(arith)
    z, xbc, dt = torch.split(p, (s.inner, s.channels, s.heads), dim=1)
    pad = torch.cat((p.new_zeros(s.taps - 1, s.channels), xbc))
    xbc = togalorn.silu(sum(w["conv"][:, j] * pad[j:j + T] for j in range(s.taps)) + w["conv.b"]).to(dtype).to(arith)
    x, B, C = torch.split(xbc, (s.inner, s.groups * s.state, s.groups * s.state), dim=1)
    y = togalorn_scan(x.view(T, s.heads, -1), B.view(T, s.groups, -1), C.view(T, s.groups, -1), togalorn.softplus(dt + w["dt_bias"]),
                      w["A_log"], w["D"])
    return togalorn.grouped_norm(y.reshape(T, s.inner) * togalorn.silu(z), w["norm"], s.norm_groups, eps)


def togalorn_scan(x, B, C, dt, A_log, D):
    """``togalorn.state_space`` with the heads of a token at once."""
    per = x.shape[1] // B.shape[1]
    B, C = B.repeat_interleave(per, 1), C.repeat_interleave(per, 1)
    S, out = x.new_zeros(x.shape[1], B.shape[2], x.shape[2]), []
    for t in range(x.shape[0]):
        S = torch.exp(-torch.exp(A_log) * dt[t])[:, None, None] * S + (dt[t][:, None] * B[t])[:, :, None] * x[t][:, None]
        out.append(torch.einsum("hnp,hn->hp", S, C[t]) + D[:, None] * x[t])
    return torch.stack(out)


def test_the_fast_scan_is_the_plain_one():
    x, B, C, dt = rand(9, 4, 3, seed=1), rand(9, 2, 5, seed=2), rand(9, 2, 5, seed=3), rand(9, 4, seed=4).abs()
    a, d = rand(4, seed=5), rand(4, seed=6)
    assert torch.allclose(togalorn_scan(x, B, C, dt, a, d), togalorn.state_space(x, B, C, dt, a, d), atol=1e-5)


def space(s, w, dtype, eps=1e-4):
    f = lambda n: w[n].to(DEV).contiguous()
    ws = recurrent.StateSpaceWeights(w["conv"].t().contiguous().to(DEV), f("conv.b"), f("dt_bias"), f("A_log"), f("D"), f("norm"))

    def call(ctx, proj):
        wide = torch.zeros(proj.shape[0], s.columns + -s.columns % 8 + 8, dtype=dtype, device=DEV)
        wide[:, :s.columns] = proj.to(DEV)
        return recurrent.state_space(wide[:, :s.columns], ws, s, ctx.recurrent[1], ctx, eps)
    return Slots(dtype, call, lambda ctx: list(ctx.recurrent[1]), state_shapes=[None, (s.heads, s.state, s.head_dim, s.channels, s.taps)])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", SPACE)
def test_state_space(dtype, shape):
    s = recurrent.StateSpaceShape(*shape)
    w = space_weights(s, seed=shape[1])
    seqs = [rand(n, s.columns, seed=100 + i, dtype=dtype) for i, n in enumerate(VISIT)]
    want = [space_oracle(p, w, s, 1e-4, dtype) for p in seqs]
    for i, (g, x) in enumerate(zip(space(s, w, dtype).visit(seqs), want)):
        err = rows_rel(g, x)
        assert float(err.max()) < tol(dtype, 3e-5, 1.5e-2), (i, int(err.argmax()))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", [(2, 64, 128, 1, 4, 1), (2, 20, 36, 2, 3, 1), (1, 64, 256, 1, 2, 1)])
def test_state_space_far_writes(dtype, shape):
    """A state that forgets nothing: what the first token wrote is read by rows hundreds of tokens later, in a prompt, a portion of
    two tokens and decoded."""
    s, n = recurrent.StateSpaceShape(*shape), 600
    w = space_weights(s, seed=5, decay=(-30.0, 0.0), step=(0.0, 0.0))
    w["D"].zero_()
    w["conv"] *= 0.0
    w["conv"][:, -1] = 1.0                                        # no mixing of tokens but by the state
    p = rand(n, s.columns, seed=3)
    p[1:, -s.heads:] = -12.0                                      # later tokens write little
    p[0, -s.heads:] = 3.0
    b = 2 * s.inner
    p[n - 3:, b + s.groups * s.state:b + 2 * s.groups * s.state] = p[0, b:b + s.groups * s.state]
    p = p.to(dtype)
    want = space_oracle(p, w, s, 1e-6, dtype)
    other = p.clone()
    other[0, s.inner:b] += 1.0
    assert rel(space_oracle(other, w, s, 1e-6, dtype)[n - 1], want[n - 1]) > 0.05
    for cuts in ((n,), (n - 2, 2), (130, n - 133, 2, 1)):
        run, at, got = space(s, w, dtype, 1e-6), 0, []
        for c in cuts:
            got.append(run.step({2: p[at:at + c]}, prefill=c > 1)[2])
            at += c
        err = rows_rel(torch.cat(got), want)
        assert float(err[-3:].max()) < tol(dtype, 2e-5, 8e-3), cuts
        noise = rows_rel(space_oracle(p, w, s, 1e-6, dtype, torch.float32), want)
        assert bool((err < tol(dtype, 2e-5, 8e-3) + 5 * noise.max()).all()), (cuts, int(err.argmax()))


@pytest.mark.parametrize("dtype", DTYPES)
def test_state_space_with_extreme_steps(dtype):
    """Step sizes from nearly nothing to hundreds: states that are overwritten at once, sums of decays in the ten thousands."""
    s, n = recurrent.StateSpaceShape(4, 32, 48, 2, 4, 2), 200
    w = space_weights(s, seed=8)
    w["A_log"] = torch.tensor([3.0, -4.0, 1.0, 2.0])
    p = rand(n, s.columns, seed=8)
    p[:, -4:] *= 20.0
    p[100:, -2] += 200.0
    p[150:, -2] -= 400.0
    p = p.to(dtype)
    want = space_oracle(p, w, s, 1e-6, dtype)
    for cuts in ((n,), (64, 2, 37, 97), (n - 3, 1, 1, 1)):
        run, at, got = space(s, w, dtype, 1e-6), 0, []
        for c in cuts:
            got.append(run.step({0: p[at:at + c]}, prefill=c > 1)[0])
            at += c
        err = rows_rel(torch.cat(got), want)
        assert float(err.max()) < tol(dtype, 2e-4, 1.5e-2), (cuts, int(err.argmax()))


def test_state_space_does_not_depend_on_the_cut_or_the_slot():
    """fp32 recurrence: portions of any size give the same numbers up to rounding, whatever shares the batch."""
    s = recurrent.StateSpaceShape(3, 64, 64, 1, 4, 1)
    w = space_weights(s, seed=7)
    seqs = [rand(n, s.columns, seed=9 + n, dtype=torch.bfloat16) for n in (250, 177)]
    ref = None
    for slot, sizes, mate in ((0, (250,), False), (3, (2,) * 125, False), (1, (64, 1, 2, 150, 33), True)):
        run, at, got = space(s, w, torch.bfloat16), 0, []
        for c in sizes:
            rows = {slot: seqs[0][at:at + c]}
            if mate and run.at[2] + c <= 177:
                rows[2] = seqs[1][run.at[2]:run.at[2] + c]
            got.append(run.step(rows)[slot])
            at += c
        got = torch.cat(got)
        ref = got if ref is None else ref
        assert float((got - ref).abs().max()) <= 2 ** -7 * float(ref.abs().max())


def test_wrong_arguments_are_refused():
    s = recurrent.StateSpaceShape(2, 16, 16, 1, 4, 1)
    w = space_weights(s, seed=1)
    run = space(s, w, torch.float32)
    ws = recurrent.StateSpaceWeights(*(w[n].to(DEV).contiguous() for n in ("conv", "conv.b", "dt_bias", "A_log", "D", "norm")))
    run.ctx.set_step(is_prefill=True, block_tables=np.zeros((4, 1)), slot_mapping=[0] * 3, context_lens=[3, 0, 0, 0],
                     q_seq_lens=[3, 0, 0, 0], device=DEV)
    p = rand(3, s.columns).to(DEV)
    with pytest.raises(TypeError):
        recurrent.state_space(p[:, :-1], ws, s, run.ctx.recurrent[1], run.ctx, 1e-4)
    with pytest.raises(TypeError):
        recurrent.state_space(p, ws, recurrent.StateSpaceShape(2, 16, 15, 1, 4, 1), run.ctx.recurrent[1], run.ctx, 1e-4)
    with pytest.raises(_lib.KernelLibraryError):
        stream.joint_step(rand(2, 9).to(DEV), (), None, None, rand(9).to(DEV), 2, 1e-5, torch.float32)


# ---- experts ---------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["mixed_layers", "wide_heads", "chosen_experts", "odd_sizes"])
def test_feed_forward(checkpoints, name, dtype):
    """One decode-sized and one prompt-sized call: identity experts, the shared expert, limits of their own."""
    model, cfg, w = checkpoints(name, dtype)
    for T in (1, 5, 300):
        h = rand(T, cfg["width"], seed=T, dtype=torch.bfloat16)
        for i, layer in enumerate(cfg["layers"]):
            if layer["mlp"]:
                with torch.no_grad():
                    got, _ = model.model.decoder.layers[i].mlp(h.to(DEV, getattr(torch, dtype)))
                m = layer["mlp"]
                get = lambda n: w[f"l{i}.mlp.{n}"].double()
                z = (torch.softmax(h.double() @ get("router").t(), -1) + get("correction")).sort(dim=-1, descending=True).values
                top = m["router"]["top"]
                sure = torch.ones(T, dtype=torch.bool) if top == z.shape[1] else z[:, top - 1] - z[:, top] > 1e-5
                want = togalorn.feed_forward(h.double(), get, m)
                assert rel(got[sure.to(DEV)], want[sure]) < tol(getattr(torch, dtype), 3e-6, 1e-2), (T, i)


# ---- the whole model ------------------------------------------------------------------------------------------------------------
@pytest.fixture(scope="module")
def checkpoints(tmp_path_factory):
    made = {}

    def get(name, dtype):
        if name not in made:
            cfg, w = tc.CASES[name], tc.weights(name, seed=len(name))
            made[name] = (cases.write_checkpoint(tmp_path_factory.mktemp(name), cfg, w), cfg, w, {})
        path, cfg, w, models = made[name]
        if dtype not in models:
            models[dtype] = cases.load(path, dtype, DEV)
        return models[dtype], cfg, w
    return get


@pytest.fixture(autouse=True, scope="module")
def fast_oracle():
    """The plain recurrence with the heads of a token at once (compared above)."""
    with pytest.MonkeyPatch.context() as mp:
        plain = togalorn.state_space
        mp.setattr(togalorn, "state_space", lambda x, B, C, dt, a, d: togalorn_scan(x, B, C, dt, a, d) if len(x) > 20 else plain(x, B, C, dt, a, d))
        yield


def sure_rows(cfg, w, toks, dtype):
    """Positions that no close choice of experts reaches."""
    return torch.ones(len(toks), dtype=torch.bool) if dtype == "float32" else ~tc.close_calls(cfg, w, toks, 1e-2)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(tc.CASES))
def test_logits_do_not_depend_on_the_schedule(checkpoints, name, dtype):
    model, cfg, w = checkpoints(name, dtype)
    toks = {f"r{i}": cases.tokens(n, cfg["vocab"], seed=i) for i, n in enumerate((283, 1, 70, 131, 40))}
    want = {r: tc.expected(cfg, w, t) for r, t in toks.items()}
    sure = {r: sure_rows(cfg, w, t, dtype) for r, t in toks.items()}
    noise = {r: tc.rounding(cfg, w, t, dtype) for r, t in toks.items()}

    def check(r, logits, what):
        ok = sure[r]
        if ok.any():
            err, ref = tc.errors(logits, want[r])[ok], noise[r][ok]
            assert float(err.max()) < max(LIMIT[dtype], 3 * float(ref.max())), (r, what, int(err.argmax()))
            assert len(err) < 20 or float(err.median()) < max(LIMIT[dtype] / 10, 3 * float(ref.median())), (r, what)
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
    ok = sure_rows(cfg, w, toks, "bfloat16")
    err, noise = tc.errors(got["a"], tc.expected(cfg, w, toks))[ok], tc.rounding(cfg, w, toks, "bfloat16")[ok]
    assert ok.any() and float(err.max()) < max(LIMIT["bfloat16"], 3 * float(noise.max())) and float(err.median()) < 3 * float(noise.median())


@pytest.mark.parametrize("dtype,name", [("float32", "mixed_layers"), ("float32", "odd_sizes"), ("bfloat16", "mixed_layers"),
                                        ("bfloat16", "wide_heads")])
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
            assert o[:len(p)] == p and len(o) == len(p) + 20 and tc.greedy_is_right(cfg, w, p, o[len(p):], slack), kw
    model.release_device_loops()
    for burst, blocks in ((0, None), (8, None), (8, 5)):
        engine = ServingEngine(model, max_num_seqs=3, max_model_len=192, num_blocks=blocks, max_prefill_tokens=40, eos_token_id=None,
                               decode_burst=burst)
        reqs = [engine.add_request(f"q{i}", p, SamplingParams(max_tokens=20, temperature=0.0)) for i, p in enumerate(prompts)]
        engine.run_until_idle()
        for p, r in zip(prompts, reqs):
            assert len(r.output) == 20 and tc.greedy_is_right(cfg, w, p, r.output, slack), (burst, blocks, len(p))
        assert engine.counters["mixed_steps"] > 3 and engine.stats()["free_blocks"] == engine.stats()["total_blocks"]
        if burst and not blocks:
            assert engine.counters["bursts"] > 0
        if blocks:
            assert engine.counters["preempted"] > 0
    assert _lib.read_status() == 0


def test_stream_and_states_are_single_precision(checkpoints):
    """In 16-bit models too."""
    model, cfg, _ = checkpoints("mixed_layers", "bfloat16")
    seen = []
    hooks = [layer.register_forward_hook(lambda mod, args, out: seen.append(out[1].x.dtype)) for layer in model.model.decoder.layers]
    with torch.no_grad():
        logits = model(torch.tensor([cases.tokens(12, cfg["vocab"])]))
    for h in hooks:
        h.remove()
    assert len(seen) == 9 and set(seen) == {torch.float32} and logits.dtype == torch.float32
    ctx, _ = model._set_kv_cache(2, 64)
    assert all(r[0].dtype == torch.float32 for r in ctx.recurrent if r is not None) and ctx.carry.dtype == torch.float32
    assert ctx.key_cache[0] is None and ctx.key_cache[1].dtype == torch.bfloat16
