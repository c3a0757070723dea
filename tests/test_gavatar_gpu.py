"""Gavatar on the CUDA kernels, against the plain implementation of ``oracles/gavatar.py``: every kernel alone, whole prompts,
portions, decoding, mixed batches with pages and slots used again, generation through the engine."""
import numpy as np
import pytest
import torch

from mindformers_b200.inference import ragged_attention as ragged
from mindformers_b200.inference.paged_attention import KVCacheContext
from mindformers_b200.inference.ragged_attention import latent_attention, ragged_attention, talking_attention
from mindformers_b200.ops import _lib, recurrent, stream
from mindformers_b200.ops import functional as Fn
from mindformers_b200.serving import SamplingParams, ServingEngine
from mindformers_b200.serving.trace import build_engine

from oracles import cases, gavatar
from oracles import gavatar_cases as gc
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


def rows_rel(got, want):
    return (got.double().cpu() - want.double()).norm(dim=1) / want.double().norm(dim=1)


def tol(dtype, f32=3e-6, bf16=6e-3):
    return f32 if dtype == torch.float32 else bf16


# ---- embedding and stream ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("W", [8, 101, 1024])
def test_embedding(dtype, W):
    table, ids, pos = rand(50, W, dtype=dtype), torch.tensor([3, 49, 0, 3, 7]), torch.tensor([0, 1, 513, 9999, 131071])
    want = table[ids].double() * 11.3 + gavatar.position_vectors(131072, 8, torch.float64)[pos] if W == 8 else None
    if want is None:
        want = table[ids].double() * 11.3 + torch.stack([gavatar_position(int(p), W) for p in pos])
    got = stream.embed(ids.to(DEV), table.to(DEV), 11.3, pos.to(DEV), stream.sinusoidal_frequencies(W).to(DEV))
    assert got.dtype == torch.float32 and float((got.double().cpu() - want).abs().max()) < 1e-5
    plain = stream.embed(ids.to(DEV), table.to(DEV), 0.5, pos.to(DEV), None)
    assert torch.equal(plain.cpu(), table[ids].float() * 0.5)


def gavatar_position(p, W):
    c = torch.arange(W)
    angle = p * 10000.0 ** (-2.0 * (c // 2).double() / W)
    return torch.where(c % 2 == 1, torch.cos(angle), torch.sin(angle))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,W", [(1, 8), (3, 101), (5, 192), (2, 4096), (4, 1150), (2, 6152), (2, 9000)])
def test_normed_step(dtype, T, W):
    x, y = rand(T, W, seed=1), rand(T, W + 8, seed=2, dtype=dtype)
    w_in, w_out, step = (rand(W, seed=s, dtype=dtype, scale=0.3) for s in (3, 4, 5))
    d = lambda t: t.to(DEV)
    x2 = x.double() + gavatar.norm(y[:, :W].double(), w_in.double(), 1e-3)
    for st, keep, one in ((step, True, True), (None, True, True), (None, False, True), (step, True, False)):
        shift = 0.0 if one else -1.0
        x2 = x.double() + gavatar.norm(y[:, :W].double(), w_in.double() + shift, 1e-3) + (0 if st is None else st.double())
        xd = d(x)
        h, new = stream.normed_step(xd, d(y)[:, :W], d(w_in), None if st is None else d(st), d(w_out), 1e-3, one, keep=keep)
        assert h.dtype == dtype and rel(h, gavatar.norm(x2, w_out.double() + shift, 1e-3)) < tol(dtype, 2e-6)
        assert torch.equal(xd.cpu(), x) and (new is None if not keep else rel(new, x2) < 2e-6)
    h, new = stream.normed_step(xd, None, None, None, d(w_out), 1e-3, True)
    assert new is xd and rel(h, gavatar.norm(x.double(), w_out.double(), 1e-3)) < tol(dtype, 2e-6)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("W,scale", [(96, 1), (101, 1), (2048, 1), (64, 600)])
def test_token_shift(dtype, W, scale):
    """Unequal sequences in portions down to one row, idle slots, decoded rows, a slot taken over; with ``scale`` portions long
    enough for CTAs of several rows."""
    w, mu = rand(W, seed=1, dtype=dtype, scale=0.3), rand(W, seed=2, dtype=dtype)
    lens = [n * scale for n in (20, 9, 13)]
    xs = [rand(n, W, seed=10 + i) for i, n in enumerate(lens)]
    want = [gavatar.token_shift(gavatar.norm(x.double(), w.double(), 1e-5), mu.double()) for x in xs]
    ctx = KVCacheContext(2, 1, 64, 0, 0, dtype, DEV, layer_shapes=[None] * 2, slots=4, carry_width=W)
    ctx.carry.normal_(0, 9)
    at, got = [0, 0, 0], [[], [], []]

    def go(plan, prefill=True):
        """``plan``: {sequence: rows}; sequence 2 has slot 3."""
        slot = {3 if i == 2 else i: i for i in plan}
        n = [plan[slot[s]] if s in slot else 0 for s in range(4)]
        lens_ = [at[slot[s]] + n[s] if s in slot else 5 for s in range(4)]
        rows = [xs[slot[s]][at[slot[s]]:at[slot[s]] + n[s]] if s in slot else torch.full((0 if prefill else 1, W), 3.0) for s in range(4)]
        ctx.set_step(is_prefill=prefill, block_tables=np.zeros((4, 1)), slot_mapping=[0] * sum(n) if prefill else [0 if c else -1 for c in n],
                     context_lens=lens_, q_seq_lens=n if prefill else [1] * 4, device=DEV)
        kept = ctx.carry.clone()
        h, _ = stream.normed_step(torch.cat(rows).to(DEV), None, None, None, w.to(DEV), 1e-5, True, stream.Carry(mu.to(DEV), ctx, 1))
        idle = [s for s in range(4) if not n[s]]
        assert torch.equal(ctx.carry[1, idle], kept[1, idle]) and torch.equal(ctx.carry[0], kept[0])
        pos = 0
        for s in range(4):
            if n[s]:
                got[slot[s]].append(h[pos:pos + n[s]].float().cpu())
                at[slot[s]] += n[s]
            pos += rows[s].shape[0]
    go({0: 7 * scale, 1: 1})
    go({0: 2, 2: 5 * scale, 1: 4 * scale})
    go({0: 1, 2: 1}, prefill=False)
    go({1: 2, 2: 1})
    go({0: 1, 1: 1, 2: 1}, prefill=False)
    go({i: lens[i] - at[i] for i in range(3)})
    for i in range(3):
        assert float(rows_rel(torch.cat(got[i]), want[i]).max()) < tol(dtype, 3e-6), i


# ---- around the attention -------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,DV", [(4, 2, 64, 64), (8, 2, 128, 128), (6, 3, 48, 24), (3, 1, 20, 36), (2, 1, 7, 5), (2, 2, 32, 300)])
def test_unit_norms_and_cache_write(dtype, H, G, D, DV):
    T, n = 5, H * D + G * (D + DV)
    x, bias = rand(T, n + 8, seed=1, dtype=dtype), rand(n, seed=2, dtype=dtype)
    kc, vc = torch.zeros(8, 1, G, D, dtype=dtype, device=DEV), torch.zeros(8, 1, G, DV, dtype=dtype, device=DEV)
    slots = torch.tensor([3, -1, 0, 7, 2], dtype=torch.int32, device=DEV)
    none = torch.zeros(0, device=DEV)
    q = stream.qkv_rope_cache(x.to(DEV)[:, :n], bias.to(DEV), None, None, 1e-3, none, 1.0, False, torch.arange(T, device=DEV), slots,
                              kc, vc, H, G, D, DV, True, True)
    y = x[:, :n].double() + bias.double()
    want = [gavatar.rms(p.reshape(T, -1, s), 1e-3) for p, s in zip(torch.split(y, (H * D, G * D, G * DV), dim=1), (D, D, DV))]
    assert rel(q, want[0]) < tol(dtype)
    keep = torch.tensor([0, 2, 3, 4])
    at = slots.cpu()[keep].long()
    assert rel(kc[at.to(DEV), 0], want[1][keep]) < tol(dtype) and rel(vc[at.to(DEV), 0], want[2][keep]) < tol(dtype)
    assert float(kc[[1, 4, 5, 6]].abs().max()) == 0 and float(vc[[1, 4, 5, 6]].abs().max()) == 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("Q,R,more", [(64, 128, 9), (33, 7, 9), (1536, 512, 8), (264, 72, 16), (8, 2048, 0), (2056, 8, 0)])
def test_latent_norm_and_cache_write(dtype, Q, R, more):
    T = 4
    x, qn, kn = rand(T, Q + R + more, seed=1, dtype=dtype), rand(Q, seed=2, dtype=dtype) + 1, rand(R, seed=3, dtype=dtype) + 1
    cache = torch.zeros(6, 1, 1, R, dtype=dtype, device=DEV)
    slots = torch.tensor([5, 0, -1, 2], dtype=torch.int32, device=DEV)
    q = stream.latent_norm_cache(x.to(DEV)[:, :Q + R], qn.to(DEV), kn.to(DEV), 1e-3, slots, cache)
    xd = x.double()
    assert rel(q, gavatar.rms(xd[:, :Q], 1e-3) * qn.double()) < tol(dtype)
    c = gavatar.rms(xd[:, Q:Q + R], 1e-3) * kn.double()
    assert rel(cache[[5, 0, 2], 0, 0], c[[0, 1, 3]]) < tol(dtype) and float(cache[[1, 3, 4]].abs().max()) == 0


@pytest.mark.parametrize("dtype", DTYPES)
def test_output_gates(dtype):
    for T, n, m in ((3, 96, 96), (5, 96, 8), (4, 33, 11), (700, 512, 4), (9, 96, 6), (3, 64, 32)):
        x, g = rand(T, n + 8, seed=1, dtype=dtype), rand(T, m + 3, seed=2, dtype=dtype)
        wide = x.to(DEV)
        got = stream.gate_heads_(wide[:, :n], g.to(DEV)[:, :m])
        want = x[:, :n].double() * torch.sigmoid(g[:, :m].double()).repeat_interleave(n // m, 1)
        assert got.data_ptr() == wide.data_ptr() and rel(got, want) < tol(dtype) and torch.equal(wide[:, n:].cpu(), x[:, n:])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,DV", [(4, 2, 64), (32, 8, 128), (5, 1, 7), (20, 1, 40), (3, 3, 12), (1, 1, 5)])
def test_mixed_heads(dtype, H, G, DV):
    T = 7
    o, talk, gate = rand(T, H, G, DV, seed=1, dtype=dtype), rand(H, H, seed=2), rand(T, H * DV + 8, seed=3, dtype=dtype)
    own = torch.arange(H) // (H // G)
    want = torch.einsum("hg,tghv->thv", talk.double(), o.double()[:, :, own]).reshape(T, H * DV)
    assert rel(stream.talk_mix(o.to(DEV), talk.to(DEV), None), want) < tol(dtype)
    want = want * torch.sigmoid(gate[:, :H * DV].double())
    assert rel(stream.talk_mix(o.to(DEV), talk.to(DEV), gate.to(DEV)[:, :H * DV]), want) < tol(dtype)


# ---- sliding-window attention ----------------------------------------------------------------------------------------------
SHAPES = [(4, 2, 64, 64), (8, 2, 128, 128), (6, 2, 40, 24), (6, 3, 48, 96), (20, 1, 24, 40), (3, 1, 20, 36), (2, 1, 144, 12)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,DV", SHAPES)
@pytest.mark.parametrize("window,persistent", [(1, 0), (100, 1000), (128, 0), (129, 0), (5000, 1000)])
@pytest.mark.parametrize("all_values", [False, True])
def test_windowed_attention(dtype, H, G, D, DV, window, persistent, all_values, monkeypatch):
    """Portions and decoded rows of unequal sequences, with a sink, or with every head's weights on every head's values."""
    monkeypatch.setattr(ragged, "_PERSISTENT_UP_TO", persistent)
    kw = dict(window=window, all_values=all_values)
    for lens, news, bs, ragged_step in (([1, 300, 129, 517, 64, 130, 40], [1, 300, 2, 260, 1, 1, 0], 64, True),
                                        ([1, 63, 64, 129, 700], [1] * 5, 16, False)):
        ctx, table, qs, sink, scale, want = attention_case(dtype, H, G, D, DV, bs, 0, lens, news, seed=D, **kw)
        ctx.set_step(is_prefill=ragged_step, block_tables=table, slot_mapping=[0] * sum(news), context_lens=lens, q_seq_lens=news,
                     device=DEV)
        got = ragged_attention(torch.cat(qs).to(DEV), ctx, 0, scale, sink=None if all_values else sink.to(DEV), **kw)
        err = rows_rel(got, want)
        assert float(err.max()) < tol(dtype, 2e-5, 3e-2), (ragged_step, int(err.argmax()))
    assert _lib.read_status() == 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,DV", [(8, 2, 128, 128), (3, 1, 20, 36)])
@pytest.mark.parametrize("window", [64, 130])
def test_windowed_attention_at_the_edges(dtype, H, G, D, DV, window):
    """One key that stands out: the last that a row sees, the first that it does not, at page and tile borders; in a prompt, in a
    portion of two rows and decoded."""
    n, bs = 400, 16
    for qp in (399, 383, 300, 256 + window - 1, 128 + window, window, window - 1, 5):
        for kp in (qp - window + 1, qp - window, qp - window + 2, qp, qp + 1):
            for lens, news in ((n, n), (max(qp + 2, kp + 1), 2), (qp + 1, 1)):
                if lens > n or kp < 0 or kp >= lens:
                    continue
                ctx, table, qs, sink, scale, want = attention_case(dtype, H, G, D, DV, bs, 0, [lens], [news], seed=qp + kp,
                                                                   spots=[(0, qp, kp)], window=window)
                ctx.set_step(is_prefill=news > 1, block_tables=table, slot_mapping=[0] * news, context_lens=[lens], q_seq_lens=[news],
                             device=DEV)
                got = ragged_attention(qs[0].to(DEV), ctx, 0, scale, sink=sink.to(DEV), window=window)
                row = qp - (lens - news)
                err = (got[row].double().cpu() - want[row]).norm() / want[row].norm()
                assert float(err) < tol(dtype, 2e-5, 3e-2), (qp, kp, lens, news)
    assert _lib.read_status() == 0


TALK = [(4, 2, 64, 64), (32, 8, 128, 128), (6, 2, 40, 24), (6, 3, 48, 96), (20, 1, 24, 40), (34, 2, 16, 72), (3, 1, 20, 36),
        (1, 1, 8, 8), (64, 4, 32, 64), (16, 16, 64, 32), (40, 5, 128, 128), (2, 1, 144, 12)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,DV", TALK)
@pytest.mark.parametrize("window", [1, 100, 128, 5000])
def test_mixed_weights(dtype, H, G, D, DV, window):
    """Portions and decoded rows; a gate that lies in a wider matrix."""
    talk, own = rand(H, H, seed=5) * H ** -0.5 + torch.eye(H), torch.arange(H) // (H // G)
    for lens, news, bs, ragged_step in (([1, 300, 129, 257, 64, 700, 40], [1, 300, 2, 130, 1, 1, 0], 64, True),
                                        ([70, 3], [1, 1], 64, True), ([1, 63, 64, 129, 900], [1] * 5, 16, False)):
        ctx, table, qs, _, scale, o = attention_case(dtype, H, G, D, DV, bs, 0, lens, news, seed=D, window=window, all_values=True,
                                                     score_scale=4.0)
        T = sum(news)
        gate = rand(T, H * DV + 8, seed=6, dtype=dtype)
        want = torch.einsum("hg,tghv->thv", talk.double(), o.view(T, H, G, DV)[:, :, own]).reshape(T, H * DV)
        want = want * torch.sigmoid(gate[:, :H * DV].double())
        ctx.set_step(is_prefill=ragged_step, block_tables=table, slot_mapping=[0] * T, context_lens=lens, q_seq_lens=news, device=DEV)
        got = talking_attention(torch.cat(qs).to(DEV), ctx, 0, scale, talk.to(DEV), gate.to(DEV)[:, :H * DV], window)
        err = rows_rel(got, want)
        assert float(err.max()) < tol(dtype, 2e-5, 3e-2), (ragged_step, lens, int(err.argmax()))
    assert _lib.read_status() == 0


@pytest.mark.parametrize("H,G,D,DV", [(8, 2, 128, 128), (6, 3, 48, 24)])
@pytest.mark.parametrize("window", [64, 130])
def test_mixed_weights_at_the_edges(H, G, D, DV, window):
    """One key that stands out, just inside and just outside the window, decoded and in portions."""
    talk, own = rand(H, H, seed=5) * H ** -0.5 + torch.eye(H), torch.arange(H) // (H // G)
    for qp in (399, 383, 300, 128 + window, window, window - 1):
        for kp in (qp - window + 1, qp - window, qp):
            for lens, news in ((400, 400), (qp + 1, 2), (qp + 1, 1)):
                if kp < 0 or kp >= lens:
                    continue
                ctx, table, qs, _, scale, o = attention_case(torch.bfloat16, H, G, D, DV, 16, 0, [lens], [news], seed=qp + kp,
                                                             spots=[(0, qp, kp)], window=window, all_values=True)
                want = torch.einsum("hg,tghv->thv", talk.double(), o.view(news, H, G, DV)[:, :, own]).reshape(news, H * DV)
                ctx.set_step(is_prefill=news > 1, block_tables=table, slot_mapping=[0] * news, context_lens=[lens], q_seq_lens=[news],
                             device=DEV)
                got = talking_attention(qs[0].to(DEV), ctx, 0, scale, talk.to(DEV), None, window)
                row = qp - (lens - news)
                err = (got[row].double().cpu() - want[row]).norm() / want[row].norm()
                assert float(err) < 3e-2, (qp, kp, lens, news)
    assert _lib.read_status() == 0


# ---- latent attention --------------------------------------------------------------------------------------------------------
def latent_case(dtype, H, D, DV, R, bs, lens, news, window, seed=0, spots=()):
    """A paged cache of latents on shuffled pages, queries, factors, and the expected result. ``spots``: (sequence, query
    position, key position) whose score stands out: the key's latent is made the one that the query likes."""
    g = torch.Generator().manual_seed(seed)
    per = [-(-n // bs) for n in lens]
    total = sum(per) + 3
    perm = torch.randperm(total, generator=g).tolist()
    ctx = KVCacheContext(1, total, bs, 0, 0, dtype, DEV, layer_shapes=[(1, R, 0)])
    ctx.key_cache[0].copy_((torch.randn(ctx.key_cache[0].shape, generator=g) * 5).to(dtype))         # other requests' old rows
    table = torch.full((len(lens), max(per) + 2), -1, dtype=torch.int32)
    w = (torch.randn(H * (D + DV), R, generator=g) * R ** -0.5).to(dtype)
    wd = w.double()
    w_uk, w_uv = wd[:H * D].view(H, D, R), wd[H * D:].view(H, DV, R)
    scale, sink = 1.2 * D ** -0.5, torch.randn(H, generator=g) + 1
    qs, want = [], []
    for b in range(len(lens)):
        for i in range(per[b]):
            table[b, i] = perm.pop()
        c = torch.randn(lens[b], R, generator=g)
        q = torch.randn(news[b], H, D, generator=g)
        for sb, qp, kp in spots:
            if sb == b:
                like = torch.einsum("hd,hdr->r", q[qp - (lens[b] - news[b])].double(), w_uk)
                c[kp] = (like / like.norm() * R ** 0.5 * 5).float()
        c, q = c.to(dtype), q.to(dtype)
        for t in range(lens[b]):
            ctx.key_cache[0][int(table[b, t // bs]), t % bs, 0] = c[t].to(DEV)
        n, m = lens[b], news[b]
        cd = c.double()
        k, v = torch.einsum("tr,hdr->thd", cd, w_uk), torch.einsum("tr,hvr->thv", cd, w_uv)
        s = torch.einsum("qhd,khd->hqk", q.double(), k) * scale
        mask = gavatar.window_mask(n, window)[n - m:]
        p = torch.stack([gavatar.softmax(s[h], mask, sink[h].double()) for h in range(H)])
        want.append(torch.einsum("hqk,khv->qhv", p, v).reshape(m, H * DV))
        qs.append(q)
    return ctx, table, torch.cat(qs), w.to(DEV), scale, sink.to(DEV), torch.cat(want)


LATENT = [(4, 64, 64, 128), (8, 128, 128, 512), (20, 24, 40, 200), (3, 13, 11, 29), (16, 32, 96, 64), (2, 96, 32, 72), (33, 16, 8, 320)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,D,DV,R", LATENT)
@pytest.mark.parametrize("window", [1, 90, 128, 5000])
def test_latent_attention(dtype, H, D, DV, R, window):
    """Expanded portions, absorbed rows and both in one batch."""
    for lens, news, bs, ragged_step in (([1, 300, 129, 517, 64, 130, 40], [1, 300, 2, 260, 1, 1, 0], 64, True),
                                        ([70, 3], [1, 1], 64, True), ([200], [90], 16, True), ([1, 63, 64, 129, 700], [1] * 5, 16, False)):
        ctx, table, q, w, scale, sink, want = latent_case(dtype, H, D, DV, R, bs, lens, news, window, seed=R)
        ctx.set_step(is_prefill=ragged_step, block_tables=table, slot_mapping=[0] * sum(news), context_lens=lens, q_seq_lens=news,
                     device=DEV)
        got = latent_attention(q.to(DEV), ctx, 0, w, DV, scale, window, sink)
        err = rows_rel(got, want)
        assert float(err.max()) < tol(dtype, 2e-5, 4e-2), (ragged_step, lens, int(err.argmax()))
        assert float(err.median()) < tol(dtype, 1e-5, 1e-2), (ragged_step, lens)
    assert _lib.read_status() == 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,D,DV,R", [(8, 128, 128, 512), (3, 13, 11, 29)])
@pytest.mark.parametrize("window", [64, 130])
def test_latent_attention_at_the_edges(dtype, H, D, DV, R, window):
    n, bs = 400, 16
    for qp in (399, 300, 128 + window, window, window - 1):
        for kp in (qp - window + 1, qp - window, qp, qp + 1):
            for lens, news in ((n, n), (max(qp + 2, kp + 1), 2), (qp + 1, 1)):
                if lens > n or kp < 0 or kp >= lens:
                    continue
                ctx, table, q, w, scale, sink, want = latent_case(dtype, H, D, DV, R, bs, [lens], [news], window, seed=qp + kp,
                                                                  spots=[(0, qp, kp)])
                ctx.set_step(is_prefill=news > 1, block_tables=table, slot_mapping=[0] * news, context_lens=[lens], q_seq_lens=[news],
                             device=DEV)
                got = latent_attention(q.to(DEV), ctx, 0, w, DV, scale, window, sink)
                row = qp - (lens - news)
                err = (got[row].double().cpu() - want[row]).norm() / want[row].norm()
                assert float(err) < tol(dtype, 2e-5, 4e-2), (qp, kp, lens, news)
    assert _lib.read_status() == 0


# ---- matrix memory --------------------------------------------------------------------------------------------------------------
MEMORY = [(4, 32, 32), (3, 64, 40), (2, 128, 128), (2, 128, 256), (3, 20, 36), (2, 7, 5), (2, 256, 512), (1, 160, 72), (1, 300, 40),
          (5, 48, 96), (34, 16, 16), (2, 96, 200), (1, 512, 64)]


def memory_weights(H, D, DV, seed, gates=((-0.5, 1.0), (3.0, 1.0))):
    bi, bf = (mean + std * rand(H, seed=seed + i) for i, (mean, std) in enumerate(gates))
    return bi, bf, 1 + 0.2 * rand(H * DV, seed=seed + 2)


def memory_oracle(proj, w, H, D, DV, cap, eps, dtype=torch.float64):
    """Read-out of one whole sequence."""
    bi, bf, norm = (t.to(dtype) for t in w)
    T = proj.shape[0]
    q, k, v, z, i, f = torch.split(proj.to(dtype), (H * D, H * D, H * DV, H * DV, H, H), dim=1)
    i, f = gavatar.soft_cap(i + bi, cap), gavatar.log_sigmoid(gavatar.soft_cap(f + bf, cap))
    o = gavatar.matrix_memory(q.view(T, H, D) * D ** -0.5, k.view(T, H, D), v.view(T, H, DV), i, f)
    return gavatar.rms(o, eps).reshape(T, H * DV) * norm * torch.sigmoid(z)


def memory_rows(n, H, D, DV, dtype, seed):
    """A projection whose keys resemble the queries, so that read-outs do not nearly cancel."""
    p = rand(n, 2 * H * (D + DV) + 2 * H, seed=seed)
    p[:, H * D:2 * H * D] = 0.7 * p[:, :H * D] + 0.5 * p[:, H * D:2 * H * D]
    return p.to(dtype)


class Slots:
    """Sequences on state slots that are full of old values, fed in portions of a common projection matrix."""

    def __init__(self, H, D, DV, cap, w, dtype, slots=4, eps=1e-4):
        self.s, self.w, self.eps, self.n, self.dtype = recurrent.MemoryShape(H, D, DV, cap), w, eps, slots, dtype
        self.ctx = KVCacheContext(1, 1, 64, 0, 0, dtype, DEV, layer_shapes=[None], slots=slots, state_shapes=[[(H, D, DV), (H, D), (H,)]])
        for t in self.ctx.recurrent[0]:
            t.normal_(0, 9)
        self.at = [0] * slots

    def step(self, rows, prefill=True):
        """``rows``: {slot: projection of its next rows}; returns {slot: read-out}."""
        n = [len(rows[i]) if i in rows else 0 for i in range(self.n)]
        lens = [self.at[i] + n[i] if prefill or n[i] else 5 for i in range(self.n)]
        width = next(iter(rows.values())).shape[1]
        if not prefill:                       # every slot has a row; idle ones hold garbage
            rows = {i: rows.get(i, torch.full((1, width), 3.0, dtype=self.dtype)) for i in range(self.n)}
        proj = torch.cat([rows[i] for i in sorted(rows)])
        wide = torch.zeros(proj.shape[0], width + 8, dtype=self.dtype, device=DEV)
        wide[:, :width] = proj.to(DEV)
        self.ctx.set_step(is_prefill=prefill, block_tables=np.zeros((self.n, 1)),
                          slot_mapping=[0] * sum(n) if prefill else [0 if c else -1 for c in n], context_lens=lens,
                          q_seq_lens=n if prefill else [1] * self.n, device=DEV)
        idle = [i for i in range(self.n) if not n[i]]
        kept = [t[idle].clone() for t in self.ctx.recurrent[0]]
        out = recurrent.matrix_memory(wide[:, :width], *(t.to(DEV).contiguous() for t in self.w), self.s, self.ctx.recurrent[0], self.ctx,
                                      self.eps)
        assert all(torch.equal(t[idle], k) for t, k in zip(self.ctx.recurrent[0], kept))
        assert torch.isfinite(out).all()
        got, at = {}, 0
        for i in sorted(rows):
            m = len(rows[i])
            if n[i]:
                got[i] = out[at:at + m].float().cpu()
            at += m
        self.at = [self.at[i] + n[i] for i in range(self.n)]
        return got


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,D,DV", MEMORY)
def test_matrix_memory(dtype, H, D, DV):
    """Unequal sequences in portions down to one row, idle slots, decoded rows, slots taken over by new sequences."""
    w, cap = memory_weights(H, D, DV, seed=D), 6.0
    seqs = [memory_rows(n, H, D, DV, dtype, seed=100 + DV + i) for i, n in enumerate((270, 9, 141, 30))]
    want = [memory_oracle(p, w, H, D, DV, cap, 1e-4) for p in seqs]
    run = Slots(H, D, DV, cap, w, dtype)
    got, at = [[] for _ in seqs], [0] * 4

    def go(plan, prefill=True, slot=lambda i: i):
        rows = {slot(i): seqs[i][at[i]:at[i] + c] for i, c in plan.items()}
        for k, v in run.step(rows, prefill).items():
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
    run.at[1] = 0
    one = lambda i: {3: 1}.get(i, i)
    go({3: 1}, prefill=False, slot=one)
    go({3: 1}, prefill=False, slot=one)
    go({3: 28}, slot=one)
    assert at == [270, 9, 141, 30]
    for i in range(4):
        err = rows_rel(torch.cat(got[i]), want[i])
        assert float(err.max()) < tol(dtype, 3e-5, 8e-3), (i, int(err.argmax()))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("D,DV", [(128, 128), (20, 36), (256, 64)])
def test_matrix_memory_far_writes(dtype, D, DV):
    """A memory that forgets nothing: what the first token wrote is read by rows hundreds of tokens later with its own key, in a
    prompt, a portion of two tokens and decoded."""
    n, H, cap = 600, 2, 40.0
    w = memory_weights(H, D, DV, seed=5, gates=((0.0, 0.1), (39.0, 0.0)))
    p = memory_rows(n, H, D, DV, dtype, seed=3)
    gi = 2 * H * (D + DV)
    p[:, gi + H:] = 0
    p[1:, gi:gi + H] -= 7.0                                      # later tokens write little
    for t in (n - 3, n - 2, n - 1):
        p[t, :H * D] = p[0, H * D:2 * H * D]
    want = memory_oracle(p, w, H, D, DV, cap, 1e-4)
    other = p.clone()
    other[0, 2 * H * D:2 * H * D + H * DV] += 1.0
    assert rel(memory_oracle(other, w, H, D, DV, cap, 1e-4)[n - 1], want[n - 1]) > 0.05
    for cuts in ((n,), (n - 2, 2), (130, n - 133, 2, 1)):
        run, at, got = Slots(H, D, DV, cap, w, dtype), 0, []
        for c in cuts:
            got.append(run.step({2: p[at:at + c]}, prefill=c > 1)[2])
            at += c
        # rows whose read-out nearly cancels differ by what 32-bit arithmetic alone does there
        err, noise = rows_rel(torch.cat(got), want), rows_rel(memory_oracle(p, w, H, D, DV, cap, 1e-4, torch.float32), want)
        assert bool((err < tol(dtype, 1e-5, 8e-3) + 5 * noise.max()).all()), (cuts, int(err.argmax()))
        assert float(err[-3:].max()) < tol(dtype, 1e-5, 8e-3), cuts


@pytest.mark.parametrize("dtype", DTYPES)
def test_matrix_memory_with_extreme_gates(dtype):
    """Gates at their caps in both directions: memories that are overwritten at once, closed input gates, a running maximum
    that rises and falls by tens, and a read-out that only the floor of the normaliser divides."""
    n, H, D, DV, cap = 200, 4, 32, 48, 30.0
    w = (torch.tensor([0.0, 25.0, -25.0, 0.0]), torch.tensor([0.0, -25.0, 25.0, 3.0]), torch.ones(H * DV))
    p = memory_rows(n, H, D, DV, dtype, seed=8).float()
    gi = 2 * H * (D + DV)
    p[:, gi:] *= 12.0
    p[100:, gi + 3] += 60.0
    p[150:, gi + 3] -= 120.0
    p[50:60, :2 * H * D] *= 1e-3
    p = p.to(dtype)
    want = memory_oracle(p, w, H, D, DV, cap, 1e-6)
    for cuts in ((n,), (64, 2, 37, 97), (n - 3, 1, 1, 1)):
        run, at, got = Slots(H, D, DV, cap, w, dtype, eps=1e-6), 0, []
        for c in cuts:
            got.append(run.step({0: p[at:at + c]}, prefill=c > 1)[0])
            at += c
        got = torch.cat(got).double().view(n, H, DV)
        err = (got - want.view(n, H, DV)).norm(dim=2) / want.view(n, H, DV).norm(dim=2)
        assert float(err.max()) < tol(dtype, 2e-4, 1.5e-2), (cuts, divmod(int(err.argmax()), H))


def test_matrix_memory_does_not_depend_on_the_cut_or_the_slot():
    """fp32 recurrence: portions of any size give the same numbers up to rounding, whatever shares the batch."""
    H, D, DV = 3, 64, 64
    w = memory_weights(H, D, DV, seed=7)
    seqs = [memory_rows(n, H, D, DV, torch.bfloat16, seed=9 + n) for n in (250, 177)]
    ref = None
    for slot, sizes, mate in ((0, (250,), False), (3, (2,) * 125, False), (1, (64, 1, 2, 150, 33), True)):
        run, at, got = Slots(H, D, DV, 6.0, w, torch.bfloat16), 0, []
        for c in sizes:
            rows = {slot: seqs[0][at:at + c]}
            if mate and run.at[2] + c <= 177:
                rows[2] = seqs[1][run.at[2]:run.at[2] + c]
            got.append(run.step(rows)[slot])
            at += c
        got = torch.cat(got)
        ref = got if ref is None else ref
        assert float((got - ref).abs().max()) <= 2 ** -7 * float(ref.abs().max())


def test_matrix_memory_refuses_wrong_arguments():
    w = memory_weights(2, 16, 16, seed=1)
    run = Slots(2, 16, 16, 6.0, w, torch.float32)
    p = memory_rows(3, 2, 16, 16, torch.float32, seed=1).to(DEV)
    run.ctx.set_step(is_prefill=True, block_tables=np.zeros((4, 1)), slot_mapping=[0] * 3, context_lens=[3, 0, 0, 0],
                     q_seq_lens=[3, 0, 0, 0], device=DEV)
    args = [t.to(DEV) for t in w]
    with pytest.raises(TypeError):
        recurrent.matrix_memory(p[:, :-1], *args, run.s, run.ctx.recurrent[0], run.ctx, 1e-4)
    with pytest.raises(TypeError):
        recurrent.matrix_memory(p, *args, recurrent.MemoryShape(2, 16, 15, 6.0), run.ctx.recurrent[0], run.ctx, 1e-4)


# ---- experts ---------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("R,F", [(128, 64), (300, 50), (640, 200)])
def test_swiglu_of_any_size(dtype, R, F):
    x = rand(R, 2 * F, seed=1, dtype=dtype, scale=2.0)
    g, u = x.double().chunk(2, dim=1)
    assert rel(Fn.clamped_glu(x.to(DEV), float("inf"), 1.0, shift=0.0), gavatar.silu(g) * u) < tol(dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["mixed_layers", "chosen_experts", "odd_sizes"])
def test_feed_forward(checkpoints, name, dtype):
    """One decode-sized and one prompt-sized call; the router's bias decides and weighs."""
    model, cfg, w = checkpoints(name, dtype)
    for T in (1, 5, 300):
        h = rand(T, cfg["width"], seed=T, dtype=torch.bfloat16)
        for i, layer in enumerate(cfg["layers"]):
            if layer["mlp"]:
                with torch.no_grad():
                    got, _ = model.model.decoder.layers[i].mlp(h.to(DEV, getattr(torch, dtype)))
                m = layer["mlp"]
                get = lambda n: w[f"l{i}.mlp.{n}"].double()
                z = (h.double() @ get("router").t() + get("router.b")).sort(dim=-1, descending=True).values
                top = m["router"]["top"]
                sure = torch.ones(T, dtype=torch.bool) if top == m["router"]["experts"] else z[:, top - 1] - z[:, top] > 1e-4
                want = gavatar.feed_forward(h.double(), get, m)
                assert rel(got[sure.to(DEV)], want[sure]) < tol(getattr(torch, dtype), 3e-6, 1e-2), (T, i)


# ---- the whole model ------------------------------------------------------------------------------------------------------------
@pytest.fixture(scope="module")
def checkpoints(tmp_path_factory):
    made = {}

    def get(name, dtype):
        if name not in made:
            cfg, w = gc.CASES[name], gc.weights(name, seed=len(name))
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
    return ~gc.close_calls(cfg, w, toks, 0.02)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(gc.CASES))
def test_logits_do_not_depend_on_the_schedule(checkpoints, name, dtype):
    model, cfg, w = checkpoints(name, dtype)
    toks = {f"r{i}": cases.tokens(n, cfg["vocab"], seed=i) for i, n in enumerate((283, 1, 70, 131, 40))}
    want = {r: gc.expected(cfg, w, t) for r, t in toks.items()}
    sure = {r: sure_rows(name, cfg, w, t, dtype) for r, t in toks.items()}
    noise = {r: gc.rounding(cfg, w, t, dtype) for r, t in toks.items()}

    def check(r, logits, what):
        ok = sure[r]
        if ok.any():
            err, ref = gc.errors(logits, want[r])[ok], noise[r][ok]
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
    """Far past every window."""
    model, cfg, w = checkpoints(name, "bfloat16")
    toks = cases.tokens(330, cfg["vocab"], seed=9)
    got = cases.run_schedule(build_engine(model, 384), {"a": toks}, [{"a": 3}] + [{"a": 1}] * 327)
    err, noise = gc.errors(got["a"], gc.expected(cfg, w, toks)), gc.rounding(cfg, w, toks, "bfloat16")
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
            assert o[:len(p)] == p and len(o) == len(p) + 20 and gc.greedy_is_right(cfg, w, p, o[len(p):], slack), kw
    model.release_device_loops()
    for burst, blocks in ((0, None), (8, None), (8, 5)):
        engine = ServingEngine(model, max_num_seqs=3, max_model_len=192, num_blocks=blocks, max_prefill_tokens=40, eos_token_id=None,
                               decode_burst=burst)
        reqs = [engine.add_request(f"q{i}", p, SamplingParams(max_tokens=20, temperature=0.0)) for i, p in enumerate(prompts)]
        engine.run_until_idle()
        for p, r in zip(prompts, reqs):
            assert len(r.output) == 20 and gc.greedy_is_right(cfg, w, p, r.output, slack), (burst, blocks, len(p))
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
    assert all(t.dtype == torch.float32 for r in ctx.recurrent if r is not None for t in r) and ctx.carry.dtype == torch.float32
    assert ctx.key_cache[0] is None and ctx.key_cache[1].dtype == torch.bfloat16
