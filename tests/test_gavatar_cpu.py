"""Gavatar on the host side: configuration and registry, checkpoint names and loading, states per slot, scheduling through the
engine and the trace replay, generation, against the plain implementation of ``oracles/gavatar.py`` (CPU bodies of the ops)."""
import io
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

from mindformers_b200.checkpoint import name_maps
from mindformers_b200.inference import ragged_attention as ragged
from mindformers_b200.inference.paged_attention import KVCacheContext
from mindformers_b200.models import AutoConfig, AutoModel, GavatarConfig, GavatarForCausalLM
from mindformers_b200.ops import build as kernels
from mindformers_b200.ops import recurrent, stream
from mindformers_b200.parallel.layers.transformer_layer import SandwichTransformerLayer
from mindformers_b200.serving import SamplingParams, ServingEngine
from mindformers_b200.serving.trace import build_engine, replay

from oracles import cases, gavatar
from oracles import gavatar_cases as gc
from oracles.paged import attention_case


@pytest.fixture(scope="module")
def checkpoint(tmp_path_factory):
    cfg = gc.CASES["mixed_layers"]
    w = gc.weights("mixed_layers", seed=3)
    return cases.write_checkpoint(tmp_path_factory.mktemp("gavatar"), cfg, w), cfg, w


@pytest.fixture(scope="module")
def model(checkpoint):
    return cases.load(checkpoint[0], "float32", "cpu")


def rand(*shape, seed=0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed))


# ---- configuration and weights ----------------------------------------------------------------------------------------------
def test_config_resolves_by_architecture_and_describes_every_layer(checkpoint):
    path, cfg, w = checkpoint
    config = AutoConfig.from_pretrained(path)
    assert isinstance(config, GavatarConfig)
    m = AutoModel.from_config(config, device="cpu", dtype="float32")
    assert isinstance(m, GavatarForCausalLM)
    tc, dec = m.config, m.model.decoder
    assert tc.num_layers == 5 and tc.moe_layer_freq == [1, 0, 1, 1, 0] and tc.embedding_scale == 3.0
    assert tc.layer_runs() == gavatar.layer_runs(cfg) == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (1, 2), (2, None),
                                                          (3, None), (4, None)]
    assert dec.run_order == [0, 1, 2, 1, 2, 1, 2, 3, 4] and dec.num_runs == 9 and dec.loop_step.shape == (3, 160)
    for i, layer in enumerate(cfg["layers"]):
        c, mix, module = tc.for_layer(i), layer["mixer"], dec.layers[i]
        assert isinstance(module, SandwichTransformerLayer) and (module.mlp is None) == (layer["mlp"] is None)
        if layer["type"] == "mlstm":
            assert (c.mixer, c.memory_heads, c.memory_key_dim, c.memory_value_dim, c.memory_gate_cap) == (
                "matrix_memory", mix["heads"], mix["dim"], mix["vdim"], mix["gate_cap"])
        else:
            assert (c.num_attention_heads, c.kv_channels, c.v_channels, c.softmax_scale, c.attention_window) == (
                mix["heads"], mix["dim"], mix["vdim"], mix["scale"], mix["mask"]["size"])
        if layer["type"] == "attention":
            assert c.mixer == "attention" and c.num_query_groups == mix["kv_heads"] and c.attention_talk and not c.attention_sink
        if layer["type"] == "latent_attention":
            assert (c.mixer, c.q_lora_rank, c.kv_lora_rank) == ("latent", mix["q_rank"], mix["kv_rank"]) and c.attention_sink
        if layer["mlp"]:
            r = layer["mlp"]["router"]
            assert (c.num_moe_experts, c.moe_router_topk, c.moe_ffn_hidden_size) == (r["experts"], r["top"], layer["mlp"]["expert"]["ff"])
    attn, lat = (2, 48, 32), (1, 136, 0)
    assert dec.cache_shapes() == [None, attn, lat, attn, lat, attn, lat, (4, 24, 56), None]
    assert dec.state_shapes()[0] == [(6, 40, 24), (6, 40), (6,)] and dec.state_shapes()[1] is None and dec.carry_width() == 160
    ctx, _ = m._set_kv_cache(3, 64)
    assert ctx.carry.shape == (9, 3, 160) and ctx.has_state and ctx.value_cache[2] is None
    for bad, what in ((dict(cfg["layers"][0], type="other"), "unknown mixer"),
                      (dict(cfg["layers"][0], mlp=dict(kind="dense", ff=8)), "unknown feed-forward"),
                      (dict(cfg["layers"][0], mlp=gc.moe(2, 3)), "experts")):
        with pytest.raises(ValueError, match=what):
            GavatarConfig(**dict(cfg, loop=None, layers=[bad])).to_transformer_dict()
    with pytest.raises(ValueError, match="layer_loop"):
        AutoModel.from_config(dict(cfg, loop=dict(start=2, stop=7, times=2)), device="cpu", dtype="float32")


def test_default_configuration_and_preset_build():
    assert GavatarConfig().to_transformer_dict()["num_layers"] == 3
    m = AutoModel.from_pretrained("tiny_gavatar", device="cpu", dtype="float32")
    assert isinstance(m, GavatarForCausalLM) and m.model.decoder.num_runs == 5
    assert torch.isfinite(m(torch.randint(0, 100, (2, 9)))).all()


def test_checkpoint_names_round_trip(checkpoint, model, tmp_path):
    path, cfg, w = checkpoint
    own = dict(model.named_parameters())
    fw = name_maps.hf_to_framework(w, model.config, "gavatar")
    assert set(fw) == set(own)
    for n, t in fw.items():
        assert torch.equal(own[n].detach(), t.float()), n
    back = name_maps.framework_to_hf({n: p.detach() for n, p in own.items()}, model.config, "gavatar")
    assert set(back) == set(w) and all(torch.equal(back[n], w[n].float()) for n in w)
    for kw in (dict(hf_names=True), dict(hf_names=False)):          # the design's own names, the framework's names
        model.save_pretrained(str(tmp_path / str(kw)), **kw)
        again = AutoModel.from_pretrained(str(tmp_path / str(kw)), dtype="float32", device="cpu", strict=True)
        assert all(torch.equal(a, b) for a, b in zip(again.parameters(), model.parameters()))
    with pytest.raises(KeyError, match="counterpart"):
        name_maps.hf_to_framework(dict(w, **{"l0.mix.unknown": w["final.norm"]}), model.config, "gavatar")
    for gone, what in (("l1.mix.talk", "talk"), ("l2.mix.uv", "missing"), ("loop.step", "loop_step"), ("l3.mlp.router.b", "router.bias")):
        missing = {k: v for k, v in w.items() if k != gone}
        with pytest.raises(KeyError, match=what):
            AutoModel.from_pretrained(cases.write_checkpoint(tmp_path / gone, cfg, missing), dtype="float32", device="cpu", strict=True)


def test_kernel_sources_of_the_model_exist():
    assert len(kernels._sources(GavatarForCausalLM.kernel_sources)) == len(GavatarForCausalLM.kernel_sources)


# ---- single mechanisms --------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("width", [24, 7])
def test_embedding(width):
    table, ids, pos = rand(11, width), torch.tensor([3, 10, 0, 3]), torch.tensor([0, 1, 513, 100003])
    want = table[ids].double() * 2.5 + gavatar.position_vectors(100004, width, torch.float64)[pos]
    got = stream.embed(ids, table, 2.5, pos, stream.sinusoidal_frequencies(width))
    assert got.dtype == torch.float32 and torch.allclose(got.double(), want, atol=1e-6)
    assert torch.equal(stream.embed(ids, table, 2.5, pos, None), table[ids] * 2.5)


def test_layer_runs_of_the_plain_implementation():
    cfg = gc.config([gc.mlstm()] * 4, loop=(1, 3, 2))
    assert [i for i, _ in gavatar.layer_runs(cfg)] == [0, 1, 2, 1, 2, 3]
    assert [t for _, t in gavatar.layer_runs(cfg)] == [None, 0, None, 1, None, None]


def test_normed_step_with_a_shift_over_portions_and_idle_rows():
    W, eps = 20, 1e-3
    w_in, w_out, mu, step = (rand(W, seed=i) * 0.3 for i in range(4))
    x, y = rand(13, W, seed=5), rand(13, W, seed=6)
    x2 = x + gavatar.norm(y, w_in, eps) + step
    want = gavatar.token_shift(gavatar.norm(x2, w_out, eps), mu)
    ctx = KVCacheContext(2, 1, 64, 0, 0, torch.float32, "cpu", layer_shapes=[None] * 2, slots=3, carry_width=W)
    ctx.carry.normal_(0, 9)
    kept, at, got = ctx.carry.clone(), 0, []
    for n, prefill in ((2, True), (1, True), (5, True), (1, False), (1, False), (3, True)):
        ctx.set_step(is_prefill=prefill, block_tables=np.zeros((3, 1)), slot_mapping=[0] * n if prefill else [-1, at, -1],
                     context_lens=[7, at + n, 40], q_seq_lens=[0, n, 0] if prefill else [1] * 3, device="cpu")
        rows = torch.arange(at, at + n) if prefill else torch.tensor([0, at, 0])
        h, new = stream.normed_step(x[rows], y[rows], w_in, step, w_out, eps, True, stream.Carry(mu, ctx, 1))
        assert torch.allclose(new, x2[rows], atol=1e-6)
        got.append(h if prefill else h[1:2])
        at += n
    assert torch.allclose(torch.cat(got), want, atol=1e-5)
    assert torch.equal(ctx.carry[0], kept[0]) and torch.equal(ctx.carry[1, [0, 2]], kept[1, [0, 2]])
    h, new = stream.normed_step(x, None, None, None, w_out, eps, False)
    assert new is x and torch.allclose(h, gavatar.rms(x, eps) * w_out, atol=1e-6)


def test_mixed_weights_are_mixed_results():
    """Mixing the softmax weights over heads before the product with the values, and after it."""
    g = torch.Generator().manual_seed(2)
    H, G, T, DV = 6, 2, 9, 5
    p, v, talk = torch.rand(H, T, T, generator=g), torch.randn(T, G, DV, generator=g), torch.randn(H, H, generator=g)
    own = torch.arange(H) // (H // G)
    want = torch.einsum("hqk,khd->qhd", gavatar.talk_over_heads(p, talk), v[:, own]).reshape(T, H * DV)
    gate = torch.randn(T, H * DV, generator=g)
    got = stream.talk_mix(torch.einsum("hqk,kgd->qhgd", p, v), talk, gate)
    assert torch.allclose(got, want * torch.sigmoid(gate), atol=1e-5)


@pytest.mark.parametrize("window", [1, 5, 16, 33, 1000])
def test_windows_of_the_paged_attention(window):
    lens, news = [1, 40, 33, 60, 17], [1, 40, 2, 25, 1]
    for kw in (dict(), dict(all_values=True)):
        ctx, table, qs, sink, scale, want = attention_case(torch.float32, 4, 2, 8, 6, 16, 0, lens, news, device="cpu", window=window, **kw)
        ctx.set_step(is_prefill=True, block_tables=table.clamp(min=0), slot_mapping=[0] * sum(news), context_lens=lens, q_seq_lens=news,
                     device="cpu")
        got = ragged.ragged_attention(torch.cat(qs), ctx, 0, scale, sink=None if kw else sink, window=window, **kw)
        assert torch.allclose(got.double(), want, atol=1e-5)


def test_prefill_work_with_a_window():
    assert ragged.first_visible(10, 0, 4) == 7 and ragged.first_visible(2, 0, 4) == 0 and ragged.first_visible(10, 8, 100) == 8
    work = ragged.prefill_work([300, 1, 130], [300, 50, 1130], 0, 100)
    assert sorted(work) == [(0, 0, 128, 0), (0, 128, 128, 128), (0, 256, 44, 256), (2, 301, 128, 1000), (2, 429, 2, 1128)]
    tiles = [(p + n - 1) // 128 - ragged.first_visible(p, 0, 100) // 128 for _, _, n, p in work]
    assert tiles == sorted(tiles, reverse=True)


def test_state_belongs_to_the_slot_and_needs_no_clearing():
    """A slot that held another sequence, a portion that starts at 0, and idle rows of a decode step."""
    H, D, DV, T, eps = 3, 8, 12, 11, 1e-4
    s = recurrent.MemoryShape(H, D, DV, 4.0)
    n = 2 * H * (D + DV) + 2 * H
    proj, norm, bi, bf = rand(T, n, seed=1), 1 + 0.2 * rand(H * DV, seed=2), rand(H, seed=3), 2 + rand(H, seed=4)
    named, at = {"norm": norm, "i.b": bi, "f.b": bf, "o": torch.eye(H * DV)}, 0
    for name, rows in (("q", H * D), ("k", H * D), ("v", H * DV), ("g", H * DV), ("i", H), ("f", H)):
        named[name] = torch.eye(n)[at:at + rows]
        at += rows
    want = gavatar.mlstm(proj, lambda x: named[x], dict(heads=H, dim=D, vdim=DV, gate_cap=4.0), eps)
    ctx = KVCacheContext(1, 2, 64, 0, 0, torch.float32, "cpu", layer_shapes=[None], state_shapes=[[(H, D, DV), (H, D), (H,)]], slots=3)
    for t in ctx.recurrent[0]:
        t.normal_(0, 5)                                                  # what earlier sequences left
    other = [t[[0, 2]].clone() for t in ctx.recurrent[0]]
    got, at = [], 0
    for n, prefill in ((1, True), (2, True), (4, True), (1, False), (1, False), (2, True)):
        ctx.set_step(is_prefill=prefill, block_tables=np.zeros((3, 1)), slot_mapping=[0] * n if prefill else [-1, at, -1],
                     context_lens=[7, at + n, 40], q_seq_lens=[0, n, 0] if prefill else [1] * 3, device="cpu")
        rows = torch.arange(at, at + n) if prefill else torch.tensor([0, at, 0])
        o = recurrent.matrix_memory(proj[rows], bi, bf, norm, s, ctx.recurrent[0], ctx, eps)
        got.append(o if prefill else o[1:2])
        at += n
    assert torch.allclose(torch.cat(got), want, atol=1e-5)
    assert all(torch.equal(t[[0, 2]], o) for t, o in zip(ctx.recurrent[0], other))


# ---- the whole model ---------------------------------------------------------------------------------------------------------------
LENGTHS = (("a", 130), ("b", 1), ("c", 75), ("d", 52), ("e", 20))
SCHEDULES = (
    ([{r: n} for r, n in LENGTHS], 192),
    ([{r: c} for r, n in LENGTHS for c in cases.portions(n, (2, 31, 1, 2, 19, 3))], 192),
    ([{"a": 20, "b": 1, "c": 2, "d": 30}, {"a": 2, "c": 72}, {"a": 1, "e": 18, "d": 21}, {"c": 1, "e": 2, "a": 107}, {"d": 1}], 448))


def test_schedules_give_the_same_logits(checkpoint, model):
    _, cfg, w = checkpoint
    toks = {r: cases.tokens(n, cfg["vocab"], seed=n) for r, n in LENGTHS}
    want = {r: gc.expected(cfg, w, t) for r, t in toks.items()}
    for schedule, pool in SCHEDULES:
        got = cases.run_schedule(build_engine(model, pool), toks, schedule)
        for r in toks:
            assert cases.worst(got[r], want[r]) < 2e-5, (r, schedule[0])


@pytest.mark.parametrize("name", ["chosen_experts", "odd_sizes"])
def test_other_sizes(name, tmp_path):
    cfg, w = gc.CASES[name], gc.weights(name, seed=5)
    m = cases.load(cases.write_checkpoint(tmp_path, cfg, w), "float32", "cpu")
    toks = cases.tokens(110, cfg["vocab"], seed=1)
    got = cases.run_schedule(build_engine(m, 128), {"a": toks}, [{"a": c} for c in (17, 2, 1, 1, 3, 68, 16, 2)])
    assert cases.worst(got["a"], gc.expected(cfg, w, toks)) < 2e-5


def test_layer_runs_follow_the_plain_implementation(checkpoint, model):
    """The stream after every layer run (the run's last output enters it in the next step)."""
    _, cfg, w = checkpoint
    toks, trace, seen = cases.tokens(30, cfg["vocab"], seed=5), [], []
    gavatar.forward(cfg, w, toks, torch.float64, trace)

    def after(mod, args, out):
        y, res, _ = out
        seen.append(res.x + gavatar.norm(y, res.norm.weight, 1e-5))
    hooks = [layer.register_forward_hook(after) for layer in model.model.decoder.layers]
    logits = model(torch.tensor([toks]))
    for h in hooks:
        h.remove()
    assert len(seen) == len(trace) == 9
    for a, b in zip(seen, trace):
        assert torch.allclose(a.double(), b, rtol=1e-4, atol=1e-3)
    assert cases.worst(logits, gc.expected(cfg, w, toks)) < 2e-5


def test_mistakes_would_show(checkpoint, monkeypatch):
    """The checkpoint is sensitive: what a wrong window, sink, state, shift, matrix or pass would do moves the logits far beyond
    the limits used here."""
    _, cfg, w = checkpoint
    toks = cases.tokens(150, cfg["vocab"], seed=6)
    want = gc.expected(cfg, w, toks)

    def changed(edit_cfg=None, edit_w=None, patch=None):
        c, v = json.loads(json.dumps(cfg)), dict(w)
        if edit_cfg:
            edit_cfg(c)
        if edit_w:
            edit_w(v)
        with monkeypatch.context() as mp:
            for name, fn in (patch or {}).items():
                mp.setattr(gavatar, name, fn)
            return cases.worst(gc.expected(c, v, toks), want)
    memory, shift = gavatar.matrix_memory, gavatar.token_shift

    def lost(*a):                                               # the state is lost at token 30
        return torch.cat((memory(*(t[:30] for t in a)), memory(*(t[30:] for t in a))))

    def lost_shift(h, mu):
        return torch.cat((shift(h[:30], mu), shift(h[30:], mu)))
    zero = lambda n: (lambda v: v.update({n: torch.zeros_like(v[n])}))
    assert changed(patch=dict(matrix_memory=lost)) > 1e-2
    assert changed(patch=dict(token_shift=lost_shift)) > 1e-2
    assert changed(patch=dict(talk_over_heads=lambda p, t: p)) > 1e-2
    for i in (1, 2, 3):                                         # a window that is one token off
        for d in (-1, 1):
            assert changed(lambda c: c["layers"][i]["mixer"]["mask"].update(size=c["layers"][i]["mixer"]["mask"]["size"] + d)) > 1e-3, (i, d)
    assert changed(None, lambda v: v.update({"l2.mix.sink": v["l2.mix.sink"] - 30})) > 1e-3
    assert changed(None, lambda v: v.update({"l1.mix.talk": v["l1.mix.talk"].t()})) > 1e-3
    assert changed(lambda c: c["loop"].update(times=2)) > 1e-2
    assert changed(None, lambda v: v.update({"loop.step": v["loop.step"].flip(0)})) > 1e-2
    assert changed(lambda c: c["layers"][0]["mixer"].update(gate_cap=6.0)) > 1e-3
    for name in ("l1.mix.v.b", "l1.mix.q.b", "l3.mlp.router.b", "l0.mix.f.b", "l2.mix.g", "l0.mix.g", "l1.mix.g", "final.norm"):
        assert changed(None, zero(name)) > 1e-3, name
    assert changed(patch=dict(position_vectors=lambda T, W, dt: torch.zeros(T, W, dtype=dt))) > 1e-2


def test_a_far_token_decides_and_is_found(tmp_path):
    """A memory that keeps everything (forget gates of 1): what the first token wrote is read through portions and decoded
    tokens."""
    cfg = gc.config([gc.mlstm(2, 16, 16, 40.0, None)], width=64, vocab=90)
    w = gavatar.random_weights(cfg, seed=4, gates=((0.0, 0.1), (30.0, 0.0)))
    m = cases.load(cases.write_checkpoint(tmp_path, cfg, w), "float32", "cpu")
    a = cases.tokens(260, 90, seed=2)
    b = [(a[0] + 1) % 90] + a[1:]                              # the same tokens but for the first
    want_a, want_b = gc.expected(cfg, w, a), gc.expected(cfg, w, b)
    assert cases.worst(want_b[200:], want_a[200:]) > 1e-3
    for toks, want in ((a, want_a), (b, want_b)):
        got = cases.run_schedule(build_engine(m, 320), {"a": toks}, [{"a": c} for c in (100, 2, 64, 61)] + [{"a": 1}] * 33)["a"]
        assert cases.worst(got, want) < 2e-5


# ---- generation and serving -----------------------------------------------------------------------------------------------------------
def greedy_reference(cfg, w, prompt, n):
    out = list(prompt)
    for _ in range(n):
        out.append(int(gc.expected(cfg, w, out)[-1].argmax()))
    return out[len(prompt):]


def test_greedy_generation_through_generate_and_the_engine(checkpoint, model):
    _, cfg, w = checkpoint
    prompts = [cases.tokens(n, cfg["vocab"], seed=30 + n) for n in (40, 1, 66)]
    want = [greedy_reference(cfg, w, p, 6) for p in prompts]
    for kw in (dict(), dict(chunk_prefill_size=17), dict(use_cuda_graph=True)):
        out = model.generate(prompts, max_new_tokens=6, do_sample=False, eos_token_id=None, **kw)
        assert [o[len(p):] for o, p in zip(out, prompts)] == want, kw
    for burst, blocks in ((0, None), (4, None), (4, 3)):
        engine = ServingEngine(model, max_num_seqs=2, max_model_len=128, num_blocks=blocks, max_prefill_tokens=25, eos_token_id=None,
                               decode_burst=burst)
        reqs = [engine.add_request(f"r{i}", p, SamplingParams(max_tokens=6, temperature=0.0)) for i, p in enumerate(prompts)]
        engine.run_until_idle()
        assert [r.output for r in reqs] == want, (burst, blocks)
        assert engine.counters["mixed_steps"] >= 3 and engine.stats()["free_blocks"] == engine.stats()["total_blocks"]


def test_beams_and_shared_prefixes_carry_their_states(checkpoint, model):
    """The best beam scores what the plain implementation gives it; a shared prefix gives the same tokens; drafts, which take
    tokens back, are refused."""
    _, cfg, w = checkpoint
    p = cases.tokens(20, cfg["vocab"], seed=3)
    out = model.generate([p], max_new_tokens=4, num_beams=3, do_sample=False, eos_token_id=None)[0]

    def score(seq):
        lp = torch.log_softmax(gc.expected(cfg, w, seq), dim=-1)
        return float(sum(lp[i - 1, seq[i]] for i in range(len(p), len(seq))))
    beams = [(0.0, p)]
    for _ in range(4):
        cand = []
        for s, seq in beams:
            lp = torch.log_softmax(gc.expected(cfg, w, seq)[-1], dim=-1)
            v, i = lp.topk(6)
            cand += [(s + float(a), seq + [int(b)]) for a, b in zip(v, i)]
        beams = sorted(cand, reverse=True)[:3]
    assert abs(score(out) - beams[0][0]) < 1e-4
    head = cases.tokens(70, cfg["vocab"], seed=9)
    prompts = [head + [1, 2], head + [3], head + [4, 5, 6]]
    plain = model.generate(prompts, max_new_tokens=4, do_sample=False, eos_token_id=None)
    assert model.generate(prompts, max_new_tokens=4, do_sample=False, eos_token_id=None, parallel_decoding="prefix_cache") == plain
    with pytest.raises(NotImplementedError, match="recurrent"):
        model.generate(prompts, max_new_tokens=4, do_sample=False, eos_token_id=None, parallel_decoding="la")


def test_sampling_is_seeded(model):
    engine = ServingEngine(model, max_num_seqs=2, max_model_len=64, eos_token_id=None)
    a, b = engine.generate([[1, 2, 3], [1, 2, 3]], SamplingParams(max_tokens=6, temperature=0.8, top_k=20, seed=7))
    assert a.token_ids == b.token_ids and len(a.token_ids) == 6


def test_trace_replay(checkpoint, model, tmp_path):
    _, cfg, w = checkpoint
    toks = cases.tokens(30, cfg["vocab"], seed=8)
    lines = [json.dumps(dict(step=0, entries=[dict(id="x", tokens=toks[:20], want=[])], end=[])),
             json.dumps(dict(step=1, entries=[dict(id="x", tokens=toks[20:29], want=[0, 8])], end=[])), "",
             json.dumps(dict(step=2, entries=[dict(id="x", tokens=toks[29:], want=[0])], end=["x"]))]
    out = io.StringIO()
    engine = build_engine(model, 64)
    replay(engine, lines, str(tmp_path), out)
    assert out.getvalue() == "done 0\ndone 1\ndone 2\n" and engine.tables.pool.num_free == 1
    assert engine.ctx.recurrent[0][0].shape[0] == 4 and engine.ctx.carry.shape[1] == 4       # a state for each of the four slots
    want = gc.expected(cfg, w, toks)
    assert not os.path.exists(tmp_path / "0.f32")
    for step, rows in ((1, [20, 28]), (2, [29])):
        got = np.fromfile(tmp_path / f"{step}.f32", dtype="<f4").reshape(len(rows), -1)
        assert cases.worst(torch.from_numpy(got), want[rows]) < 1e-4


def test_command_line_predict(checkpoint, tmp_path):
    path, cfg, w = checkpoint
    yaml = tmp_path / "p.yaml"
    yaml.write_text("run_mode: predict\nuse_parallel: false\nuse_legacy: false\noutput_dir: " + str(tmp_path) + "\n"
                    "trainer: {type: CausalLanguageModelingTrainer, model_name: Gavatar}\n"
                    "processor: {tokenizer: {type: ByteTokenizer}}\n")
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    env = dict(os.environ, CUDA_VISIBLE_DEVICES="")
    res = subprocess.run([sys.executable, os.path.join(root, "run_mindformer.py"), "--config", str(yaml), "--run_mode", "predict",
                          "--pretrained_model_dir", path, "--predict_data", "abc", "--save_file", str(tmp_path / "out.txt")],
                         capture_output=True, text=True, timeout=300, env=env, cwd=str(tmp_path))
    assert res.returncode == 0 and "abc" in (tmp_path / "out.txt").read_text(), res.stdout[-1500:] + res.stderr[-3000:]
