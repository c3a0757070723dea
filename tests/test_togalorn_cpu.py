"""Togalorn on the host side: configuration and registry, checkpoint names and loading, states per slot, scheduling through the
engine and the trace replay, generation, against the plain implementation of ``oracles/togalorn.py`` (CPU bodies of the ops)."""
import io
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

from mindformers_b200.checkpoint import name_maps
from mindformers_b200.inference.paged_attention import KVCacheContext
from mindformers_b200.models import AutoConfig, AutoModel, TogalornConfig, TogalornForCausalLM
from mindformers_b200.ops import build as kernels
from mindformers_b200.ops import recurrent, stream
from mindformers_b200.parallel.layers import ragged_attention as layers
from mindformers_b200.parallel.layers.transformer_layer import ParallelTransformerLayer
from mindformers_b200.serving import SamplingParams, ServingEngine
from mindformers_b200.serving.trace import build_engine, replay

from oracles import cases, togalorn
from oracles import togalorn_cases as tc


@pytest.fixture(scope="module")
def checkpoint(tmp_path_factory):
    cfg = tc.CASES["mixed_layers"]
    w = tc.weights("mixed_layers", seed=3)
    return cases.write_checkpoint(tmp_path_factory.mktemp("togalorn"), cfg, w), cfg, w


@pytest.fixture(scope="module")
def model(checkpoint):
    return cases.load(checkpoint[0], "float32", "cpu")


def rand(*shape, seed=0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed))


# ---- configuration and weights ----------------------------------------------------------------------------------------------
def test_config_resolves_by_architecture_and_describes_every_layer(checkpoint):
    path, cfg, w = checkpoint
    config = AutoConfig.from_pretrained(path)
    assert isinstance(config, TogalornConfig)
    m = AutoModel.from_config(config, device="cpu", dtype="float32")
    assert isinstance(m, TogalornForCausalLM)
    c0, dec = m.config, m.model.decoder
    assert c0.num_layers == 5 and c0.moe_layer_freq == [1, 0, 1, 1, 0] and c0.embedding_scale == 3.0 and c0.norm_groups == 5
    assert c0.layer_runs() == togalorn.layer_runs(cfg)
    assert dec.run_order == [0, 1, 2, 1, 2, 1, 2, 3, 4] and dec.loop_step.shape == (3, 160) and dec.loop_in.shape == (160, 320)
    for i, layer in enumerate(cfg["layers"]):
        c, mix, module = c0.for_layer(i), layer["mixer"], dec.layers[i]
        assert isinstance(module, ParallelTransformerLayer) and (module.mlp is None) == (layer["mlp"] is None)
        assert module.input_conv.shape == (3, 160)
        if layer["type"] == "mamba2":
            assert (c.mixer, c.ssm_heads, c.ssm_head_dim, c.ssm_state, c.ssm_groups, c.ssm_conv_taps, c.ssm_norm_groups) == (
                "state_space", mix["heads"], mix["vdim"], mix["state"], mix["groups"], mix["conv"], mix["norm_groups"])
        else:
            assert (c.mixer, c.num_attention_heads, c.kv_channels, c.v_channels, c.softmax_scale, c.rotary_dim, c.rotary_base,
                    c.q_lora_rank, c.kv_lora_rank) == ("latent", mix["heads"], mix["dim"], mix["vdim"], mix["scale"], mix["rot_dim"],
                                                       mix["rot"]["base"], mix["q_rank"], mix["kv_rank"])
        if layer["mlp"]:
            r, e, s = (layer["mlp"][k] for k in ("router", "expert", "shared"))
            assert (c.num_moe_experts, c.moe_identity_experts, c.moe_router_topk, c.moe_ffn_hidden_size, c.moe_activation_limit) == (
                r["experts"], r["identity"], r["top"], e["ff"], e["limit"])
            assert (c.moe_shared_expert_intermediate_size, c.moe_shared_expert_activation_limit) == (s["ff"], s["limit"])
            assert module.mlp.router.weight.shape == (r["experts"] + r["identity"], 160)
    a, b = (1, 152, 0), (1, 72, 0)
    assert dec.cache_shapes() == [None, a, None, a, None, a, None, b, None]
    assert dec.state_shapes()[0] == (6, 40, 24, 6 * 24 + 2 * 3 * 40, 4) and dec.state_shapes()[1] is None and dec.carry_width() == 320
    ctx, _ = m._set_kv_cache(3, 64)
    assert ctx.carry.shape == (9, 3, 320) and ctx.has_state and ctx.value_cache[1] is None
    bad_rot = json.loads(json.dumps(cfg["layers"][1]))
    bad_rot["mixer"]["rot"]["dims"] = 4
    for bad, what in ((dict(cfg["layers"][0], type="other"), "unknown mixer"), (bad_rot, "rotated"),
                      (dict(cfg["layers"][0], mlp=dict(kind="dense", ff=8)), "unknown feed-forward"),
                      (dict(cfg["layers"][0], mlp=tc.moe(2, 1, 4)), "experts")):
        with pytest.raises(ValueError, match=what):
            TogalornConfig(**dict(cfg, loop=None, layers=[bad])).to_transformer_dict()
    for bad, what in ((dict(norm=dict(eps=1e-5, groups=7)), "parts"), (dict(loop=dict(start=2, stop=7, times=2)), "layer_loop"),
                      (dict(layers=[tc.mamba(6, 16, 24, 4)], loop=None), "state space")):
        with pytest.raises(ValueError, match=what):
            AutoModel.from_config(dict(cfg, **bad), device="cpu", dtype="float32")


def test_default_configuration_and_preset_build():
    assert TogalornConfig().to_transformer_dict()["num_layers"] == 3
    m = AutoModel.from_pretrained("tiny_togalorn", device="cpu", dtype="float32")
    assert isinstance(m, TogalornForCausalLM) and m.model.decoder.num_runs == 5
    assert torch.isfinite(m(torch.randint(0, 100, (2, 9)))).all()


def tensors(m):
    return {**dict(m.named_parameters()), **{n: b for n, b in m.named_buffers() if n.endswith("expert_bias")}}


def test_checkpoint_names_round_trip(checkpoint, model, tmp_path):
    path, cfg, w = checkpoint
    own = tensors(model)
    fw = name_maps.hf_to_framework(w, model.config, "togalorn")
    assert set(fw) == set(own)
    for n, t in fw.items():
        assert torch.equal(own[n].detach(), t.float()), n
    back = name_maps.framework_to_hf({n: p.detach() for n, p in own.items()}, model.config, "togalorn")
    assert set(back) == set(w) and all(torch.equal(back[n], w[n].float()) for n in w)
    for kw in (dict(hf_names=True), dict(hf_names=False)):          # the design's own names, the framework's names
        model.save_pretrained(str(tmp_path / str(kw)), **kw)
        again = AutoModel.from_pretrained(str(tmp_path / str(kw)), dtype="float32", device="cpu", strict=True)
        assert all(torch.equal(a, b) for a, b in zip(tensors(again).values(), own.values()))
    with pytest.raises(KeyError, match="counterpart"):
        name_maps.hf_to_framework(dict(w, **{"l0.mix.unknown": w["final.norm"]}), model.config, "togalorn")
    for gone, what in (("l1.mix.g", "missing"), ("l1.mix.uv", "missing"), ("loop.in", "loop_in"), ("l3.mlp.router", "router.weight"),
                       ("l2.canon1", "input_conv"), ("l0.mlp.shared.up", "missing"), ("l3.mlp.correction", "correction")):
        missing = {k: v for k, v in w.items() if k != gone}
        with pytest.raises(KeyError, match=what):
            AutoModel.from_pretrained(cases.write_checkpoint(tmp_path / gone, cfg, missing), dtype="float32", device="cpu", strict=True)


def test_kernel_sources_of_the_model_exist():
    assert len(kernels._sources(TogalornForCausalLM.kernel_sources)) == len(TogalornForCausalLM.kernel_sources)


# ---- single mechanisms --------------------------------------------------------------------------------------------------------
def context(slots=3, **kw):
    return KVCacheContext(2, 1, 64, 0, 0, torch.float32, "cpu", layer_shapes=[None] * 2, slots=slots, **kw)


PORTIONS = ((2, True), (1, True), (5, True), (1, False), (1, False), (3, True))       # 13 rows of slot 1


def walk(ctx, step):
    """``step(rows) -> result`` of the portions of one sequence in slot 1 of three; the rows of slot 1 put together."""
    got, at = [], 0
    for n, prefill in PORTIONS:
        ctx.set_step(is_prefill=prefill, block_tables=np.zeros((3, 1)), slot_mapping=[0] * n if prefill else [-1, at, -1],
                     context_lens=[7, at + n, 40], q_seq_lens=[0, n, 0] if prefill else [1] * 3, device="cpu")
        out = step(torch.arange(at, at + n) if prefill else torch.tensor([0, at, 0]))
        got.append(out if prefill else out[1:2])
        at += n
    return torch.cat(got)


@pytest.mark.parametrize("taps,groups", [(1, 1), (2, 4), (3, 2), (4, 5), (7, 1)])
def test_joint_step_over_portions_and_idle_rows(taps, groups):
    W, eps = 20, 1e-3
    x, y0, y1, base = (rand(13, W, seed=i) for i in range(4))
    w, vec, conv = rand(W, seed=5), rand(W, seed=6), rand(W, taps, seed=7)
    x2 = x + y0 + y1 + base + vec
    h = togalorn.grouped_norm(x2, w, groups, eps)
    want = h + togalorn.causal_conv(h, conv)
    ctx = context(carry_width=(taps - 1) * W)
    kept = None
    if taps > 1:
        ctx.carry.normal_(0, 9)                                      # what earlier sequences left
        kept = ctx.carry.clone()
    ic = stream.InputConv(conv.t().contiguous(), ctx, 1)

    def step(rows):
        a, b, new = stream.joint_step(x[rows], (y0[rows], y1[rows]), base[rows], vec, w, groups, eps, torch.float32, ic)
        assert torch.allclose(new, x2[rows], atol=1e-6) and torch.allclose(a, h[rows], atol=1e-5)
        return b
    assert torch.allclose(walk(ctx, step), want, atol=1e-5)
    if kept is not None:
        assert torch.equal(ctx.carry[0], kept[0]) and torch.equal(ctx.carry[1, [0, 2]], kept[1, [0, 2]])
    a, b, new = stream.joint_step(x, (None, y1), None, None, None, 1, 0.0, torch.bfloat16, want_h=True, keep=False)
    assert new is None and b is None and torch.equal(a, (x + y1).to(torch.bfloat16))


@pytest.mark.parametrize("heads,P,N,groups,taps,norm_groups", [(3, 8, 6, 1, 4, 1), (4, 3, 5, 2, 1, 6), (2, 4, 7, 2, 6, 2)])
def test_state_space_belongs_to_the_slot_and_needs_no_clearing(heads, P, N, groups, taps, norm_groups):
    """A slot that held another sequence, a portion that starts at 0, and idle rows of a decode step."""
    s = recurrent.StateSpaceShape(heads, P, N, groups, taps, norm_groups)
    proj, conv, eps = rand(13, s.columns, seed=1), rand(s.channels, taps, seed=2), 1e-4
    named = {"in": torch.eye(s.columns), "conv": conv, "conv.b": rand(s.channels, seed=3), "dt_bias": rand(heads, seed=4),
             "A_log": rand(heads, seed=5), "D": rand(heads, seed=6), "norm": 1 + 0.2 * rand(s.inner, seed=7), "o": torch.eye(s.inner)}
    want = togalorn.mamba2(proj, lambda n: named[n], dict(heads=heads, vdim=P, state=N, groups=groups, norm_groups=norm_groups), eps)
    ctx = context(state_shapes=[None, (heads, N, P, s.channels, taps)])
    for t in ctx.recurrent[1]:
        t.normal_(0, 5)
    other = [t[[0, 2]].clone() for t in ctx.recurrent[1]]
    w = recurrent.StateSpaceWeights(conv.t().contiguous(), *(named[n] for n in ("conv.b", "dt_bias", "A_log", "D", "norm")))
    got = walk(ctx, lambda rows: recurrent.state_space(proj[rows], w, s, ctx.recurrent[1], ctx, eps))
    assert torch.allclose(got, want, atol=2e-5)
    assert all(torch.equal(t[[0, 2]], o) for t, o in zip(ctx.recurrent[1], other))


def test_rotation_and_key_factors():
    """Rotated parts of queries and cached keys; a factor with unit rows makes a head's whole key."""
    T, H, D, P, R, Q = 5, 3, 6, 4, 10, 8
    freqs, pos = 100.0 ** (-torch.arange(0, P, 2, dtype=torch.float32) / P), torch.tensor([0, 1, 7, 300, 5000])
    q = rand(T, H, D + P, seed=1)
    got = stream.rotate_tail_(q.clone(), freqs, pos)
    assert torch.equal(got[..., :D], q[..., :D])
    assert torch.allclose(got[..., D:], togalorn.rotate(q[..., D:], 100.0, pos), atol=3e-4)
    assert torch.allclose(got[:3, :, D:], togalorn.rotate(q[:3, :, D:], 100.0, pos[:3]), atol=1e-5)
    proj, qn, kn, cache = rand(T, Q + R + P + 3, seed=2), rand(Q, seed=3), rand(R, seed=4), torch.zeros(2, 4, 1, R + P)
    slots = torch.tensor([1, -1, 5, 0, 7], dtype=torch.int32)
    c_q = stream.latent_norm_cache(proj, qn, kn, 1e-4, slots, cache, freqs, pos)
    assert torch.allclose(c_q, togalorn.rms(proj[:, :Q], 1e-4) * qn, atol=1e-6)
    row = torch.cat((togalorn.rms(proj[:, Q:Q + R], 1e-4) * kn, togalorn.rotate(proj[:, Q + R:Q + R + P], 100.0, pos)), dim=1)
    keep = slots >= 0
    assert torch.allclose(cache.view(8, -1)[slots[keep].long()], row[keep], atol=3e-4)
    uk, uv = rand(H * D, R, seed=5), rand(H * 7, R, seed=6)
    w = layers.expand_kv_up(uk, uv, H, D, P)
    assert all(torch.equal(a, b) for a, b in zip(layers.split_kv_up(w, H, D, P, R), (uk, uv)))
    kv = row @ w.t()
    keys = kv[:, :H * (D + P)].view(T, H, D + P)
    assert torch.equal(keys[..., D:], row[:, None, R:].expand(T, H, P)) and torch.allclose(kv[:, H * (D + P):], row[:, :R] @ uv.t(), atol=1e-5)
    assert torch.allclose(keys[..., :D].flatten(1), row[:, :R] @ uk.t(), atol=1e-5)


def test_identity_and_shared_experts(tmp_path):
    from mindformers_b200.parallel.layers.moe import GroupedMLP, MoELayer, SharedExpertMLP, TopKRouter
    cfg = tc.config([tc.mamba(mlp=tc.moe(3, 6, 3, 24, 0.5, 40, 0.3))], width=32)
    w = togalorn.random_weights(cfg, seed=2)
    layer = cases.load(cases.write_checkpoint(tmp_path, cfg, w), "float32", "cpu").model.decoder.layers[0].mlp
    assert isinstance(layer, MoELayer) and isinstance(layer.router, TopKRouter) and isinstance(layer.experts, GroupedMLP)
    assert isinstance(layer.shared_experts, SharedExpertMLP)
    h = rand(100, 32, seed=1)
    get = lambda n: w["l0.mlp." + n].float()
    share, ids = togalorn.router(h, get, 3)
    assert (ids >= 3).any() and (ids < 3).any() and (ids >= 3).all(-1).any()          # also tokens of identity experts alone
    with torch.no_grad():
        probs, got_ids, _ = layer.router(h)
        out, _ = layer(h)
    assert torch.equal(got_ids.sort(-1).values, ids.sort(-1).values) and torch.allclose(probs.sort(-1).values, share.sort(-1).values, atol=1e-6)
    assert torch.allclose(out, togalorn.feed_forward(h, get, cfg["layers"][0]["mlp"]), atol=1e-4)
    # weights that do not sum to one before they are normalised, and choices that the correction turns around
    assert not torch.equal(togalorn.router(h, lambda n: get(n) * (n != "correction"), 3)[1].sort(-1).values, ids.sort(-1).values)


# ---- the whole model ---------------------------------------------------------------------------------------------------------------
LENGTHS = (("a", 130), ("b", 1), ("c", 75), ("d", 52), ("e", 20))
SCHEDULES = (
    ([{r: n} for r, n in LENGTHS], 192),
    ([{r: c} for r, n in LENGTHS for c in cases.portions(n, (2, 31, 1, 2, 19, 3))], 192),
    ([{"a": 20, "b": 1, "c": 2, "d": 30}, {"a": 2, "c": 72}, {"a": 1, "e": 18, "d": 21}, {"c": 1, "e": 2, "a": 107}, {"d": 1}], 448))


def test_schedules_give_the_same_logits(checkpoint, model):
    _, cfg, w = checkpoint
    toks = {r: cases.tokens(n, cfg["vocab"], seed=n) for r, n in LENGTHS}
    want = {r: tc.expected(cfg, w, t) for r, t in toks.items()}
    for schedule, pool in SCHEDULES:
        got = cases.run_schedule(build_engine(model, pool), toks, schedule)
        for r in toks:
            assert cases.worst(got[r], want[r]) < 2e-5, (r, schedule[0])


@pytest.mark.parametrize("name", ["chosen_experts", "odd_sizes"])
def test_other_sizes(name, tmp_path):
    cfg, w = tc.CASES[name], tc.weights(name, seed=5)
    m = cases.load(cases.write_checkpoint(tmp_path, cfg, w), "float32", "cpu")
    toks = cases.tokens(110, cfg["vocab"], seed=1)
    got = cases.run_schedule(build_engine(m, 128), {"a": toks}, [{"a": c} for c in (17, 2, 1, 1, 3, 68, 16, 2)])
    assert cases.worst(got["a"], tc.expected(cfg, w, toks)) < 2e-5


def test_layer_runs_follow_the_plain_implementation(checkpoint, model):
    """The stream after every layer run (the run's outputs enter it in the next step)."""
    _, cfg, w = checkpoint
    toks, trace, seen = cases.tokens(30, cfg["vocab"], seed=5), [], []
    togalorn.forward(cfg, w, toks, torch.float64, trace)

    def after(mod, args, out):
        y, res, _ = out
        seen.append(res.x + y + (0 if res.mixed is None else res.mixed))
    hooks = [layer.register_forward_hook(after) for layer in model.model.decoder.layers]
    logits = model(torch.tensor([toks]))
    for h in hooks:
        h.remove()
    assert len(seen) == len(trace) == 9
    for a, b in zip(seen, trace):
        assert torch.allclose(a.double(), b, rtol=1e-4, atol=1e-3)
    assert cases.worst(logits, tc.expected(cfg, w, toks)) < 2e-5


def test_mistakes_would_show(checkpoint, monkeypatch):
    """The checkpoint is sensitive: what a wrong rotation, state, convolution, expert or pass would do moves the logits far beyond
    the limits used here."""
    _, cfg, w = checkpoint
    toks = cases.tokens(120, cfg["vocab"], seed=6)
    want = tc.expected(cfg, w, toks)

    def changed(edit_cfg=None, edit_w=None, patch=None):
        c, v = json.loads(json.dumps(cfg)), dict(w)
        if edit_cfg:
            edit_cfg(c)
        if edit_w:
            edit_w(v)
        with monkeypatch.context() as mp:
            for name, fn in (patch or {}).items():
                mp.setattr(togalorn, name, fn)
            return cases.worst(tc.expected(c, v, toks), want)
    space, conv, rotate, norm, enter = (getattr(togalorn, n) for n in ("state_space", "causal_conv", "rotate", "grouped_norm", "enter_pass"))

    def lost(x, B, C, dt, A, D):                                # the state is lost at token 30
        return torch.cat((space(x[:30], B[:30], C[:30], dt[:30], A, D), space(x[30:], B[30:], C[30:], dt[30:], A, D)))

    def lost_conv(x, k):
        return torch.cat((conv(x[:30], k), conv(x[30:], k)))
    zero = lambda n: (lambda v: v.update({n: torch.zeros_like(v[n])}))
    assert changed(patch=dict(state_space=lost)) > 1e-2
    assert changed(patch=dict(causal_conv=lost_conv)) > 1e-2
    assert changed(patch=dict(rotate=lambda x, base, p=None: x)) > 1e-2
    assert changed(patch=dict(rotate=lambda x, base, p=None: rotate(x, base, torch.arange(x.shape[0]).clamp(max=100)))) > 1e-3
    assert changed(patch=dict(grouped_norm=lambda x, k, g, e: norm(x, k, 1, e))) > 1e-2
    assert changed(patch=dict(enter_pass=lambda x, x0, k, s: enter(x, x, k, s))) > 1e-2
    assert changed(lambda c: c["loop"].update(times=2)) > 1e-2
    assert changed(None, lambda v: v.update({"loop.step": v["loop.step"].flip(0)})) > 1e-2
    assert changed(lambda c: c["layers"][0]["mlp"]["expert"].update(limit=0.6)) > 1e-3
    assert changed(lambda c: c["layers"][0]["mlp"]["shared"].update(limit=1.1)) > 1e-3
    for name in ("l0.canon1", "l4.canon1", "l0.mix.D", "l0.mix.conv.b", "l0.mix.dt_bias", "l1.mix.g", "l2.mix.A_log", "final.norm"):
        assert changed(None, zero(name)) > 1e-3, name


def test_a_far_token_decides_and_is_found(tmp_path):
    """A state that forgets nothing: what the first token wrote is read through portions and decoded tokens."""
    cfg = tc.config([tc.mamba(2, 16, 16, 1, 1, 1, None)], width=64, vocab=90, taps=1, groups=1)
    w = togalorn.random_weights(cfg, seed=4, decay=(-30.0, 0.0))
    m = cases.load(cases.write_checkpoint(tmp_path, cfg, w), "float32", "cpu")
    a = cases.tokens(260, 90, seed=2)
    b = [(a[0] + 1) % 90] + a[1:]                              # the same tokens but for the first
    want_a, want_b = tc.expected(cfg, w, a), tc.expected(cfg, w, b)
    assert cases.worst(want_b[200:], want_a[200:]) > 1e-3
    for toks, want in ((a, want_a), (b, want_b)):
        got = cases.run_schedule(build_engine(m, 320), {"a": toks}, [{"a": c} for c in (100, 2, 64, 61)] + [{"a": 1}] * 33)["a"]
        assert cases.worst(got, want) < 2e-5


# ---- generation and serving -----------------------------------------------------------------------------------------------------------
def greedy_reference(cfg, w, prompt, n):
    out = list(prompt)
    for _ in range(n):
        out.append(int(tc.expected(cfg, w, out)[-1].argmax()))
    return out[len(prompt):]


def test_greedy_generation_through_generate_and_the_engine(checkpoint, model):
    _, cfg, w = checkpoint
    prompts = [cases.tokens(n, cfg["vocab"], seed=30 + n) for n in (40, 1, 66)]
    want = [greedy_reference(cfg, w, p, 5) for p in prompts]
    for kw in (dict(), dict(chunk_prefill_size=17), dict(use_cuda_graph=True)):
        out = model.generate(prompts, max_new_tokens=5, do_sample=False, eos_token_id=None, **kw)
        assert [o[len(p):] for o, p in zip(out, prompts)] == want, kw
    for burst, blocks in ((0, None), (4, None), (4, 3)):
        engine = ServingEngine(model, max_num_seqs=2, max_model_len=128, num_blocks=blocks, max_prefill_tokens=25, eos_token_id=None,
                               decode_burst=burst)
        reqs = [engine.add_request(f"r{i}", p, SamplingParams(max_tokens=5, temperature=0.0)) for i, p in enumerate(prompts)]
        engine.run_until_idle()
        assert [r.output for r in reqs] == want, (burst, blocks)
        assert engine.counters["mixed_steps"] >= 3 and engine.stats()["free_blocks"] == engine.stats()["total_blocks"]


def test_shared_prefixes_carry_their_states(checkpoint, model):
    """A shared prefix gives the same tokens; drafts, which take tokens back, are refused."""
    _, cfg, w = checkpoint
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
    want = tc.expected(cfg, w, toks)
    assert not os.path.exists(tmp_path / "0.f32")
    for step, rows in ((1, [20, 28]), (2, [29])):
        got = np.fromfile(tmp_path / f"{step}.f32", dtype="<f4").reshape(len(rows), -1)
        assert cases.worst(torch.from_numpy(got), want[rows]) < 1e-4


def test_command_line_predict(checkpoint, tmp_path):
    path, cfg, w = checkpoint
    yaml = tmp_path / "p.yaml"
    yaml.write_text("run_mode: predict\nuse_parallel: false\nuse_legacy: false\noutput_dir: " + str(tmp_path) + "\n"
                    "trainer: {type: CausalLanguageModelingTrainer, model_name: Togalorn}\n"
                    "processor: {tokenizer: {type: ByteTokenizer}}\n")
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    env = dict(os.environ, CUDA_VISIBLE_DEVICES="")
    res = subprocess.run([sys.executable, os.path.join(root, "run_mindformer.py"), "--config", str(yaml), "--run_mode", "predict",
                          "--pretrained_model_dir", path, "--predict_data", "abc", "--save_file", str(tmp_path / "out.txt")],
                         capture_output=True, text=True, timeout=300, env=env, cwd=str(tmp_path))
    assert res.returncode == 0 and "abc" in (tmp_path / "out.txt").read_text(), res.stdout[-1500:] + res.stderr[-3000:]
