"""Kukupel on the host side: configuration and registry, checkpoint names and loading, states per slot, scheduling through
the engine and the trace replay, generation, tensor-parallel ranks, against the plain implementation of
``oracles/kukupel.py`` (CPU bodies of the ops)."""
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
from mindformers_b200.inference.weights_utils import tensor_shapes
from mindformers_b200.models import AutoConfig, AutoModel, KukupelConfig, KukupelForCausalLM
from mindformers_b200.ops import build as kernels
from mindformers_b200.ops import functional as Fn
from mindformers_b200.ops import recurrent, stream
from mindformers_b200.parallel.layers.transformer_layer import StreamTransformerLayer
from mindformers_b200.serving import SamplingParams, ServingEngine
from mindformers_b200.serving.trace import build_engine, replay

from oracles import cases, kukupel
from oracles import kukupel_cases as kc


@pytest.fixture(scope="module")
def checkpoint(tmp_path_factory):
    cfg = kc.CASES["mixed_layers"]
    w = kc.weights("mixed_layers", seed=3)
    return cases.write_checkpoint(tmp_path_factory.mktemp("kukupel"), cfg, w), cfg, w


@pytest.fixture(scope="module")
def model(checkpoint):
    return cases.load(checkpoint[0], "float32", "cpu")


# ---- configuration and weights ----------------------------------------------------------------------------------------------
def test_config_resolves_by_architecture_and_describes_every_layer(checkpoint):
    path, cfg, w = checkpoint
    config = AutoConfig.from_pretrained(path)
    assert isinstance(config, KukupelConfig)
    config.complete_from_checkpoint(tensor_shapes(path))
    m = AutoModel.from_config(config, device="cpu", dtype="float32")
    assert isinstance(m, KukupelForCausalLM)
    tc = m.config
    assert tc.num_layers == 4 and tc.residual_streams == 3 and tc.moe_layer_freq == [1, 0, 1, 1]
    for i, layer in enumerate(cfg["layers"]):
        c, mix, module = tc.for_layer(i), layer["mixer"], m.model.decoder.layers[i]
        assert isinstance(module, StreamTransformerLayer) and (module.mlp is None) == (layer["mlp"] is None)
        right = mix
        if layer["type"] == "parallel":
            a, right = mix["left"], mix["right"]
            assert (c.num_attention_heads, c.num_query_groups, c.kv_channels, c.v_channels, c.softmax_scale, c.attention_softcap) == (
                a["heads"], a["kv_heads"], a["dim"], a["vdim"], a["scale"], a["softcap"])
            assert c.parallel_scales == (mix["left_scale"], mix["right_scale"])
            assert (c.delta_decay_rank, c.delta_gate_rank) == kc.RANKS["mixed_layers"]
        assert (c.delta_heads, c.delta_kv_heads, c.delta_key_dim, c.delta_value_dim, c.delta_conv_taps) == (
            right["heads"], right["kv_heads"], right["dim"], right["vdim"], right["conv"])
        assert (c.delta_decay, c.delta_gate) == (("channel", "sigmoid") if layer["type"] == "parallel" else ("head", "silu"))
        if layer["mlp"]:
            r = layer["mlp"]["router"]
            assert (c.num_moe_experts, c.moe_router_topk, c.moe_ffn_hidden_size, c.moe_activation_limit) == (
                r["experts"], r["top"], layer["mlp"]["expert"]["ff"], layer["mlp"]["expert"]["limit"])
    assert m.model.decoder.cache_shapes() == [(2, 48, 32), None, None, (4, 24, 56)]
    assert m.model.decoder.state_shapes()[1] == (4, 64, 40, 2 * 2 * 64 + 4 * 40, 5)
    for bad, what in ((dict(cfg["layers"][0], type="other"), "unknown mixer"),
                      (dict(cfg["layers"][0], mlp=dict(kind="dense", ff=8)), "unknown feed-forward"),
                      (dict(cfg["layers"][0], mlp=kc.moe(2, 3)), "experts")):
        with pytest.raises(ValueError, match=what):
            KukupelConfig(**dict(cfg, layers=[bad])).to_transformer_dict()


def test_default_configuration_and_preset_build():
    assert KukupelConfig().to_transformer_dict()["num_layers"] == 4
    m = AutoModel.from_pretrained("tiny_kukupel", device="cpu", dtype="float32")
    assert isinstance(m, KukupelForCausalLM)
    assert torch.isfinite(m(torch.randint(0, 100, (2, 9)))).all()


def test_checkpoint_names_round_trip(checkpoint, model, tmp_path):
    path, cfg, w = checkpoint
    own = dict(model.named_parameters())
    fw = name_maps.hf_to_framework(w, model.config, "kukupel")
    assert set(fw) == set(own)
    for n, t in fw.items():
        assert torch.equal(own[n].detach(), t.float()), n
    back = name_maps.framework_to_hf({n: p.detach() for n, p in own.items()}, model.config, "kukupel")
    assert set(back) == set(w) and all(torch.equal(back[n], w[n].float()) for n in w)
    for kw in (dict(hf_names=True), dict(hf_names=False)):          # the design's own names, the framework's names
        model.save_pretrained(str(tmp_path / str(kw)), **kw)
        again = AutoModel.from_pretrained(str(tmp_path / str(kw)), dtype="float32", device="cpu", strict=True)
        assert all(torch.equal(a, b) for a, b in zip(again.parameters(), model.parameters()))
    with pytest.raises(KeyError, match="counterpart"):
        name_maps.hf_to_framework(dict(w, **{"l0.mix.right.unknown": w["final.norm"]}), model.config, "kukupel")
    missing = {k: v for k, v in w.items() if k != "l1.mix.A_log"}
    with pytest.raises(KeyError, match="a_log"):
        AutoModel.from_pretrained(cases.write_checkpoint(tmp_path / "cut", cfg, missing), dtype="float32", device="cpu", strict=True)


def test_kernel_sources_of_the_model_exist():
    assert len(kernels._sources(KukupelForCausalLM.kernel_sources)) == len(KukupelForCausalLM.kernel_sources)


# ---- single mechanisms --------------------------------------------------------------------------------------------------------
def test_residual_streams_step():
    g = torch.Generator().manual_seed(0)
    for n in (1, 2, 5):
        e, y, w = (torch.randn(*s, generator=g) for s in ((4, 24), (4, 24), (24,)))
        mix, write, read = torch.randn(n, n, generator=g), torch.randn(n, generator=g), torch.randn(n, generator=g)
        h, x = stream.residual_streams(e, n, None, None, None, read, w, 1e-3)
        assert x is e and torch.allclose(h, kukupel.rms_norm(read.sum() * e, w, 1e-3), atol=1e-5)
        xs = torch.stack([e] * n)
        for keep in (True, True, False):
            xs = kukupel.write_streams(xs, mix, write, y)
            h, x = stream.residual_streams(x, n, y, mix, write, read if keep else None, w, 1e-3, keep)
            u = kukupel.read_streams(xs, read) if keep else xs.sum(0)
            assert torch.allclose(h, kukupel.rms_norm(u, w, 1e-3), atol=1e-4)
            assert x is None if not keep else torch.allclose(x, xs.transpose(0, 1), rtol=1e-4, atol=1e-4)


def test_clamped_glu():
    x = torch.randn(5, 12, generator=torch.Generator().manual_seed(0)) * 3
    one = torch.eye(6, dtype=torch.float64)
    want = kukupel.expert(x.double(), torch.cat((one, 0 * one), 1), torch.cat((0 * one, one), 1), one, 0.8)
    assert torch.allclose(Fn.clamped_glu(x, 0.8, 1.702).double(), want, atol=1e-6)


def test_state_belongs_to_the_slot_and_needs_no_clearing():
    """A slot that held another sequence, a portion that starts at 0, and idle rows of a decode step."""
    m, eps = kc.delta(4, 2, 16, 12, 4), 1e-4
    g = torch.Generator().manual_seed(1)
    s = recurrent.DeltaShape(4, 2, 16, 12, 4, False, True)
    C, T = s.channels, 9
    w = recurrent.DeltaWeights(torch.randn(4, C, generator=g) * 0.5, torch.randn(4, generator=g), torch.randn(4, generator=g) - 2,
                               1 + 0.2 * torch.randn(12, generator=g))
    x, b, a, gate = (torch.randn(T, n, generator=g) for n in (C, 4, 4, 48))
    named = {"q.conv": w.conv[:, :32].t(), "k.conv": w.conv[:, 32:64].t(), "v.conv": w.conv[:, 64:].t(), "A_log": w.a_log,
             "dt_bias": w.dt_bias, "norm": w.norm, "o": torch.eye(48)}
    ident = {n: torch.zeros(r, C + 8 + 48) for n, r in (("q", 32), ("k", 32), ("v", 48), ("b", 4), ("a", 4), ("g", 48))}
    at = 0
    for n in ("q", "k", "v", "b", "a", "g"):
        ident[n][:, at:at + ident[n].shape[0]] = torch.eye(ident[n].shape[0])
        at += ident[n].shape[0]
    want = kukupel.delta(torch.cat((x, b, a, gate), 1), lambda n: {**named, **ident}[n], m, eps, False)
    ctx = KVCacheContext(1, 2, 64, 0, 0, torch.float32, "cpu", layer_shapes=[None], state_shapes=[(4, 16, 12, C, 4)], slots=3)
    for t in ctx.recurrent[0]:
        t.normal_(0, 5)                                                  # what earlier sequences left
    other = [t[[0, 2]].clone() for t in ctx.recurrent[0]]
    got, at = [], 0
    for n, prefill in ((1, True), (2, True), (3, True), (1, False), (1, False), (1, False)):
        lens = [7, at + n, 40]
        ctx.set_step(is_prefill=prefill, block_tables=np.zeros((3, 1)), slot_mapping=[0] * n if prefill else [-1, at, -1],
                     context_lens=lens, q_seq_lens=[0, n, 0] if prefill else [1] * 3, device="cpu")
        rows = [slice(at, at + n)] if prefill else [slice(0, 1), slice(at, at + 1), slice(0, 1)]
        pick = lambda t: torch.cat([t[r] for r in rows])
        o = recurrent.delta_rule(pick(x), pick(b), pick(a), pick(gate), w, s, ctx.recurrent[0], ctx, eps)
        got.append(o if prefill else o[1:2])
        at += n
    assert torch.allclose(torch.cat(got), want, atol=1e-5)
    assert all(torch.equal(t[[0, 2]], o) for t, o in zip(ctx.recurrent[0], other))


# ---- the whole model ---------------------------------------------------------------------------------------------------------------
SCHEDULES = (
    ([{"a": 90}, {"b": 1}, {"c": 75}, {"d": 52}, {"e": 20}], 128),
    ([{r: c} for r, n in (("a", 90), ("b", 1), ("c", 75), ("d", 52), ("e", 20)) for c in cases.portions(n, (2, 31, 1, 2, 19, 3))], 128),
    ([{"a": 20, "b": 1, "c": 2, "d": 30}, {"a": 2, "c": 72}, {"a": 1, "e": 18, "d": 21}, {"c": 1, "e": 2, "a": 67}, {"d": 1}], 384))


def test_schedules_give_the_same_logits(checkpoint, model):
    _, cfg, w = checkpoint
    toks = {r: cases.tokens(n, cfg["vocab"], seed=n) for r, n in (("a", 90), ("b", 1), ("c", 75), ("d", 52), ("e", 20))}
    want = {r: kc.expected(cfg, w, t) for r, t in toks.items()}
    for schedule, pool in SCHEDULES:
        got = cases.run_schedule(build_engine(model, pool), toks, schedule)
        for r in toks:
            assert cases.worst(got[r], want[r]) < 2e-5, (r, schedule[0])


@pytest.mark.parametrize("name", ["chosen_experts", "odd_sizes"])
def test_other_sizes(name, tmp_path):
    cfg, w = kc.CASES[name], kc.weights(name, seed=5)
    m = cases.load(cases.write_checkpoint(tmp_path, cfg, w), "float32", "cpu")
    toks = cases.tokens(40, cfg["vocab"], seed=1)
    got = cases.run_schedule(build_engine(m, 64), {"a": toks}, [{"a": 17}, {"a": 2}, {"a": 1}, {"a": 1}, {"a": 3}, {"a": 16}])
    assert cases.worst(got["a"], kc.expected(cfg, w, toks)) < 2e-5


def test_layer_outputs_follow_the_plain_implementation(checkpoint, model):
    """The sum of the streams after every layer (the layer's last output enters them in the next step)."""
    _, cfg, w = checkpoint
    toks, trace, seen = cases.tokens(30, cfg["vocab"], seed=5), [], []
    kukupel.forward(cfg, w, toks, torch.float64, trace)

    def after(mod, args, out):
        y, res, _ = out
        xs = res.x[:, None].expand(-1, 3, -1) if res.x.dim() == 2 else res.x
        seen.append((torch.einsum("sd,tsw->tdw", res.link.mix, xs) + res.link.write[:, None] * y[:, None]).sum(1))
    hooks = [layer.register_forward_hook(after) for layer in model.model.decoder.layers]
    logits = model(torch.tensor([toks]))
    for h in hooks:
        h.remove()
    assert len(seen) == len(trace) == 4
    for a, b in zip(seen, trace):
        assert torch.allclose(a.double(), b, rtol=1e-4, atol=1e-3)
    assert cases.worst(logits, kc.expected(cfg, w, toks)) < 2e-5


def test_mistakes_would_show(checkpoint, monkeypatch):
    """The checkpoint is sensitive: what a wrong state, tap, cap, stream or router would do moves the logits far beyond the
    limits used here."""
    _, cfg, w = checkpoint
    toks = cases.tokens(60, cfg["vocab"], seed=6)
    want = kc.expected(cfg, w, toks)

    def changed(edit_cfg=None, edit_w=None, patch=None):
        c, v = json.loads(json.dumps(cfg)), dict(w)
        if edit_cfg:
            edit_cfg(c)
        if edit_w:
            edit_w(v)
        with monkeypatch.context() as mp:
            for name, fn in (patch or {}).items():
                mp.setattr(kukupel, name, fn)
            return cases.worst(kc.expected(c, v, toks), want)
    scan, conv = kukupel.delta_scan, kukupel.short_conv

    def lost(q, k, v, beta, g):                               # the state is lost at token 30
        return torch.cat((scan(q[:30], k[:30], v[:30], beta[:30], g[:30]), scan(q[30:], k[30:], v[30:], beta[30:], g[30:])))

    def lost_conv(x, taps):
        return torch.cat((conv(x[:30], taps), conv(x[30:], taps)))

    def read_first(q, k, v, beta, g):                         # the read-out does not see the current token's write
        o = scan(q, k, v, beta, g)
        z = torch.zeros_like(v)
        for t in range(len(q)):
            z[t] = o[t] - (beta[t][:, None] * v[t]) * (q[t] * k[t]).sum(-1, keepdim=True)
        return z
    assert changed(patch=dict(delta_scan=lost)) > 1e-2
    assert changed(patch=dict(short_conv=lost_conv)) > 1e-2
    assert changed(patch=dict(delta_scan=read_first)) > 1e-2
    assert changed(patch=dict(capped=lambda s, cap: s)) > 1e-3
    assert changed(lambda c: c["layers"][0]["mixer"].update(right_scale=0.46)) > 1e-3
    assert changed(None, lambda v: v.update({"l1.hc1.mix": v["l1.hc1.mix"].t()})) > 1e-3
    assert changed(lambda c: c["layers"][0]["mlp"]["expert"].update(limit=1.1)) > 1e-3
    assert changed(None, lambda v: v.update({"l2.mlp.router": v["l2.mlp.router"] * 1.1})) > 1e-3
    assert changed(None, lambda v: v.update({"l0.mix.right.dt_bias": v["l0.mix.right.dt_bias"] + 0.1})) > 1e-3


def test_a_far_token_decides_and_is_found(tmp_path):
    """One head that keeps everything (decays of 1): a key written hundreds of tokens ago is read through portions and
    decoded tokens."""
    cfg = kc.config([kc.layer(kc.delta(2, 1, 16, 16, 1), mlp=None)], width=64, vocab=90, streams=2)
    w = kukupel.random_weights(cfg, seed=4, decay=(-30.0, 0.0))
    m = cases.load(cases.write_checkpoint(tmp_path, cfg, w), "float32", "cpu")
    a = cases.tokens(260, 90, seed=2)
    b = [(a[0] + 1) % 90] + a[1:]                              # the same tokens but for the first
    want_a, want_b = kc.expected(cfg, w, a), kc.expected(cfg, w, b)
    assert cases.worst(want_b[200:], want_a[200:]) > 1e-3
    for toks, want in ((a, want_a), (b, want_b)):
        got = cases.run_schedule(build_engine(m, 320), {"a": toks}, [{"a": c} for c in (100, 2, 64, 61)] + [{"a": 1}] * 33)["a"]
        assert cases.worst(got, want) < 2e-5


# ---- generation and serving -----------------------------------------------------------------------------------------------------------
def greedy_reference(cfg, w, prompt, n):
    out = list(prompt)
    for _ in range(n):
        out.append(int(kc.expected(cfg, w, out)[-1].argmax()))
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


def test_beams_carry_their_states(checkpoint, model):
    """The best beam scores what the plain implementation gives it."""
    _, cfg, w = checkpoint
    p = cases.tokens(20, cfg["vocab"], seed=3)
    out = model.generate([p], max_new_tokens=5, num_beams=3, do_sample=False, eos_token_id=None)[0]

    def score(seq):
        lp = torch.log_softmax(kc.expected(cfg, w, seq), dim=-1)
        return float(sum(lp[i - 1, seq[i]] for i in range(len(p), len(seq))))
    beams = [(0.0, p)]
    for _ in range(5):
        cand = []
        for s, seq in beams:
            lp = torch.log_softmax(kc.expected(cfg, w, seq)[-1], dim=-1)
            v, i = lp.topk(6)
            cand += [(s + float(a), seq + [int(b)]) for a, b in zip(v, i)]
        beams = sorted(cand, reverse=True)[:3]
    assert abs(score(out) - beams[0][0]) < 1e-4


def test_shared_prefixes_copy_states_and_drafts_are_refused(checkpoint, model):
    _, cfg, w = checkpoint
    head = cases.tokens(70, cfg["vocab"], seed=9)
    prompts = [head + [1, 2], head + [3], head + [4, 5, 6]]
    plain = model.generate(prompts, max_new_tokens=4, do_sample=False, eos_token_id=None)
    shared = model.generate(prompts, max_new_tokens=4, do_sample=False, eos_token_id=None, parallel_decoding="prefix_cache")
    assert shared == plain
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
    assert engine.ctx.recurrent[0][0].shape[0] == 4                          # a state for each of the four slots
    want = kc.expected(cfg, w, toks)
    assert not os.path.exists(tmp_path / "0.f32")
    for step, rows in ((1, [20, 28]), (2, [29])):
        got = np.fromfile(tmp_path / f"{step}.f32", dtype="<f4").reshape(len(rows), -1)
        assert cases.worst(torch.from_numpy(got), want[rows]) < 1e-4


def test_command_line_predict(checkpoint, tmp_path):
    path, cfg, w = checkpoint
    yaml = tmp_path / "p.yaml"
    yaml.write_text("run_mode: predict\nuse_parallel: false\nuse_legacy: false\noutput_dir: " + str(tmp_path) + "\n"
                    "trainer: {type: CausalLanguageModelingTrainer, model_name: Kukupel}\n"
                    "processor: {tokenizer: {type: ByteTokenizer}}\n")
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    env = dict(os.environ, CUDA_VISIBLE_DEVICES="")
    res = subprocess.run([sys.executable, os.path.join(root, "run_mindformer.py"), "--config", str(yaml), "--run_mode", "predict",
                          "--pretrained_model_dir", path, "--predict_data", "abc", "--save_file", str(tmp_path / "out.txt")],
                         capture_output=True, text=True, timeout=300, env=env, cwd=str(tmp_path))
    assert res.returncode == 0 and "abc" in (tmp_path / "out.txt").read_text(), res.stdout[-1500:] + res.stderr[-3000:]


def test_tensor_parallel_ranks_give_the_same_logits(tmp_path):
    """Two gloo ranks: heads, states, short convolutions, decays and vocabulary are sharded, low-rank factors and a single
    shared key head are replicated."""
    cfg = kc.config([kc.layer(kc.delta(4, 2, 16, 24, 3), kc.attention(4, 2, 16, 24), kc.moe(3, 2, 40)),
                     kc.layer(kc.delta(4, 1, 16, 8, 4), mlp=kc.moe(2, 2, 24))], width=64, vocab=130)
    w = kukupel.random_weights(cfg, seed=11)
    path = cases.write_checkpoint(tmp_path / "m", cfg, w)
    toks = cases.tokens(50, cfg["vocab"], seed=1)
    torch.save(kc.expected(cfg, w, toks), tmp_path / "want.pt")
    script = os.path.join(os.path.dirname(os.path.abspath(__file__)), "dist", "run_layer_list_tp.py")
    res = subprocess.run([sys.executable, "-m", "torch.distributed.run", "--nnodes=1", "--nproc-per-node", "2", "--master-addr",
                          "127.0.0.1", "--master-port", "29673", script, path, str(tmp_path / "want.pt")],
                         capture_output=True, text=True, timeout=300)
    assert res.returncode == 0, res.stdout[-2000:] + res.stderr[-3000:]
