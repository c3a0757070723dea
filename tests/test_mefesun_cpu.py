"""Mefesun on the host side: configuration and registry, checkpoint names and loading, per-layer caches, scheduling through
the engine and the trace replay, against the plain implementation of ``oracles/mefesun.py`` (CPU bodies of the ops)."""
import io
import json
import math
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

from mindformers_b200.checkpoint import name_maps
from mindformers_b200.inference.ragged_attention import prefill_work
from mindformers_b200.models import AutoConfig, AutoModel, MefesunConfig, MefesunForCausalLM
from mindformers_b200.ops import build as kernels
from mindformers_b200.ops import stream
from mindformers_b200.parallel.layers.rotary import RotaryFrequencies
from mindformers_b200.serving import SamplingParams, ServingEngine
from mindformers_b200.serving.trace import build_engine, replay

from oracles import cases, mefesun


@pytest.fixture(scope="module")
def checkpoint(tmp_path_factory):
    cfg = cases.CASES["mixed_layers"]
    w = mefesun.random_weights(cfg, seed=3)
    return cases.write_checkpoint(tmp_path_factory.mktemp("mefesun"), cfg, w), cfg, w


@pytest.fixture(scope="module")
def model(checkpoint):
    return cases.load(checkpoint[0], "float32", "cpu")


def test_config_resolves_by_architecture_and_describes_every_layer(checkpoint):
    path, cfg, _ = checkpoint
    config = AutoConfig.from_pretrained(path)
    assert isinstance(config, MefesunConfig)
    m = AutoModel.from_config(config, device="cpu", dtype="float32")
    assert isinstance(m, MefesunForCausalLM)
    tc = m.config
    assert tc.num_layers == len(cfg["layers"]) and tc.layer_sharing == [0, 1, 2, 1, 0]
    assert m.model.decoder.num_runs == 5 and len(m.model.decoder.layers) == 3
    for i, layer in enumerate(cfg["layers"]):
        c, mix = tc.for_layer(i), layer["mixer"]
        assert (c.num_attention_heads, c.num_query_groups, c.kv_channels, c.v_channels, c.attention_chunk_size, c.rotary_dim) == (
            mix["heads"], mix["kv_heads"], mix["dim"], mix["vdim"], mix["mask"]["size"], mix["rot"]["dims"])
        assert c.softmax_scale == mix["scale"] and c.ffn_hidden_size == (layer["mlp"]["ff"] if layer["mlp"] else 0)
    assert m.model.decoder.layers[1].mlp is None
    loop = [dict(cfg["layers"][0], weights_of=1), dict(cfg["layers"][0], weights_of=0)]
    with pytest.raises(ValueError, match="circle"):
        MefesunConfig(**dict(cfg, layers=loop)).to_transformer_dict()
    ahead = [dict(cfg["layers"][0], weights_of=1), cfg["layers"][0]]
    assert MefesunConfig(**dict(cfg, layers=ahead)).to_transformer_dict()["layer_sharing"] == [1, 1]
    with pytest.raises(ValueError, match="unknown mixer"):
        MefesunConfig(**dict(cfg, layers=[dict(cfg["layers"][0], type="other")])).to_transformer_dict()


def test_checkpoint_names_round_trip(checkpoint, model, tmp_path):
    path, cfg, w = checkpoint
    own = dict(model.named_parameters())
    fw = name_maps.hf_to_framework(w, model.config, "mefesun")
    assert set(fw) == set(own)
    for n, t in fw.items():
        assert torch.equal(own[n].detach(), t.float()), n
    back = name_maps.framework_to_hf({n: p.detach() for n, p in own.items()}, model.config, "mefesun")
    assert set(back) == set(w) and all(torch.equal(back[n], w[n].float()) for n in w)
    model.save_pretrained(str(tmp_path), hf_names=True)
    again = AutoModel.from_pretrained(str(tmp_path), dtype="float32", device="cpu", strict=True)
    assert all(torch.equal(a, b) for a, b in zip(again.parameters(), model.parameters()))
    with pytest.raises(KeyError):
        name_maps.convert_name("l0.mix.unknown", "mefesun")
    missing = {k: v for k, v in w.items() if k != "l1.mix.sink"}
    with pytest.raises(KeyError, match="sink"):
        AutoModel.from_pretrained(cases.write_checkpoint(tmp_path / "cut", cfg, missing), dtype="float32", device="cpu", strict=True)


@pytest.mark.parametrize("dims,base,factor,original,fast,slow", [(16, 300.0, 2.5, 20, 16.0, 1.0), (64, 1e6, 40.0, 4096, 32.0, 1.0),
                                                               (12, 5000.0, 1.0, 64, 8.0, 2.0), (8, 50.0, 3.0, 4, 1.0, 0.01)])
def test_yarn_frequencies(dims, base, factor, original, fast, slow):
    """Also where the ramp is empty (its bounds cross) and where it reaches past the last pair."""
    r = RotaryFrequencies(dims, base, dict(type="yarn", factor=factor, original_max_position_embeddings=original, beta_fast=fast,
                                           beta_slow=slow), device="cpu")
    want, amp = mefesun.yarn_frequencies(dims, base, dict(factor=factor, original=original, fast=fast, slow=slow))
    assert np.allclose(r.freqs.numpy(), want, rtol=1e-6) and math.isclose(r.amplitude, amp)
    plain = RotaryFrequencies(dims, base, None, device="cpu")
    assert np.allclose(plain.freqs.numpy(), mefesun.rotary_frequencies(dims, base), rtol=1e-6) and plain.amplitude == 1.0


def test_prefill_work_covers_every_row_once():
    q, ctx = [1, 300, 0, 129, 2], [5, 300, 9, 700, 130]
    for chunk in (0, 64, 200):
        items = prefill_work(q, ctx, chunk)
        assert sorted(items) == [(1, 1, 128, 0), (1, 129, 128, 128), (1, 257, 44, 256), (3, 301, 128, 571), (3, 429, 1, 699),
                                 (4, 430, 2, 128)]
    assert prefill_work(q, ctx, 0)[0][0] == 3                                # the rows that see the most keys come first


def test_norm_bodies():
    g = torch.Generator().manual_seed(0)
    x, y = torch.randn(3, 40, generator=g), torch.randn(3, 40, generator=g) + 1
    w, b, ls, bias = (torch.randn(40, generator=g) for _ in range(4))
    _, s = stream.add_normed(x, y, bias, w, b, ls, 1e-3, True)
    assert torch.allclose(s, x + ls * mefesun.layer_norm(y + bias, w, b, 1e-3), atol=1e-5)
    _, s = stream.add_normed(x, y, None, w, None, None, 1e-3, False)
    assert torch.allclose(s, x + mefesun.rms_norm(y, w, 1e-3), atol=1e-5)


def test_schedules_give_the_same_logits(checkpoint, model):
    _, cfg, w = checkpoint
    toks = {r: cases.tokens(n, cfg["vocab"], seed=n) for r, n in (("a", 90), ("b", 1), ("c", 75), ("d", 52), ("e", 20))}
    want = {r: cases.expected(cfg, w, t) for r, t in toks.items()}
    whole = [{r: len(t)} for r, t in toks.items()]
    cut = [{r: c} for r, t in toks.items() for c in cases.portions(len(t), (2, 31, 1, 19))]
    mixed = [{"a": 20, "b": 1, "c": 2, "d": 30}, {"a": 2, "c": 72}, {"a": 1, "e": 18, "d": 21}, {"c": 1, "e": 2, "a": 67}, {"d": 1}]
    for schedule, pool in ((whole, 128), (cut, 128), (mixed, 384)):
        got = cases.run_schedule(build_engine(model, pool), toks, schedule)
        for r in toks:
            assert cases.worst(got[r], want[r]) < 2e-5, (r, schedule[0])


def test_layer_outputs_follow_the_plain_implementation(checkpoint, model):
    """The stream after every layer run, layers that share weights included (each run has a cache of its own)."""
    _, cfg, w = checkpoint
    toks, trace, seen = cases.tokens(60, cfg["vocab"], seed=5), [], []
    mefesun.forward(cfg, w, toks, torch.float64, trace)
    hooks = [layer.register_forward_hook(lambda mod, args, out: seen.append(out[1].clone())) for layer in model.model.decoder.layers]
    logits = model(torch.tensor([toks]))
    for h in hooks:
        h.remove()
    assert len(seen) == len(trace) == 5
    for a, b in zip(seen, trace):
        assert torch.allclose(a.double(), b, atol=1e-4)
    assert cases.worst(logits, cases.expected(cfg, w, toks)) < 2e-5


def test_mistakes_would_show(checkpoint):
    """The checkpoint is sensitive: a chunk one position longer, no sink, another layer's weights, halves instead of pairs
    or no layer scale move the logits far beyond the limits used above."""
    _, cfg, w = checkpoint
    toks = cases.tokens(75, cfg["vocab"], seed=6)
    want = cases.expected(cfg, w, toks)

    def changed(edit_cfg=None, edit_w=None):
        c, v = json.loads(json.dumps(cfg)), dict(w)
        if edit_cfg:
            edit_cfg(c)
        if edit_w:
            edit_w(v)
        return cases.worst(cases.expected(c, v, toks), want)

    def chunk(c):
        c["layers"][0]["mixer"]["mask"]["size"] += 1
    assert changed(chunk) > 1e-2
    assert changed(None, lambda v: v.update({"l1.mix.sink": torch.full_like(v["l1.mix.sink"], -100)})) > 1e-2
    assert changed(lambda c: c["layers"].pop()) > 1e-2
    assert changed(None, lambda v: v.update({"l2.ls2": torch.ones_like(v["l2.ls2"])})) > 1e-2
    assert changed(lambda c: c["layers"][2]["mixer"]["rot"]["scaling"].update(factor=2.6)) > 1e-4


def greedy_reference(cfg, w, prompt, n):
    out = list(prompt)
    for _ in range(n):
        out.append(int(cases.expected(cfg, w, out)[-1].argmax()))
    return out[len(prompt):]


def test_greedy_generation_through_generate_and_the_engine(checkpoint, model):
    _, cfg, w = checkpoint
    prompts = [cases.tokens(n, cfg["vocab"], seed=30 + n) for n in (40, 1, 66)]
    want = [greedy_reference(cfg, w, p, 8) for p in prompts]
    for kw in (dict(), dict(chunk_prefill_size=17)):
        out = model.generate(prompts, max_new_tokens=8, do_sample=False, eos_token_id=None, **kw)
        assert [o[len(p):] for o, p in zip(out, prompts)] == want
    for burst in (0, 4):
        engine = ServingEngine(model, max_num_seqs=2, max_model_len=128, max_prefill_tokens=25, eos_token_id=None, decode_burst=burst)
        reqs = [engine.add_request(f"r{i}", p, SamplingParams(max_tokens=8, temperature=0.0)) for i, p in enumerate(prompts)]
        engine.run_until_idle()
        assert [r.output for r in reqs] == want
        assert engine.counters["mixed_steps"] >= 3 and engine.stats()["free_blocks"] == engine.stats()["total_blocks"]
    beams = model.generate(prompts[:1], max_new_tokens=4, num_beams=2, do_sample=False, eos_token_id=None)
    assert len(beams[0]) == len(prompts[0]) + 4


def test_command_line_predict(checkpoint, tmp_path):
    """``run_mindformer.py --run_mode predict`` on a model directory: greedy text of the plain implementation."""
    path, cfg, w = checkpoint
    yaml = tmp_path / "p.yaml"
    yaml.write_text("run_mode: predict\nuse_parallel: false\nuse_legacy: false\noutput_dir: " + str(tmp_path) + "\n"
                    "trainer: {type: CausalLanguageModelingTrainer, model_name: Mefesun}\n"
                    "processor: {tokenizer: {type: ByteTokenizer}}\n")
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    env = dict(os.environ, CUDA_VISIBLE_DEVICES="")
    res = subprocess.run([sys.executable, os.path.join(root, "run_mindformer.py"), "--config", str(yaml), "--run_mode", "predict",
                          "--pretrained_model_dir", path, "--predict_data", "abc", "--save_file", str(tmp_path / "out.txt")],
                         capture_output=True, text=True, timeout=300, env=env, cwd=str(tmp_path))
    assert res.returncode == 0 and "abc" in (tmp_path / "out.txt").read_text(), res.stdout[-1500:] + res.stderr[-3000:]


def test_sampling_is_seeded(model):
    engine = ServingEngine(model, max_num_seqs=2, max_model_len=64, eos_token_id=None)
    p = SamplingParams(max_tokens=6, temperature=0.8, top_k=20, seed=7)
    a, b = engine.generate([[1, 2, 3], [1, 2, 3]], p)
    assert a.token_ids == b.token_ids and len(a.token_ids) == 6


def test_pool_is_exact_and_given_back(model):
    engine = build_engine(model, 130)                                       # three blocks of 64 tokens
    assert engine.tables.pool.num_blocks == 3 and engine.ctx.key_cache[0].shape[0] == 3
    engine.attach("a")
    engine.advance({"a": list(range(120))}, {})
    engine.attach("b")
    engine.advance({"b": [1] * 60, "a": [2]}, {"b": []})
    assert engine.tables.pool.num_free == 0
    with pytest.raises(RuntimeError):
        engine.advance({"b": [1] * 5}, {})
    engine.detach("a")
    engine.detach("b")
    assert engine.tables.pool.num_free == 3
    for r in "abcd":
        engine.attach(r)
    with pytest.raises(RuntimeError, match="slots"):
        engine.attach("e")
    with pytest.raises(ValueError):
        engine.advance({"a": [0] * 500}, {})


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
    want = cases.expected(cfg, w, toks)
    assert not os.path.exists(tmp_path / "0.f32")
    got = np.fromfile(tmp_path / "1.f32", dtype="<f4").reshape(2, -1)
    assert cases.worst(torch.from_numpy(got), want[[20, 28]]) < 2e-5
    got = np.fromfile(tmp_path / "2.f32", dtype="<f4").reshape(1, -1)
    assert cases.worst(torch.from_numpy(got), want[[29]]) < 1e-4


def test_kernel_sources_of_the_model_exist():
    assert len(kernels._sources(MefesunForCausalLM.kernel_sources)) == len(MefesunForCausalLM.kernel_sources)
    with pytest.raises(ValueError, match="no kernel sources"):
        kernels._sources(("nonexistent",))


def test_tensor_parallel_ranks_give_the_same_logits(tmp_path):
    """Two gloo ranks: heads, sinks, feed-forward and vocabulary are sharded, everything else is replicated."""
    cfg = cases.config([cases.layer(4, 2, 16, 24, chunk=20, ff=64, rot=8), cases.layer(6, 2, 16, chunk=33, ff=96)], width=64, vocab=130)
    w = mefesun.random_weights(cfg, seed=11)
    path = cases.write_checkpoint(tmp_path / "m", cfg, w)
    toks = cases.tokens(50, cfg["vocab"], seed=1)
    torch.save(cases.expected(cfg, w, toks), tmp_path / "want.pt")
    script = os.path.join(os.path.dirname(os.path.abspath(__file__)), "dist", "run_layer_list_tp.py")
    res = subprocess.run([sys.executable, "-m", "torch.distributed.run", "--nnodes=1", "--nproc-per-node", "2", "--master-addr",
                          "127.0.0.1", "--master-port", "29671", script, path, str(tmp_path / "want.pt")],
                         capture_output=True, text=True, timeout=300)
    assert res.returncode == 0, res.stdout[-2000:] + res.stderr[-3000:]
