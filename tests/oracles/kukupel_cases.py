"""Small configurations for the Kukupel tests."""
import copy

import torch

from . import cases, kukupel


def delta(heads=4, kv_heads=2, dim=32, vdim=48, conv=4):
    return dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv)


def attention(heads=4, kv_heads=2, dim=32, vdim=40, scale=0.3, softcap=6.0):
    return dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, softcap=softcap)


def moe(experts=4, top=2, ff=72, limit=1.5):
    return dict(kind="moe", router=dict(experts=experts, top=top), expert=dict(ff=ff, limit=limit))


def layer(mixer=None, left=None, mlp="default", scales=(0.7, 0.45)):
    """A delta layer, or with ``left`` a parallel one."""
    mixer = mixer or delta()
    if left:
        mixer = dict(left=left, right=mixer, left_scale=scales[0], right_scale=scales[1])
    return dict(type="parallel" if left else "delta", mixer=mixer, mlp=moe() if mlp == "default" else mlp)


def config(layers, width=160, vocab=211, streams=3, eps=1e-5):
    return dict(architecture="Kukupel", vocab=vocab, width=width, streams=streams, norm=dict(eps=eps), layers=copy.deepcopy(layers))


# Routers that choose among experts make 16-bit runs differ where two scores are close; configurations whose routers take
# every expert (top == experts) have no such places.
CASES = {
    # every size differs from every other; query / key heads shared in both mixers; a layer without a feed-forward
    "mixed_layers": config([layer(delta(6, 3, 40, 24, 3), attention(6, 2, 48, 32, 0.2, 4.0), moe(5, 5, 64, 1.0)),
                            layer(delta(4, 2, 64, 40, 5), mlp=None),
                            layer(delta(3, 1, 32, 56, 2), mlp=moe(3, 3, 40, 0.8)),
                            layer(delta(8, 8, 16, 16, 4), attention(4, 4, 24, 56, 0.35, 30.0), moe(2, 2, 88, 2.0), (1.3, 0.8))]),
    # tensor-core head sizes, aligned experts
    "wide_heads": config([layer(delta(4, 2, 128, 128, 4), attention(8, 2, 128, 128, 0.09, 20.0), moe(4, 4, 128, 7.0)),
                          layer(delta(2, 2, 128, 64, 4), mlp=moe(2, 2, 192, 1.0))], width=256, vocab=264, streams=4, eps=1e-3),
    # chosen experts; one key head for all; one stream; one tap
    "chosen_experts": config([layer(delta(5, 1, 24, 32, 1), attention(5, 1, 64, 64, 0.12, 9.0), moe(8, 1, 64, 1.0)),
                              layer(delta(2, 1, 96, 32, 2), mlp=moe(7, 3, 96, 1.0))], width=128, vocab=515, streams=1),
    # sizes that no vector access, tensor-core kernel or one-kernel decode step takes; five streams
    "odd_sizes": config([layer(delta(3, 1, 20, 36, 4), attention(3, 1, 20, 36, 0.25, 5.0), moe(3, 3, 50, 1.2)),
                         layer(delta(2, 1, 7, 5, 3), mlp=moe(2, 2, 33, 0.9)),
                         layer(delta(1, 1, 200, 176, 6), attention(2, 2, 144, 12, 0.1, 8.0), moe(4, 4, 20, 1.0))], width=100,
                        vocab=77, streams=5),
}
RANKS = {"mixed_layers": (12, 20), "wide_heads": (128, 64), "chosen_experts": (8, 8), "odd_sizes": (5, 11)}


def weights(name, seed=0, **kw):
    return kukupel.random_weights(CASES[name], seed, RANKS[name], **kw)


def expected(cfg, w, toks):
    return kukupel.forward(cfg, w, toks, torch.float64)


def greedy_is_right(cfg, w, prompt, out, slack):
    """Every generated token is the plain implementation's best one, up to rounding."""
    logits = expected(cfg, w, prompt + out)[len(prompt) - 1:-1]
    best = logits.max(-1).values
    took = logits[torch.arange(len(out)), torch.tensor(out)]
    return float((best - took).max()) <= slack * float(logits.std())


def errors(got, want):
    """Per position: root mean square over the vocabulary of the difference with its mean taken off, relative to the spread of
    the wanted logits."""
    d = got.double() - want
    d = d - d.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / want.std()


def rounding(cfg, w, toks, dtype):
    """What rounding alone does to the logits of the plain implementation: 32-bit arithmetic, or 16-bit inputs of every
    matrix product."""
    if dtype == "float32":
        return errors(kukupel.forward(cfg, w, toks, torch.float32), expected(cfg, w, toks))
    real = kukupel.linear
    kukupel.linear = lambda x, m: real(x.to(torch.bfloat16).to(x.dtype), m)
    try:
        return errors(expected(cfg, w, toks), real_expected(real, cfg, w, toks))
    finally:
        kukupel.linear = real


def real_expected(linear, cfg, w, toks):
    kept, kukupel.linear = kukupel.linear, linear
    try:
        return expected(cfg, w, toks)
    finally:
        kukupel.linear = kept


def close_calls(cfg, w, toks, gap):
    """Positions at which some router's choice rests on a score difference below ``gap`` (and all later positions, whose
    states those enter): where 16-bit runs may take another expert."""
    hit = torch.zeros(len(toks), dtype=torch.bool)
    seen = []
    real = kukupel.feed_forward

    def watch(h, get, m):
        s = torch.sigmoid(kukupel.linear(h, get("router"))).sort(dim=-1, descending=True).values
        top, n = m["router"]["top"], m["router"]["experts"]
        if top < n:
            seen.append(s[:, top - 1] - s[:, top] < gap)
        return real(h, get, m)
    kukupel.feed_forward = watch
    try:
        expected(cfg, w, toks)
    finally:
        kukupel.feed_forward = real
    for s in seen:
        hit |= s
    return hit.cumsum(0) > 0


__all__ = ["CASES", "RANKS", "attention", "cases", "close_calls", "config", "delta", "errors", "expected", "greedy_is_right", "layer", "moe",
           "rounding", "weights"]
