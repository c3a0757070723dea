"""Small configurations for the Gavatar tests."""
import copy

import torch

from . import cases, gavatar


def moe(experts=4, top=2, ff=72):
    return dict(kind="moe", router=dict(experts=experts, top=top), expert=dict(ff=ff))


def _layer(kind, mixer, mlp):
    return dict(type=kind, mixer=mixer, mlp=moe() if mlp == "default" else mlp)


def attention(heads=4, kv_heads=2, dim=32, vdim=40, scale=1.5, window=37, mlp="default"):
    return _layer("attention", dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, mask=dict(size=window)), mlp)


def latent(heads=4, dim=24, vdim=32, q_rank=56, kv_rank=48, scale=0.3, window=50, mlp="default"):
    return _layer("latent_attention", dict(heads=heads, dim=dim, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank, scale=scale,
                                           mask=dict(size=window)), mlp)


def mlstm(heads=3, dim=16, vdim=24, cap=7.0, mlp="default"):
    return _layer("mlstm", dict(heads=heads, dim=dim, vdim=vdim, gate_cap=cap), mlp)


def config(layers, width=160, vocab=211, eps=1e-5, scale=3.0, loop=None):
    return dict(architecture="Gavatar", vocab=vocab, width=width, norm=dict(eps=eps), embedding=dict(scale=scale),
                loop=None if loop is None else dict(start=loop[0], stop=loop[1], times=loop[2]), layers=copy.deepcopy(layers))


# Routers that choose among experts make 16-bit runs differ where two logits are close; configurations whose routers take
# every expert (top == experts) have no such places.
CASES = {
    # every size differs from every other; a loop in the middle; a layer without a feed-forward
    "mixed_layers": config([mlstm(6, 40, 24, 9.0, moe(5, 5, 64)), attention(6, 2, 48, 32, 1.2, 45, None),
                            latent(5, 40, 24, 72, 136, 0.25, 70, moe(3, 3, 40)), attention(8, 4, 24, 56, 0.9, 100, moe(2, 2, 88)),
                            mlstm(2, 64, 80, 5.0, None)], loop=(1, 3, 3)),
    # tensor-core head sizes, aligned experts; the whole stack runs twice
    "wide_heads": config([latent(8, 128, 128, 192, 512, 0.09, 200, moe(4, 4, 128)), mlstm(2, 128, 256, 15.0, moe(2, 2, 192)),
                          attention(8, 2, 128, 128, 1.0, 150, moe(2, 2, 64))], width=256, vocab=264, eps=1e-3, scale=16.0,
                         loop=(0, 3, 2)),
    # chosen experts; one key / value head, one head; windows of one token and beyond the sequence; no loop
    "chosen_experts": config([attention(5, 1, 64, 64, 0.8, 1, moe(8, 1, 64)), latent(1, 32, 96, 24, 64, 0.3, 4000, moe(7, 3, 96)),
                              attention(1, 1, 32, 16, 1.0, 500, None), mlstm(1, 96, 32, 3.0, moe(6, 2, 40))], width=128, vocab=515,
                             scale=1.0),
    # sizes that no vector access and no tensor-core kernel takes; a loop of one pass at the end
    "odd_sizes": config([mlstm(3, 20, 36, 8.0, moe(3, 3, 50)), attention(3, 3, 20, 36, 1.1, 33, moe(2, 2, 33)),
                         latent(3, 13, 11, 17, 29, 0.3, 64, moe(4, 4, 20)), mlstm(2, 7, 5, 4.0, None),
                         attention(2, 2, 144, 12, 1.3, 90, None)], width=101, vocab=77, loop=(2, 5, 1)),
}


def weights(name, seed=0, **kw):
    return gavatar.random_weights(CASES[name], seed, **kw)


def expected(cfg, w, toks):
    return gavatar.forward(cfg, w, toks, torch.float64)


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
    want = expected(cfg, w, toks)
    if dtype == "float32":
        return errors(gavatar.forward(cfg, w, toks, torch.float32), want)
    real = gavatar.linear
    gavatar.linear = lambda x, m: real(x.to(torch.bfloat16).to(x.dtype), m).to(torch.bfloat16).to(x.dtype)
    try:
        return errors(expected(cfg, w, toks), want)
    finally:
        gavatar.linear = real


def close_calls(cfg, w, toks, gap):
    """Positions at which some router's choice rests on a logit difference below ``gap`` (and all later positions, whose
    states and windows those enter): where 16-bit runs may take another expert."""
    hit = torch.zeros(len(toks), dtype=torch.bool)
    real = gavatar.router

    def watch(h, get, top):
        z = (gavatar.linear(h, get("router")) + get("router.b")).sort(dim=-1, descending=True).values
        if top < z.shape[1]:
            hit.logical_or_(z[:, top - 1] - z[:, top] < gap)
        return real(h, get, top)
    gavatar.router = watch
    try:
        expected(cfg, w, toks)
    finally:
        gavatar.router = real
    return hit.cumsum(0) > 0


__all__ = ["CASES", "attention", "cases", "close_calls", "config", "errors", "expected", "greedy_is_right", "latent", "mlstm", "moe",
           "rounding", "weights"]
