"""Small configurations for the Togalorn tests."""
import copy

import torch

from . import cases, togalorn


def moe(experts=4, identity=2, top=2, ff=72, limit=1.0, shared_ff=56, shared_limit=0.8):
    return dict(kind="moe", router=dict(experts=experts, identity=identity, top=top), expert=dict(ff=ff, limit=limit),
                shared=dict(ff=shared_ff, limit=shared_limit))


def _layer(kind, mixer, mlp):
    return dict(type=kind, mixer=mixer, mlp=moe() if mlp == "default" else mlp)


def latent(heads=4, dim=24, rot=8, vdim=32, q_rank=56, kv_rank=48, scale=0.4, base=300.0, mlp="default"):
    return _layer("latent_attention", dict(heads=heads, dim=dim, rot_dim=rot, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank, scale=scale,
                                           rot=dict(base=base, dims=rot)), mlp)


def mamba(heads=6, vdim=16, state=24, groups=2, conv=4, norm_groups=3, mlp="default"):
    return _layer("mamba2", dict(heads=heads, vdim=vdim, state=state, groups=groups, conv=conv, norm_groups=norm_groups), mlp)


def config(layers, width=160, vocab=211, eps=1e-5, groups=2, taps=4, scale=3.0, loop=None):
    return dict(architecture="Togalorn", vocab=vocab, width=width, norm=dict(eps=eps, groups=groups), canon=dict(taps=taps),
                embedding=dict(scale=scale), loop=None if loop is None else dict(start=loop[0], stop=loop[1], times=loop[2]),
                layers=copy.deepcopy(layers))


# Routers that choose among experts make 16-bit runs differ where two logits are close; configurations whose routers take
# every expert (top == experts + identity) have no such places.
CASES = {
    # every size differs from every other; a loop in the middle; layers without a feed-forward; one and several identity experts
    "mixed_layers": config([mamba(6, 24, 40, 3, 4, 2, moe(3, 1, 4, 64, 0.7, 88, 1.2)), latent(5, 40, 16, 32, 72, 136, 0.25, 50.0, None),
                            mamba(4, 40, 16, 1, 2, 5, moe(2, 3, 5, 40, 2.0, 24, 0.5)),
                            latent(8, 24, 8, 56, 48, 64, 0.5, 1000.0, moe(2, 1, 3, 88, 1.1, 136, 0.9)), mamba(3, 32, 56, 3, 3, 1, None)],
                           groups=5, taps=3, loop=(1, 3, 3)),
    # tensor-core head sizes, aligned experts; the whole stack runs twice
    "wide_heads": config([latent(8, 96, 32, 128, 192, 512, 0.15, 10000.0, moe(3, 1, 4, 128, 1.0, 256, 1.0)),
                          mamba(8, 64, 128, 2, 4, 4, moe(1, 2, 3, 192)), latent(20, 64, 64, 64, 128, 256, 0.1, 500.0, moe(2, 0, 2, 64)),
                          mamba(4, 128, 256, 1, 3, 1, None)], width=256, vocab=264, eps=1e-3, groups=2, taps=4, scale=16.0, loop=(0, 4, 2)),
    # chosen experts; one head, one group, one part, one tap; no loop
    "chosen_experts": config([latent(1, 32, 2, 96, 24, 64, 0.5, 7.0, moe(7, 2, 3, 96)), mamba(1, 96, 32, 1, 1, 1, moe(8, 4, 1, 64)),
                              mamba(8, 64, 64, 8, 4, 8, moe(6, 0, 2, 40))], width=128, vocab=515, groups=1, taps=1, scale=1.0),
    # sizes that no vector access and no tensor-core kernel takes; many taps; a loop of one pass at the end
    "odd_sizes": config([mamba(3, 7, 5, 1, 6, 1, moe(3, 1, 4, 50, 0.9, 33)), latent(3, 13, 6, 11, 17, 29, 0.4, 20.0, moe(2, 2, 4, 33)),
                         mamba(6, 5, 20, 3, 3, 2, None), latent(2, 130, 14, 12, 40, 50, 0.1, 90.0, moe(1, 1, 2, 20))], width=105, vocab=77,
                        groups=3, taps=6, loop=(2, 4, 1)),
}


def weights(name, seed=0, **kw):
    return togalorn.random_weights(CASES[name], seed, **kw)


def expected(cfg, w, toks):
    return togalorn.forward(cfg, w, toks, torch.float64)


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
        return errors(togalorn.forward(cfg, w, toks, torch.float32), want)
    real = togalorn.linear
    togalorn.linear = lambda x, m: real(x.to(torch.bfloat16).to(x.dtype), m).to(torch.bfloat16).to(x.dtype)
    try:
        return errors(expected(cfg, w, toks), want)
    finally:
        togalorn.linear = real


def close_calls(cfg, w, toks, gap):
    """Positions at which some router's choice rests on a difference below ``gap`` (and all later positions, whose states those
    enter): where 16-bit runs may take another expert."""
    hit = torch.zeros(len(toks), dtype=torch.bool)
    real = togalorn.router

    def watch(h, get, top):
        z = torch.softmax(togalorn.linear(h, get("router")), dim=-1) + get("correction")
        z = z.sort(dim=-1, descending=True).values
        if top < z.shape[1]:
            hit.logical_or_(z[:, top - 1] - z[:, top] < gap)
        return real(h, get, top)
    togalorn.router = watch
    try:
        expected(cfg, w, toks)
    finally:
        togalorn.router = real
    return hit.cumsum(0) > 0


__all__ = ["CASES", "cases", "close_calls", "config", "errors", "expected", "greedy_is_right", "latent", "mamba", "moe", "rounding",
           "weights"]
