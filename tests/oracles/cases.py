"""Small configurations for the Mefesun tests and helpers that feed a model in portions."""
import copy
import json
import os

import torch
from safetensors.torch import save_file

from . import mefesun


def layer(heads=4, kv_heads=2, dim=32, vdim=None, chunk=48, ff=160, rot=None, base=5000.0, scale=None, factor=4.0,
          original=64, fast=16.0, slow=1.0, mlp=True):
    rot = dim if rot is None else rot
    return dict(type="attention",
                mixer=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim or dim, scale=scale or dim ** -0.5,
                           mask=dict(size=chunk), rot=dict(base=base, dims=rot, scaling=dict(
                               factor=factor, original=original, fast=fast, slow=slow))),
                mlp=dict(kind="dense", ff=ff) if mlp else None)


def config(layers, width=192, vocab=300, cap=20.0, eps=1e-5):
    return dict(architecture="Mefesun", vocab=vocab, width=width, norm=dict(eps=eps), logit_softcap=cap,
                layers=copy.deepcopy(layers))


def shared(layers, order):
    """Append runs of the layers named in ``order`` with their weights."""
    out = copy.deepcopy(layers)
    for j in order:
        out.append(dict(copy.deepcopy(layers[j]), weights_of=j))
    return out


CASES = {
    # every size differs from every other; unequal key and value sizes; part of a head rotated; a layer without
    # feed-forward; a layer whose weights run again, not in order
    "mixed_layers": config(shared([layer(6, 2, 40, 24, chunk=50, ff=136, rot=16, scale=0.21), layer(3, 3, 32, 48, chunk=33, mlp=False),
                                   layer(8, 1, 16, 16, chunk=70, ff=72, rot=8, base=300.0, factor=2.5, original=20)], [1, 0]),
                           width=176, vocab=301),
    "wide_heads": config([layer(4, 2, 128, chunk=200, ff=264), layer(4, 4, 64, 128, chunk=96, ff=128, rot=32)], width=256,
                         vocab=264, cap=9.0, eps=1e-3),
    "one_kv_head": config([layer(5, 1, 64, chunk=130, ff=320, rot=48), layer(20, 1, 24, 40, chunk=64, ff=96)], width=128, vocab=515),
    # sizes that no tensor-core kernel takes
    "odd_sizes": config([layer(3, 1, 20, 36, chunk=21, ff=90, rot=12), layer(2, 2, 144, 12, chunk=40, ff=50)], width=100, vocab=77),
}


def write_checkpoint(path, cfg, weights):
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({k: v.contiguous() for k, v in weights.items()}, os.path.join(path, "model.safetensors"))
    return str(path)


def load(path, dtype, device):
    from mindformers_b200.models import AutoModel
    return AutoModel.from_pretrained(str(path), dtype=dtype, device=device, strict=True).eval()


def tokens(n, vocab, seed=0):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def run_schedule(engine, requests, schedule):
    """``requests``: {name: tokens}; ``schedule``: steps of {name: number of next tokens}. Returns {name: [T, vocab]}."""
    from mindformers_b200.serving.trace import run_step
    at = {r: 0 for r in requests}
    got = {r: [] for r in requests}
    for n, step in enumerate(schedule):
        entries, end = [], []
        for r, count in step.items():
            lo, hi = at[r], at[r] + count
            entries.append(dict(id=r, tokens=requests[r][lo:hi], want=list(range(count))))
            at[r] = hi
            if hi == len(requests[r]):
                end.append(r)
        out = run_step(engine, dict(step=n, entries=entries, end=end))
        pos = 0
        for r, count in step.items():
            got[r].append(torch.from_numpy(out[pos:pos + count]))
            pos += count
    return {r: torch.cat(v) for r, v in got.items()}


def portions(n, sizes):
    out, i = [], 0
    while n > 0:
        c = min(n, sizes[i % len(sizes)])
        out.append(c)
        n -= c
        i += 1
    return out


def worst(got, want):
    """Largest error over the positions: root mean square over the vocabulary of the difference with its mean taken off,
    relative to the spread of the wanted logits."""
    d = got.double() - want.double()
    d = d - d.mean(-1, keepdim=True)
    return float((d.pow(2).mean(-1).sqrt() / want.double().std()).max())


def expected(cfg, w, toks):
    return mefesun.forward(cfg, w, toks, torch.float64)
