"""Plain, slow implementation of the Mefesun design, one function per mechanism.

Everything runs on whole sequences of one request with dense masks; nothing is shared with the product code. ``cfg`` is
the ``config.json`` dictionary, ``w`` the checkpoint's tensors by name, both as a user would supply them. The dtype of
the arithmetic is the dtype the weights are converted to (float32 or float64).
"""
import math

import torch


def linear(x, w, b=None):
    y = x @ w.t()
    return y if b is None else y + b


def rms_norm(x, weight, eps):
    return x / torch.sqrt(torch.mean(x * x, dim=-1, keepdim=True) + eps) * weight


def layer_norm(x, weight, bias, eps):
    mean = x.mean(dim=-1, keepdim=True)
    dev = x - mean
    return dev / torch.sqrt((dev * dev).mean(dim=-1, keepdim=True) + eps) * weight + bias


def rotary_frequencies(dims, base):
    """Frequency of pair i: ``base ** (-2 i / dims)``."""
    return [base ** (-2.0 * i / dims) for i in range(dims // 2)]


def yarn_frequencies(dims, base, scaling):
    """Interpolated frequencies and the factor on cos and sin."""
    factor, original = scaling["factor"], scaling["original"]

    def boundary(turns):
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(boundary(scaling["fast"])), 0)
    hi = min(math.ceil(boundary(scaling["slow"])), dims - 1)
    out = []
    for i, f in enumerate(rotary_frequencies(dims, base)):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / factor * ramp + f * (1.0 - ramp))
    return out, 0.1 * math.log(factor) + 1.0


def rotate_pairs(x, positions, freqs, amplitude=1.0):
    """x [T, heads, dim]: dimensions (2i, 2i + 1) of the first ``2 * len(freqs)`` are rotated by position * freq_i."""
    y = x.clone()
    for i, f in enumerate(freqs):
        a = positions.to(torch.float64) * f
        c = (torch.cos(a) * amplitude).to(x.dtype)[:, None]
        s = (torch.sin(a) * amplitude).to(x.dtype)[:, None]
        u, v = x[:, :, 2 * i], x[:, :, 2 * i + 1]
        y[:, :, 2 * i] = u * c - v * s
        y[:, :, 2 * i + 1] = v * c + u * s
    return y


def chunk_mask(n, size):
    """[query, key]: causal, and both in the same chunk of ``size`` positions counted from 0."""
    q = torch.arange(n)[:, None]
    k = torch.arange(n)[None, :]
    return (k <= q) & (torch.div(q, size, rounding_mode="floor") == torch.div(k, size, rounding_mode="floor"))


def softmax_with_sink(scores, mask, sink):
    """scores [heads, q, k]; the denominator of head h also holds exp(sink[h])."""
    s = scores.masked_fill(~mask[None], float("-inf"))
    top = torch.maximum(s.max(dim=-1, keepdim=True).values, sink[:, None, None])
    e = torch.exp(s - top)
    return e / (e.sum(dim=-1, keepdim=True) + torch.exp(sink[:, None, None] - top))


def attention(h, get, mixer, eps):
    """The attention mixer on one whole sequence; ``get(name)`` returns the mixer's tensors (None when absent)."""
    T = h.shape[0]
    H, G, D, DV = mixer["heads"], mixer["kv_heads"], mixer["dim"], mixer["vdim"]
    q = linear(h, get("q"), get("q.b")).view(T, H, D)
    k = linear(h, get("k"), get("k.b")).view(T, G, D)
    v = linear(h, get("v"), get("v.b")).view(T, G, DV)
    q = rms_norm(q, get("q.norm"), eps)
    k = rms_norm(k, get("k.norm"), eps)
    rot = mixer["rot"]
    if rot.get("scaling"):
        freqs, amp = yarn_frequencies(rot["dims"], rot["base"], rot["scaling"])
    else:
        freqs, amp = rotary_frequencies(rot["dims"], rot["base"]), 1.0
    pos = torch.arange(T)
    q = rotate_pairs(q, pos, freqs, amp)
    k = rotate_pairs(k, pos, freqs, amp)
    reps = H // G
    kk = torch.stack([k[:, i // reps] for i in range(H)], dim=1)
    vv = torch.stack([v[:, i // reps] for i in range(H)], dim=1)
    scores = torch.einsum("qhd,khd->hqk", q, kk) * mixer["scale"]
    p = softmax_with_sink(scores, chunk_mask(T, mixer["mask"]["size"]), get("sink"))
    o = torch.einsum("hqk,khd->qhd", p, vv).reshape(T, H * DV)
    return linear(o, get("o"), get("o.b"))


def feed_forward(h, up, down):
    a = torch.relu(linear(h, up))
    return linear(a * a, down)


def softcap(x, cap):
    return cap * torch.tanh(x / cap)


def forward(cfg, w, tokens, dtype=torch.float64, trace=None):
    """Logits ``[T, vocab]`` of every position of one sequence; ``trace`` (a list) collects the stream after each layer."""
    t = {n: x.to(dtype) for n, x in w.items()}
    eps = cfg["norm"]["eps"]
    x = t["embed"][torch.as_tensor(tokens)]
    for i, layer in enumerate(cfg["layers"]):
        j = i
        while cfg["layers"][j].get("weights_of") is not None:
            j = cfg["layers"][j]["weights_of"]
        p = f"l{j}."
        y = attention(x, lambda n: t.get(p + "mix." + n), layer["mixer"], eps)
        x = x + layer_norm(y, t[p + "norm1"], t[p + "norm1.b"], eps) * t[p + "ls1"]
        if layer.get("mlp"):
            y = feed_forward(x, t[p + "mlp.up"], t[p + "mlp.down"])
            x = x + layer_norm(y, t[p + "norm2"], t[p + "norm2.b"], eps) * t[p + "ls2"]
        if trace is not None:
            trace.append(x)
    x = layer_norm(x, t["final.norm"], t["final.norm.b"], eps)
    return softcap(linear(x, t["embed"]), cfg["logit_softcap"])


def random_weights(cfg, seed=0, sink_scale=1.0):
    """A checkpoint of bfloat16 tensors with every tensor of the design away from its neutral value."""
    g = torch.Generator().manual_seed(seed)
    W = cfg["width"]

    def mat(n, k, gain=1.0):
        return torch.randn(n, k, generator=g) * gain / math.sqrt(k)

    def vec(n, mean=0.0, std=0.2):
        return mean + torch.randn(n, generator=g) * std

    w = {"embed": torch.randn(cfg["vocab"], W, generator=g), "final.norm": vec(W, 1.0), "final.norm.b": vec(W)}
    for i, layer in enumerate(cfg["layers"]):
        if layer.get("weights_of") is not None:
            continue
        m, p = layer["mixer"], f"l{i}."
        w[p + "mix.q"], w[p + "mix.q.b"] = mat(m["heads"] * m["dim"], W), vec(m["heads"] * m["dim"])
        w[p + "mix.k"], w[p + "mix.k.b"] = mat(m["kv_heads"] * m["dim"], W), vec(m["kv_heads"] * m["dim"])
        w[p + "mix.v"], w[p + "mix.v.b"] = mat(m["kv_heads"] * m["vdim"], W), vec(m["kv_heads"] * m["vdim"])
        w[p + "mix.q.norm"], w[p + "mix.k.norm"] = vec(m["dim"], 1.2), vec(m["dim"], 1.2)
        w[p + "mix.sink"] = vec(m["heads"], 1.0, sink_scale)
        w[p + "mix.o"], w[p + "mix.o.b"] = mat(W, m["heads"] * m["vdim"]), vec(W)
        w[p + "norm1"], w[p + "norm1.b"], w[p + "ls1"] = vec(W, 1.0), vec(W), vec(W, 0.7)
        if layer.get("mlp"):
            f = layer["mlp"]["ff"]
            w[p + "mlp.up"], w[p + "mlp.down"] = mat(f, W), mat(W, f)
            w[p + "norm2"], w[p + "norm2.b"], w[p + "ls2"] = vec(W, 1.0), vec(W), vec(W, 0.7)
    return {n: t.to(torch.bfloat16) for n, t in w.items()}
