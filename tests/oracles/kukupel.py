"""Plain, slow implementation of the Kukupel design, one function per mechanism.

Everything runs on whole sequences of one request, token by token where the design is recurrent; nothing is shared with
the product code. ``cfg`` is the ``config.json`` dictionary, ``w`` the checkpoint's tensors by name. The dtype of the
arithmetic is the dtype the weights are converted to (float32 or float64).
"""
import math

import torch


def linear(x, w):
    return x @ w.t()


def rms(x, eps):
    return x / torch.sqrt(torch.mean(x * x, dim=-1, keepdim=True) + eps)


def rms_norm(x, weight, eps):
    return rms(x, eps) * weight


def silu(x):
    return x * torch.sigmoid(x)


def softplus(x):
    return torch.log1p(torch.exp(-x.abs())) + torch.clamp(x, min=0)


# ---- residual streams ------------------------------------------------------------------------------------------------
def read_streams(xs, read):
    """xs [s, T, W]; the sub-layer's input is a weighted sum of the streams."""
    u = torch.zeros_like(xs[0])
    for s in range(xs.shape[0]):
        u = u + read[s] * xs[s]
    return u


def write_streams(xs, mix, write, y):
    """New streams, all from the old ones: mix[from, to], plus the sub-layer's output times write[to]."""
    out = []
    for t in range(xs.shape[0]):
        z = write[t] * y
        for s in range(xs.shape[0]):
            z = z + mix[s, t] * xs[s]
        out.append(z)
    return torch.stack(out)


# ---- softmax attention with capped scores, no positions -----------------------------------------------------------------
def capped(score, cap):
    return cap * torch.tanh(score / cap)


def attention(h, get, m):
    T, H, G, D, DV = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = linear(h, get("q")).view(T, H, D)
    k = linear(h, get("k")).view(T, G, D)
    v = linear(h, get("v")).view(T, G, DV)
    causal = torch.arange(T)[None, :] <= torch.arange(T)[:, None]
    heads = []
    for i in range(H):
        g = i // (H // G)
        s = capped(q[:, i] @ k[:, g].t() * m["scale"], m["softcap"])
        p = torch.softmax(s.masked_fill(~causal, float("-inf")), dim=-1)
        heads.append(p @ v[:, g])
    return linear(torch.cat(heads, dim=-1), get("o"))


# ---- gated delta rule -----------------------------------------------------------------------------------------------------
def short_conv(x, taps):
    """x [T, channels], taps [channels, n]: causal, the last tap belongs to the current token, zeros before the start."""
    n = taps.shape[1]
    padded = torch.cat((x.new_zeros(n - 1, x.shape[1]), x))
    out = torch.zeros_like(x)
    for j in range(n):
        out = out + padded[j:j + x.shape[0]] * taps[:, j]
    return out


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_scan(q, k, v, beta, decay):
    """q, k [T, H, D], v [T, H, DV], beta [T, H], decay [T, H, D] -> [T, H, DV]. State [H, D, DV] from zero."""
    T, H, D = q.shape
    S = q.new_zeros(H, D, v.shape[-1])
    out = []
    for t in range(T):
        S = S * decay[t][:, :, None]
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + torch.einsum("hd,hv->hdv", k[t], u)
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out)


def head_decay(h, get, heads, dim):
    """One decay per head."""
    g = torch.exp(-torch.exp(get("A_log")) * softplus(linear(h, get("a")) + get("dt_bias")))
    return g[:, :, None].expand(-1, -1, dim)


def channel_decay(h, get, heads, dim):
    """One decay per head and key channel, from a low-rank projection."""
    a = linear(linear(h, get("a1")), get("a2")) + get("dt_bias")
    return torch.exp(-torch.exp(get("A_log"))[None, :, None] * softplus(a).view(-1, heads, dim))


def delta(h, get, m, eps, by_channel):
    T, H, G, D, DV = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(short_conv(linear(h, get(n)), get(n + ".conv"))) for n in "qkv")
    rep = torch.arange(H) // (H // G)
    q = (unit(q.view(T, G, D)) * D ** -0.5)[:, rep]
    k = unit(k.view(T, G, D))[:, rep]
    beta = torch.sigmoid(linear(h, get("b")))
    g = (channel_decay if by_channel else head_decay)(h, get, H, D)
    o = rms_norm(delta_scan(q, k, v.view(T, H, DV), beta, g), get("norm"), eps)
    if by_channel:
        gate = torch.sigmoid(linear(linear(h, get("g1")), get("g2")))
    else:
        gate = silu(linear(h, get("g")))
    return linear((o * gate.view(T, H, DV)).reshape(T, H * DV), get("o"))


def parallel(h, get, m, eps):
    left = attention(h, lambda n: get("left." + n), m["left"])
    right = delta(h, lambda n: get("right." + n), m["right"], eps, True)
    return m["left_scale"] * left + m["right_scale"] * right


# ---- mixture of experts ------------------------------------------------------------------------------------------------------
def expert(h, gate, up, down, limit):
    g = torch.clamp(linear(h, gate), max=limit)
    u = torch.clamp(linear(h, up), -limit, limit)
    return linear(g * torch.sigmoid(1.702 * g) * (u + 1), down)


def feed_forward(h, get, m):
    n, top = m["router"]["experts"], m["router"]["top"]
    s = torch.sigmoid(linear(h, get("router")))
    best, ids = torch.topk(s, top, dim=-1)
    y = torch.zeros_like(h)
    for e in range(n):
        for j in range(top):
            rows = (ids[:, j] == e).nonzero()[:, 0]
            if len(rows):
                x = best[rows, j][:, None] * h[rows]
                y[rows] += expert(x, get(f"e{e}.gate"), get(f"e{e}.up"), get(f"e{e}.down"), m["expert"]["limit"])
    return y


def forward(cfg, w, tokens, dtype=torch.float64, trace=None):
    """Logits ``[T, vocab]`` of every position of one sequence; ``trace`` (a list) collects the sum of the streams after
    each layer."""
    t = {n: x.to(dtype) for n, x in w.items()}
    eps = cfg["norm"]["eps"]
    x = t["embed"][torch.as_tensor(tokens)]
    xs = torch.stack([x] * cfg["streams"])
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."

        def mix(h):
            get = lambda n: t[p + "mix." + n]
            if layer["type"] == "parallel":
                return parallel(h, get, layer["mixer"], eps)
            return delta(h, get, layer["mixer"], eps, False)

        def ff(h):
            return feed_forward(h, lambda n: t[p + "mlp." + n], layer["mlp"])
        for q, sub in ((1, mix), (2, ff if layer.get("mlp") else None)):
            if sub is None:
                continue
            u = read_streams(xs, t[f"{p}hc{q}.in"])
            y = sub(rms_norm(u, t[f"{p}norm{q}"], eps))
            xs = write_streams(xs, t[f"{p}hc{q}.mix"], t[f"{p}hc{q}.out"], y)
        if trace is not None:
            trace.append(xs.sum(0))
    return linear(rms_norm(xs.sum(0), t["final.norm"], eps), t["embed"])


# ---- random checkpoints -------------------------------------------------------------------------------------------------------
def random_weights(cfg, seed=0, ranks=(12, 20), decay=(-3.0, 1.0)):
    """A checkpoint of bfloat16 tensors with every tensor of the design away from its neutral value. ``ranks``: of the
    low-rank decay and gate; ``decay``: mean and spread of dt_bias (a low mean remembers long)."""
    g = torch.Generator().manual_seed(seed)
    W, n = cfg["width"], cfg["streams"]

    def mat(rows, cols, gain=1.0):
        return torch.randn(rows, cols, generator=g) * gain / math.sqrt(cols)

    def vec(size, mean=0.0, std=0.2):
        return mean + torch.randn(size, generator=g) * std

    w = {"embed": torch.randn(cfg["vocab"], W, generator=g), "final.norm": vec(W, 1.0)}

    def delta_tensors(p, m, by_channel):
        H, G, D, DV = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        for name, rows in (("q", G * D), ("k", G * D), ("v", H * DV)):
            w[p + name], w[p + name + ".conv"] = mat(rows, W, 1.5), vec((rows, m["conv"]), 0.2, 0.5)
        # keys that resemble the queries, so that no read-out is a sum that nearly cancels before it is normalised
        w[p + "k"], w[p + "k.conv"] = 0.4 * w[p + "k"] + w[p + "q"], w[p + "q.conv"] + 0.1 * w[p + "k.conv"]
        w[p + "b"], w[p + "A_log"], w[p + "norm"] = mat(H, W), vec(H, 0.0, 0.7), vec(DV, 1.0)
        if by_channel:
            w[p + "a1"], w[p + "a2"], w[p + "dt_bias"] = mat(ranks[0], W), mat(H * D, ranks[0]), vec(H * D, *decay)
            w[p + "g1"], w[p + "g2"] = mat(ranks[1], W), mat(H * DV, ranks[1])
        else:
            w[p + "a"], w[p + "dt_bias"], w[p + "g"] = mat(H, W), vec(H, *decay), mat(H * DV, W)
        w[p + "o"] = mat(W, H * DV, 1.5)

    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}."
        if layer["type"] == "parallel":
            a = m["left"]
            w[p + "mix.left.q"], w[p + "mix.left.k"] = mat(a["heads"] * a["dim"], W, 2.0), mat(a["kv_heads"] * a["dim"], W, 2.0)
            w[p + "mix.left.v"], w[p + "mix.left.o"] = mat(a["kv_heads"] * a["vdim"], W), mat(W, a["heads"] * a["vdim"], 3.0)
            delta_tensors(p + "mix.right.", m["right"], True)
        else:
            delta_tensors(p + "mix.", m, False)
        subs = [1]
        w[p + "norm1"] = vec(W, 1.0)
        if layer.get("mlp"):
            subs.append(2)
            w[p + "norm2"] = vec(W, 1.0)
            E, F = layer["mlp"]["router"]["experts"], layer["mlp"]["expert"]["ff"]
            w[p + "mlp.router"] = mat(E, W, 2.0)
            for e in range(E):
                w[f"{p}mlp.e{e}.gate"], w[f"{p}mlp.e{e}.up"], w[f"{p}mlp.e{e}.down"] = mat(F, W, 2.0), mat(F, W, 2.0), mat(W, F)
        for q in subs:
            w[f"{p}hc{q}.in"], w[f"{p}hc{q}.out"] = vec(n, 1.0 / n, 0.3), vec(n, 0.7, 0.4)
            w[f"{p}hc{q}.mix"] = torch.eye(n) * 0.8 + vec((n, n), 0.0, 0.15)
    return {k: v.to(torch.bfloat16) for k, v in w.items()}
