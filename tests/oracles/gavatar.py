"""Plain, slow implementation of the Gavatar design, one function per mechanism.

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


def norm(x, w, eps):
    """The weight is stored around zero."""
    return rms(x, eps) * (1 + w)


def silu(z):
    return z * torch.sigmoid(z)


# ---- embedding, order of layers, residual ---------------------------------------------------------------------------
def position_vectors(T, width, dtype):
    """sin and cos of the position at geometrically spaced frequencies, alternating."""
    out = torch.zeros(T, width, dtype=torch.float64)
    p = torch.arange(T, dtype=torch.float64)
    for c in range(width):
        angle = p * 10000.0 ** (-2.0 * (c // 2) / width)
        out[:, c] = torch.cos(angle) if c % 2 else torch.sin(angle)
    return out.to(dtype)


def embed(tokens, table, scale):
    x = table[torch.as_tensor(tokens)] * scale
    return x + position_vectors(x.shape[0], x.shape[1], x.dtype)


def layer_runs(cfg):
    """``(layer, pass)`` of every layer run; pass is None except for the first layer of a pass of the loop."""
    loop, n = cfg.get("loop"), len(cfg["layers"])
    if not loop:
        return [(i, None) for i in range(n)]
    runs = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        runs += [(i, t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return runs + [(i, None) for i in range(loop["stop"], n)]


def token_shift(h, mu):
    before = torch.cat((torch.zeros_like(h[:1]), h[:-1]))
    return h + (before - h) * mu


# ---- attention ----------------------------------------------------------------------------------------------------------
def window_mask(T, size):
    """True where the row's token sees the column's."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (i - j >= 0) & (i - j < size)


def softmax(s, mask, sink=None):
    """Over the visible keys; ``sink``: one more term of the denominator."""
    s = s.masked_fill(~mask, float("-inf"))
    top = s.max(-1, keepdim=True).values
    if sink is not None:
        top = torch.clamp(top, min=sink)
    e = torch.exp(s - top)
    total = e.sum(-1, keepdim=True)
    if sink is not None:
        total = total + torch.exp(sink - top)
    return e / total


def talk_over_heads(weights, talk):
    """weights [H, T, T]; head h becomes the combination talk[h, :] of all heads."""
    out = torch.zeros_like(weights)
    for h in range(weights.shape[0]):
        for g in range(weights.shape[0]):
            out[h] = out[h] + talk[h, g] * weights[g]
    return out


def attention(h, get, m, eps):
    T, H, G, D, DV = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms((linear(h, get("q")) + get("q.b")).view(T, H, D), eps)
    k = rms((linear(h, get("k")) + get("k.b")).view(T, G, D), eps)
    v = rms((linear(h, get("v")) + get("v.b")).view(T, G, DV), eps)
    mask = window_mask(T, m["mask"]["size"])
    own = [i // (H // G) for i in range(H)]
    weights = torch.stack([softmax(q[:, i] @ k[:, own[i]].t() * m["scale"], mask) for i in range(H)])
    weights = talk_over_heads(weights, get("talk"))
    o = torch.cat([weights[i] @ v[:, own[i]] for i in range(H)], dim=-1)
    return linear(o * torch.sigmoid(linear(h, get("g"))), get("o"))


def latent_attention(h, get, m, eps):
    T, H, D, DV = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = linear(rms(linear(h, get("dq")), eps) * get("dq.norm"), get("uq")).view(T, H, D)
    c = rms(linear(h, get("dkv")), eps) * get("dkv.norm")
    k, v = linear(c, get("uk")).view(T, H, D), linear(c, get("uv")).view(T, H, DV)
    mask, gate = window_mask(T, m["mask"]["size"]), torch.sigmoid(linear(h, get("g")))
    o = [softmax(q[:, i] @ k[:, i].t() * m["scale"], mask, get("sink")[i]) @ v[:, i] * gate[:, i:i + 1] for i in range(H)]
    return linear(torch.cat(o, dim=-1), get("o"))


# ---- matrix memory --------------------------------------------------------------------------------------------------------
def soft_cap(z, cap):
    return cap * torch.tanh(z / cap)


def log_sigmoid(z):
    return torch.clamp(z, max=0) - torch.log1p(torch.exp(-z.abs()))


def matrix_memory(q, k, v, i, f):
    """q, k [T, H, D], v [T, H, DV], log gates [T, H] -> [T, H, DV]. Memory, normaliser and running maximum from zero."""
    T, H, D = q.shape
    S, n, m = q.new_zeros(H, D, v.shape[-1]), q.new_zeros(H, D), q.new_zeros(H)
    out = []
    for t in range(T):
        new = torch.maximum(f[t] + m, i[t])
        keep, put = torch.exp(f[t] + m - new), torch.exp(i[t] - new)
        S = keep[:, None, None] * S + put[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + put[:, None] * k[t]
        m = new
        size = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out.append((S * q[t][:, :, None]).sum(1) / size[:, None])
    return torch.stack(out)


def mlstm(h, get, m, eps):
    T, H, D, DV, cap = h.shape[0], m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    q = linear(h, get("q")).view(T, H, D) * D ** -0.5
    k, v = linear(h, get("k")).view(T, H, D), linear(h, get("v")).view(T, H, DV)
    i = soft_cap(linear(h, get("i")) + get("i.b"), cap)
    f = log_sigmoid(soft_cap(linear(h, get("f")) + get("f.b"), cap))
    o = rms(matrix_memory(q, k, v, i, f), eps).reshape(T, H * DV)
    return linear(o * get("norm") * torch.sigmoid(linear(h, get("g"))), get("o"))


MIXERS = {"attention": attention, "latent_attention": latent_attention, "mlstm": mlstm}


# ---- mixture of experts ------------------------------------------------------------------------------------------------------
def expert(h, gate, up, down):
    return linear(silu(linear(h, gate)) * linear(h, up), down)


def router(h, get, top):
    z = linear(h, get("router")) + get("router.b")
    best, ids = torch.topk(z, top, dim=-1)
    return torch.softmax(best, dim=-1), ids


def feed_forward(h, get, m):
    n, top = m["router"]["experts"], m["router"]["top"]
    share, ids = router(h, get, top)
    y = torch.zeros_like(h)
    for e in range(n):
        for j in range(top):
            rows = (ids[:, j] == e).nonzero()[:, 0]
            if len(rows):
                y[rows] += share[rows, j][:, None] * expert(h[rows], get(f"e{e}.gate"), get(f"e{e}.up"), get(f"e{e}.down"))
    return y


def forward(cfg, w, tokens, dtype=torch.float64, trace=None):
    """Logits ``[T, vocab]`` of every position of one sequence; ``trace`` (a list) collects the residual after each layer
    run."""
    t = {n: x.to(dtype) for n, x in w.items()}
    eps = cfg["norm"]["eps"]
    x = embed(tokens, t["embed"], cfg["embedding"]["scale"])
    for i, step in layer_runs(cfg):
        layer, p = cfg["layers"][i], f"l{i}."
        if step is not None:
            x = x + t["loop.step"][step]
        h = token_shift(norm(x, t[p + "norm1"], eps), t[p + "shift"])
        x = x + norm(MIXERS[layer["type"]](h, lambda n: t[p + "mix." + n], layer["mixer"], eps), t[p + "norm1b"], eps)
        if layer.get("mlp"):
            y = feed_forward(norm(x, t[p + "norm2"], eps), lambda n: t[p + "mlp." + n], layer["mlp"])
            x = x + norm(y, t[p + "norm2b"], eps)
        if trace is not None:
            trace.append(x)
    return linear(norm(x, t["final.norm"], eps), t["head"])


# ---- random checkpoints -------------------------------------------------------------------------------------------------------
def random_weights(cfg, seed=0, gates=((-0.5, 1.0), (3.0, 1.0))):
    """A checkpoint of bfloat16 tensors with every tensor of the design away from its neutral value. ``gates``: mean and
    spread of the biases of the input and forget gates."""
    g = torch.Generator().manual_seed(seed)
    W = cfg["width"]

    def mat(rows, cols, gain=1.0):
        return torch.randn(rows, cols, generator=g) * gain / math.sqrt(cols)

    def vec(size, mean=0.0, std=0.2):
        return mean + torch.randn(size, generator=g) * std

    w = {"embed": mat(cfg["vocab"], W, 2.0), "final.norm": vec(W), "head": mat(cfg["vocab"], W)}
    if cfg.get("loop"):
        w["loop.step"] = vec((cfg["loop"]["times"], W), 0.0, 0.5)
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}."
        x = p + "mix."
        w[p + "norm1"], w[p + "norm1b"], w[p + "shift"] = vec(W), vec(W), vec(W, 0.4, 0.3)
        H, DV = m["heads"], m["vdim"]
        if layer["type"] == "attention":
            G, D = m["kv_heads"], m["dim"]
            for n, rows in (("q", H * D), ("k", G * D), ("v", G * DV)):
                w[x + n], w[x + n + ".b"] = mat(rows, W), vec(rows, 0.0, 0.3)
            w[x + "talk"] = torch.eye(H) * 0.7 + vec((H, H), 0.0, 0.3)
            w[x + "g"] = mat(H * DV, W)
        elif layer["type"] == "latent_attention":
            R, Q, D = m["kv_rank"], m["q_rank"], m["dim"]
            w[x + "dq"], w[x + "dq.norm"], w[x + "uq"] = mat(Q, W), vec(Q, 1.0), mat(H * D, Q, 1.5)
            w[x + "dkv"], w[x + "dkv.norm"], w[x + "uk"], w[x + "uv"] = mat(R, W), vec(R, 1.0), mat(H * D, R, 1.5), mat(H * DV, R)
            w[x + "sink"], w[x + "g"] = vec(H, 1.0, 1.0), mat(H, W)
        else:
            D = m["dim"]
            w[x + "q"], w[x + "v"] = mat(H * D, W, 1.5), mat(H * DV, W)
            # keys that resemble the queries, so that no read-out is a sum that nearly cancels before it is normalised
            w[x + "k"] = 0.7 * w[x + "q"] + mat(H * D, W, 0.5)
            w[x + "i"], w[x + "f"] = mat(H, W), mat(H, W)
            w[x + "i.b"], w[x + "f.b"] = vec(H, *gates[0]), vec(H, *gates[1])
            w[x + "norm"], w[x + "g"] = vec(H * DV, 1.0), mat(H * DV, W)
        w[x + "o"] = mat(W, H * DV)
        if layer.get("mlp"):
            w[p + "norm2"], w[p + "norm2b"] = vec(W), vec(W)
            E, F = layer["mlp"]["router"]["experts"], layer["mlp"]["expert"]["ff"]
            w[p + "mlp.router"], w[p + "mlp.router.b"] = mat(E, W, 2.0), vec(E, 0.0, 0.5)
            for e in range(E):
                w[f"{p}mlp.e{e}.gate"], w[f"{p}mlp.e{e}.up"], w[f"{p}mlp.e{e}.down"] = mat(F, W, 2.0), mat(F, W, 2.0), mat(W, F)
    return {k: v.to(torch.bfloat16) for k, v in w.items()}
