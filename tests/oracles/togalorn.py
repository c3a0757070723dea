"""Plain, slow implementation of the Togalorn design, one function per mechanism.

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


def grouped_norm(x, w, groups, eps):
    """Each of ``groups`` neighbouring parts of a vector by its own root mean square."""
    width = x.shape[-1] // groups
    parts = [rms(x[..., g * width:(g + 1) * width], eps) for g in range(groups)]
    return torch.cat(parts, dim=-1) * w


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def causal_conv(x, w):
    """x [T, C], w [C, taps]; the last column meets the current row, rows before the first are zero."""
    T, taps = x.shape[0], w.shape[1]
    out = torch.zeros_like(x)
    for t in range(T):
        for j in range(taps):
            at = t - taps + 1 + j
            if at >= 0:
                out[t] = out[t] + w[:, j] * x[at]
    return out


# ---- order of layers ------------------------------------------------------------------------------------------------
def layer_runs(cfg):
    """``(layer, pass)`` of every layer run; pass is None except for the first layer of a pass of the loop."""
    loop, n = cfg.get("loop"), len(cfg["layers"])
    if not loop:
        return [(i, None) for i in range(n)]
    runs = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        runs += [(i, t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return runs + [(i, None) for i in range(loop["stop"], n)]


def enter_pass(x, x0, w_in, step):
    """The stream and the embedding through one matrix, plus the pass's vector."""
    return linear(torch.cat((x, x0), dim=-1), w_in) + step


# ---- latent attention -----------------------------------------------------------------------------------------------
def rotate(x, base, positions=None):
    """x [T, ..., R]: neighbouring dimensions are pairs."""
    T, R = x.shape[0], x.shape[-1]
    p = torch.arange(T, dtype=torch.float64) if positions is None else positions.to(torch.float64)
    out = x.clone()
    for i in range(R // 2):
        a = (p * base ** (-2.0 * i / R)).view((T,) + (1,) * (x.dim() - 2))
        c, s = torch.cos(a).to(x.dtype), torch.sin(a).to(x.dtype)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i], out[..., 2 * i + 1] = u * c - v * s, v * c + u * s
    return out


def causal_softmax(s):
    T = s.shape[-1]
    s = s.masked_fill(torch.ones(T, T, dtype=torch.bool).triu(1), float("-inf"))
    e = torch.exp(s - s.max(-1, keepdim=True).values)
    return e / e.sum(-1, keepdim=True)


def latent_attention(h, get, m, eps):
    T, H, D, P, DV, R = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = linear(rms(linear(h, get("dq")), eps) * get("dq.norm"), get("uq")).view(T, H, D + P)
    down = linear(h, get("dkv"))
    c = rms(down[:, :R], eps) * get("dkv.norm")
    k, v = linear(c, get("uk")).view(T, H, D), linear(c, get("uv")).view(T, H, DV)
    q_rot, k_rot = rotate(q[..., D:], m["rot"]["base"]), rotate(down[:, R:], m["rot"]["base"])
    heads = []
    for i in range(H):
        s = (linear(q[:, i, :D], k[:, i]) + linear(q_rot[:, i], k_rot)) * m["scale"]
        heads.append(causal_softmax(s) @ v[:, i])
    return linear(torch.cat(heads, dim=-1) * torch.sigmoid(linear(h, get("g"))), get("o"))


# ---- state-space mixer ----------------------------------------------------------------------------------------------
def state_space(x, B, C, dt, A_log, D):
    """x [T, H, P], B and C [T, G, N], dt [T, H] (positive) -> [T, H, P]; the state starts at zero."""
    T, H, P = x.shape
    G, N = B.shape[1:]
    S, out = x.new_zeros(H, N, P), torch.zeros_like(x)
    for t in range(T):
        for h in range(H):
            g = h // (H // G)
            S[h] = torch.exp(-torch.exp(A_log[h]) * dt[t, h]) * S[h] + dt[t, h] * torch.outer(B[t, g], x[t, h])
            out[t, h] = S[h].t() @ C[t, g] + D[h] * x[t, h]
    return out


def mamba2(h, get, m, eps):
    T, H, P, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    z, xbc, dt = torch.split(linear(h, get("in")), (inner, inner + 2 * G * N, H), dim=-1)
    xbc = silu(causal_conv(xbc, get("conv")) + get("conv.b"))
    x, B, C = torch.split(xbc, (inner, G * N, G * N), dim=-1)
    dt = softplus(dt + get("dt_bias"))
    y = state_space(x.reshape(T, H, P), B.reshape(T, G, N), C.reshape(T, G, N), dt, get("A_log"), get("D"))
    return linear(grouped_norm(y.reshape(T, inner) * silu(z), get("norm"), m["norm_groups"], eps), get("o"))


MIXERS = {"latent_attention": latent_attention, "mamba2": mamba2}


# ---- mixture of experts ---------------------------------------------------------------------------------------------
def expert(h, gate, up, down, limit):
    g = torch.clamp(linear(h, gate), max=limit)
    u = torch.clamp(linear(h, up), -limit, limit)
    return linear(g * torch.sigmoid(1.702 * g) * (u + 1), down)


def router(h, get, top):
    z = linear(h, get("router"))
    e = torch.exp(z - z.max(-1, keepdim=True).values)
    s = e / e.sum(-1, keepdim=True)
    ids = torch.topk(s + get("correction"), top, dim=-1).indices
    share = torch.gather(s, -1, ids)
    return share / (share.sum(-1, keepdim=True) + 1e-20), ids


def feed_forward(h, get, m):
    real = m["router"]["experts"]
    share, ids = router(h, get, m["router"]["top"])
    y = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for j in range(ids.shape[1]):
            e = int(ids[t, j])
            if e >= real:
                y[t] = y[t] + share[t, j] * h[t]
            else:
                y[t] = y[t] + share[t, j] * expert(h[t], get(f"e{e}.gate"), get(f"e{e}.up"), get(f"e{e}.down"), m["expert"]["limit"])
    return y + expert(h, get("shared.gate"), get("shared.up"), get("shared.down"), m["shared"]["limit"])


def layer(x, cfg, i, get):
    """``x + (mixer(h + conv(h)) + ff(h))`` with ``h`` the normed stream."""
    eps, own = cfg["norm"]["eps"], cfg["layers"][i]
    h = grouped_norm(x, get("norm1"), cfg["norm"]["groups"], eps)
    y = MIXERS[own["type"]](h + causal_conv(h, get("canon1")), lambda n: get("mix." + n), own["mixer"], eps)
    if own.get("mlp"):
        y = y + feed_forward(h, lambda n: get("mlp." + n), own["mlp"])
    return x + y


def forward(cfg, w, tokens, dtype=torch.float64, trace=None):
    """Logits ``[T, vocab]`` of every position of one sequence; ``trace`` (a list) collects the residual after each layer
    run."""
    t = {n: x.to(dtype) for n, x in w.items()}
    x0 = t["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"]
    x = x0
    for i, step in layer_runs(cfg):
        if step is not None:
            x = enter_pass(x, x0, t["loop.in"], t["loop.step"][step])
        x = layer(x, cfg, i, lambda n: t[f"l{i}.{n}"])
        if trace is not None:
            trace.append(x)
    return linear(grouped_norm(x, t["final.norm"], cfg["norm"]["groups"], cfg["norm"]["eps"]), t["head"])


# ---- random checkpoints ---------------------------------------------------------------------------------------------
def random_weights(cfg, seed=0, decay=(-1.0, 1.0), step=(-2.0, 1.0)):
    """A checkpoint of bfloat16 tensors with every tensor of the design away from its neutral value. ``decay`` and ``step``:
    mean and spread of ``A_log`` and ``dt_bias``."""
    g = torch.Generator().manual_seed(seed)
    W, taps = cfg["width"], cfg["canon"]["taps"]

    def mat(rows, cols, gain=1.0):
        return torch.randn(rows, cols, generator=g) * gain / math.sqrt(cols)

    def vec(size, mean=0.0, std=0.2):
        return mean + torch.randn(size, generator=g) * std

    w = {"embed": mat(cfg["vocab"], W, 2.0), "final.norm": vec(W, 1.0), "head": mat(cfg["vocab"], W)}
    if cfg.get("loop"):
        w["loop.step"], w["loop.in"] = vec((cfg["loop"]["times"], W), 0.0, 0.5), mat(W, 2 * W)
    for i, own in enumerate(cfg["layers"]):
        m, p = own["mixer"], f"l{i}."
        x = p + "mix."
        w[p + "norm1"], w[p + "canon1"] = vec(W, 1.0), vec((W, taps), 0.0, 0.6)
        H, P = m["heads"], m["vdim"]
        if own["type"] == "latent_attention":
            R, Q, D, rot = m["kv_rank"], m["q_rank"], m["dim"], m["rot_dim"]
            w[x + "dq"], w[x + "dq.norm"], w[x + "uq"] = mat(Q, W), vec(Q, 1.0), mat(H * (D + rot), Q, 1.5)
            w[x + "dkv"], w[x + "dkv.norm"] = mat(R + rot, W), vec(R, 1.0)
            w[x + "uk"], w[x + "uv"], w[x + "g"] = mat(H * D, R, 1.5), mat(H * P, R), mat(H * P, W)
        else:
            inner, bc = H * P, 2 * m["groups"] * m["state"]
            w[x + "in"] = mat(2 * inner + bc + H, W)
            w[x + "conv"], w[x + "conv.b"] = vec((inner + bc, m["conv"]), 0.0, 0.6), vec(inner + bc)
            w[x + "dt_bias"], w[x + "A_log"], w[x + "D"] = vec(H, *step), vec(H, *decay), vec(H, 1.0, 0.5)
            w[x + "norm"] = vec(inner, 1.0)
        w[x + "o"] = mat(W, H * P)
        if own.get("mlp"):
            mlp = own["mlp"]
            n = mlp["router"]["experts"] + mlp["router"].get("identity", 0)
            w[p + "mlp.router"], w[p + "mlp.correction"] = mat(n, W, 2.0), vec(n, 0.0, 0.1)
            for name, F in [(f"e{e}", mlp["expert"]["ff"]) for e in range(mlp["router"]["experts"])] + [("shared", mlp["shared"]["ff"])]:
                w[f"{p}mlp.{name}.gate"], w[f"{p}mlp.{name}.up"], w[f"{p}mlp.{name}.down"] = mat(F, W, 2.0), mat(F, W, 2.0), mat(W, F)
    return {k: v.to(torch.bfloat16) for k, v in w.items()}
