"""A plain, slow restatement of the Kopalorn decoder for tests: whole sequences, no cache, float64, one function per
mechanism.  It shares no code with the package.  Weights come as a ``{name: tensor}`` mapping and the configuration as
the dictionary config.json holds.

Notation: T tokens, W the model's width, H (query) heads, G key/value heads; ``h`` is a sub-layer's normed input ``[T, W]``.
A layer is  x <- x + m N1b(mixer(N1(x)));  x <- x + m N2b(ff(N2(x)))  with layer norms N and one number m for the model.
Layers ``loop.start .. loop.stop - 1`` run ``loop.times`` times over with the same weights; ahead of every pass a vector of
its own is added to x, and ahead of every pass but the first the embedding's rows as well.
"""
from __future__ import annotations

import math

import torch

F = torch.float64


def f64(t):
    return t.to(F)


def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def layer_norm(x, w, b, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * f64(w) + f64(b)


def silu(z):
    return z * torch.sigmoid(z)


def linear(w, name, h):
    """W h, plus the bias of the same name with ``.b`` where there is one."""
    y = h @ f64(w[name]).T
    return y + f64(w[name + ".b"]) if name + ".b" in w else y


# ---- softmax attention ------------------------------------------------------------------------------------------------------

def rotate_pairs(x, positions, dims, base):
    """x [T, ..., n]: elements 2i and 2i + 1 of the first ``dims`` turn by p base^(-2i/dims); the rest pass."""
    out = x.clone()
    for i in range(dims // 2):
        a = torch.as_tensor(list(positions), dtype=F) * float(base) ** (-2.0 * i / dims)
        a = a.reshape(-1, *([1] * (x.dim() - 2)))
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i], out[..., 2 * i + 1] = u * torch.cos(a) - v * torch.sin(a), v * torch.cos(a) + u * torch.sin(a)
    return out


def visible(T, window=None):
    """[T, T] bool: j <= i and (window is None or i - j < window)."""
    i = torch.arange(T)
    d = i[:, None] - i[None, :]
    return (d >= 0) if window is None else (d >= 0) & (d < window)


def softmax_attention(q, k, v, scale, mask):
    """One head: q, k [T, d], v [T, vd]."""
    return torch.softmax((q @ k.T * scale).masked_fill(~mask, float("-inf")), -1) @ v


def diff_lambda(w, p, diff):
    dot = lambda a, b: float((f64(w[f"{p}.{a}"]) * f64(w[f"{p}.{b}"])).sum())
    return math.exp(dot("lq1", "lk1")) - math.exp(dot("lq2", "lk2")) + diff


def differential_attention(h, w, p, m, eps):
    """Two softmax maps a head over the same values; the second one's output, times lambda, is taken from the first's."""
    T, H, G, D, V = h.shape[0], m["heads"], m.get("kv_heads") or m["heads"], m["dim"], m.get("vdim") or m["dim"]
    q, k = linear(w, p + ".q", h).view(T, H, 2, D), linear(w, p + ".k", h).view(T, G, 2, D)
    v = linear(w, p + ".v", h).view(T, G, V)
    if m.get("rot"):
        q, k = (rotate_pairs(t, range(T), m["rot"]["dims"], m["rot"]["base"]) for t in (q, k))
    mask = visible(T, m["mask"]["size"] if m.get("mask") else None)
    lam = diff_lambda(w, p, m["diff"])
    gate = torch.sigmoid(linear(w, p + ".g", h))                       # [T, H]
    heads = []
    for i in range(H):
        g = i // (H // G)
        a1, a2 = (softmax_attention(q[:, i, s], k[:, g, s], v[:, g], m["scale"], mask) for s in (0, 1))
        heads.append(rms(a1 - lam * a2, eps) * (1.0 - m["diff"]) * gate[:, i:i + 1])
    return linear(w, p + ".o", torch.cat(heads, -1))


def gated_attention(h, w, p, m):
    """Every earlier key, biases on q, k and v, no positions, a gate an element."""
    T, H, G, D, V = h.shape[0], m["heads"], m.get("kv_heads") or m["heads"], m["dim"], m.get("vdim") or m["dim"]
    q, k, v = linear(w, p + ".q", h).view(T, H, D), linear(w, p + ".k", h).view(T, G, D), linear(w, p + ".v", h).view(T, G, V)
    o = [softmax_attention(q[:, i], k[:, i // (H // G)], v[:, i // (H // G)], m["scale"], visible(T)) for i in range(H)]
    return linear(w, p + ".o", torch.cat(o, -1) * torch.sigmoid(linear(w, p + ".g", h)))


# ---- recurrent mixers -------------------------------------------------------------------------------------------------------

def stabilised_memory(q, k, v, i, f):
    """One head of the matrix memory, token by token: q, k [T, D], v [T, V], log gates i, f [T]."""
    S, n, m, out = torch.zeros(k.shape[1], v.shape[1], dtype=F), torch.zeros(k.shape[1], dtype=F), 0.0, []
    for t in range(q.shape[0]):
        new = max(float(f[t]) + m, float(i[t]))
        keep, write = math.exp(float(f[t]) + m - new), math.exp(float(i[t]) - new)
        m = new
        S = keep * S + write * torch.outer(k[t], v[t])
        n = keep * n + write * k[t]
        out.append(S.T @ q[t] / (max(abs(float(n @ q[t])), math.exp(-m)) + 1e-6))
    return torch.stack(out)


def mlstm(h, w, p, m, eps):
    T, H, D, V, cap = h.shape[0], m["heads"], m["dim"], m.get("vdim") or m["dim"], m["gate_cap"]
    q, k = linear(w, p + ".q", h).view(T, H, D) / math.sqrt(D), linear(w, p + ".k", h).view(T, H, D)
    v = linear(w, p + ".v", h).view(T, H, V)
    i = cap * torch.tanh(linear(w, p + ".i", h) / cap)
    f = torch.nn.functional.logsigmoid(cap * torch.tanh(linear(w, p + ".f", h) / cap))
    o = torch.cat([rms(stabilised_memory(q[:, j], k[:, j], v[:, j], i[:, j], f[:, j]), eps) for j in range(H)], -1)
    return linear(w, p + ".o", o * f64(w[p + ".norm"]) * torch.sigmoid(linear(w, p + ".g", h)))


def decayed_sums(q, k, v, decay):
    """One head: S <- decay S + k v^T; o = S^T q."""
    S, out = torch.zeros(k.shape[1], v.shape[1], dtype=F), []
    for t in range(q.shape[0]):
        S = decay * S + torch.outer(k[t], v[t])
        out.append(S.T @ q[t])
    return torch.stack(out)


def lightning(h, w, p, m, eps):
    T, H, D, V = h.shape[0], m["heads"], m["dim"], m.get("vdim") or m["dim"]
    q, k, v = (silu(linear(w, f"{p}.{n}", h)).view(T, H, s) for n, s in (("q", D), ("k", D), ("v", V)))
    o = torch.cat([decayed_sums(q[:, j], k[:, j], v[:, j], m["decay"][j]) for j in range(H)], -1)
    return linear(w, p + ".o", rms(o, eps) * f64(w[p + ".norm"]) * torch.sigmoid(linear(w, p + ".g", h)))


def parallel(h, w, p, m, eps):
    l, r = gated_attention(h, w, p + ".left", m["left"]), lightning(h, w, p + ".right", m["right"], eps)
    return 0.5 * (rms(l, eps) * f64(w[p + ".left.out"]) + rms(r, eps) * f64(w[p + ".right.out"]))


def mix(h, w, p, layer, eps):
    m = layer["mixer"]
    if layer["type"] == "attention":
        return differential_attention(h, w, p, m, eps)
    return mlstm(h, w, p, m, eps) if layer["type"] == "mlstm" else parallel(h, w, p, m, eps)


# ---- feed-forward -----------------------------------------------------------------------------------------------------------

def route_row(z, correction, r):
    """{expert: weight} of one row of router logits."""
    s = torch.sigmoid(z)
    choice = [float(s[e] + correction[e]) for e in range(len(z))]
    open_ = set(range(len(choice)))
    g = r.get("groups")
    if g is not None:
        per = len(choice) // g["count"]
        score = [sum(sorted(choice[j * per:(j + 1) * per])[-2:]) for j in range(g["count"])]
        best = sorted(range(g["count"]), key=lambda j: -score[j])[:g["keep"]]
        open_ = {e for e in open_ if e // per in best}
    chosen = sorted(open_, key=lambda e: -choice[e])[:r["top"]]
    total = sum(float(s[e]) for e in chosen) + 1e-20
    return {e: float(s[e]) / total * r.get("scale", 1.0) for e in chosen}


def expert(h, w, p):
    return linear(w, p + ".down", torch.relu(linear(w, p + ".up", h)) ** 2)


def moe(h, w, p, mlp):
    r = mlp["router"]
    z = linear(w, p + ".router", h)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, weight in route_row(z[t], f64(w[p + ".correction"]), r).items():
            out[t] += weight * expert(h[t], w, f"{p}.e{e}")
    if mlp.get("shared") is not None:
        out = out + torch.sigmoid(linear(w, p + ".shared.sg", h)) * expert(h, w, p + ".shared")
    return out


# ---- the model --------------------------------------------------------------------------------------------------------------

def schedule(config):
    """[(layer, pass or None)]: the order layers run in; ``pass`` on the first layer of every pass of the repeated run."""
    n, lp = len(config["layers"]), config.get("loop")
    if lp is None:
        return [(i, None) for i in range(n)]
    run = range(lp["start"], lp["stop"])
    return ([(i, None) for i in range(lp["start"])]
            + [(i, t if i == lp["start"] else None) for t in range(lp["times"]) for i in run]
            + [(i, None) for i in range(lp["stop"], n)])


def forward(config, w, tokens, after=None):
    """Logits [T, vocab].  ``after``: a list that receives the rows after every layer run."""
    eps, mult = config["norm"]["eps"], config.get("residual_mult", 1.0)
    x0 = f64(w["embed"])[torch.as_tensor(list(tokens), dtype=torch.long)]
    x = x0
    for i, t in schedule(config):
        layer, p = config["layers"][i], f"l{i}"
        if t is not None:
            if t > 0:
                x = x + x0
            x = x + f64(w["loop.step"])[t]
        norm = lambda name, y: layer_norm(y, w[f"{p}.{name}"], w[f"{p}.{name}.b"], eps)
        x = x + mult * norm("norm1b", mix(norm("norm1", x), w, p + ".mix", layer, eps))
        if layer.get("mlp") is not None:
            x = x + mult * norm("norm2b", moe(norm("norm2", x), w, p + ".mlp", layer["mlp"]))
        if after is not None:
            after.append(x)
    return layer_norm(x, w["final.norm"], w["final.norm.b"], eps) @ f64(w["head"]).T
