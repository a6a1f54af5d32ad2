"""A plain, slow restatement of the Nomutar decoder for tests: whole sequences, no cache, float64, one function per
mechanism.  It shares no code with the package.  Weights come as a ``{name: tensor}`` mapping and the configuration as
the dictionary config.json holds.

Notation: T tokens, W the model's width, H query heads, G key/value heads; ``h`` is a layer's normed input ``[T, W]``.
A layer is  h = N(x);  x <- x + m (mixer(h + C(h)) + ff(h))  with N an RMS norm over equal parts of the vector, C a short
causal convolution per channel and m one number for the model.  Layers ``loop.start .. loop.stop - 1`` run ``loop.times``
times over with the same weights.
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


def group_norm(x, w, groups, eps):
    """Every one of ``groups`` equal consecutive parts by its own root mean square, then the weight over the whole."""
    parts = x.reshape(*x.shape[:-1], groups, x.shape[-1] // groups)
    return rms(parts, eps).reshape(x.shape) * f64(w)


def silu(z):
    return z * torch.sigmoid(z)


def soft_cap(s, cap):
    """cap tanh(s / cap)."""
    return cap * torch.tanh(s / cap)


# ---- embedding ------------------------------------------------------------------------------------------------------------

def bigram_rows(tokens, mul_prev, mul_cur, buckets):
    """The row of the pair table every token adds: the hash of (token before it, token); the first token has a row of its
    own behind the hashed ones."""
    rows = [buckets]
    for a, b in zip(tokens[:-1], tokens[1:]):
        rows.append((int(a) * mul_prev + int(b) * mul_cur) % buckets)
    return rows


def embed(config, w, tokens):
    e = config["embedding"]
    x = f64(w["embed"])[torch.as_tensor(list(tokens), dtype=torch.long)] * e["scale"]
    if e.get("bigram") is not None:
        b = e["bigram"]
        x = x + f64(w["bigram"])[torch.as_tensor(bigram_rows(list(tokens), b["mul_prev"], b["mul_cur"], b["buckets"]))]
    return x


def causal_conv(h, taps_w):
    """c_t = sum_j w[:, j] h_(t - taps + 1 + j), zeros ahead of the first token."""
    T, taps = h.shape[0], taps_w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, h.shape[1], dtype=F), h], 0)
    return sum(f64(taps_w)[:, j] * padded[j:j + T] for j in range(taps))


# ---- rotations --------------------------------------------------------------------------------------------------------------

def base_frequencies(dims, base):
    return [float(base) ** (-2.0 * i / dims) for i in range(dims // 2)]


def llama3_frequencies(freqs, factor, low, high, original):
    """Short wavelengths stay, long ones are stretched by ``factor``, between them a blend by wavelength."""
    out = []
    for f in freqs:
        wave = 2.0 * math.pi / f
        if wave < original / high:
            out.append(f)
        elif wave > original / low:
            out.append(f / factor)
        else:
            s = (original / wave - low) / (high - low)
            out.append((1.0 - s) * f / factor + s * f)
    return out


def yarn_frequencies(freqs, dims, base, factor, original, fast, slow):
    """(frequencies, what cos and sin are multiplied by): a ramp over the dimensions from f to f / factor."""
    dim_of = lambda turns: dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(dim_of(fast)), 0), min(math.ceil(dim_of(slow)), dims - 1)
    out = []
    for i, f in enumerate(freqs):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / factor * ramp + f * (1.0 - ramp))
    return out, 0.1 * math.log(factor) + 1.0


def rotate(x, positions, freqs, layout, amplitude=1.0, sign=1.0):
    """x [T, heads, n]: the first 2 len(freqs) elements turn in pairs by sign p f_i (``halves``: i with i + dims/2;
    ``pairs``: 2i with 2i + 1), cos and sin times ``amplitude``; the rest pass."""
    half = len(freqs)
    dims = 2 * half
    ang = sign * torch.as_tensor(list(positions), dtype=F)[:, None, None] * torch.as_tensor(freqs, dtype=F)
    c, s = torch.cos(ang) * amplitude, torch.sin(ang) * amplitude
    out = x.clone()
    if layout == "halves":
        u, v = x[..., :half], x[..., half:dims]
        out[..., :half], out[..., half:dims] = u * c - v * s, v * c + u * s
    else:
        u, v = x[..., 0:dims:2], x[..., 1:dims:2]
        out[..., 0:dims:2], out[..., 1:dims:2] = u * c - v * s, v * c + u * s
    return out


# ---- attention --------------------------------------------------------------------------------------------------------------

def visible(T, window=None):
    """[T, T] bool: j <= i and (window is None or i - j < window)."""
    i = torch.arange(T)
    d = i[:, None] - i[None, :]
    return (d >= 0) if window is None else (d >= 0) & (d < window)


def weights_with_sink(s, mask, sink):
    """exp(s_j) / (exp(sink) + sum exp(s)) over the visible keys; ``sink`` None: no such term."""
    s = s.masked_fill(~mask, float("-inf"))
    if sink is None:
        return torch.softmax(s, -1)
    sink = torch.as_tensor(sink, dtype=F)
    top = torch.maximum(s.max(-1, keepdim=True).values, sink)
    e = torch.exp(s - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink - top))


def attention(h, w, p, kind, m, eps, store=None):
    """The three mixers; what differs: ``attention`` norms q and k whole, rotates halves (stretched by wavelength), rotates
    the values too, caps, and has a sink a head; ``attention_2`` has biases, rotates neighbours with the ramp, caps, and
    adds one to the denominator; ``attention_3`` norms q and k whole and rotates halves, nothing else."""
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    lin = lambda n: h @ f64(w[f"{p}.{n}"]).T + (f64(w[f"{p}.{n}.b"]) if kind == "attention_2" else 0.0)
    q, k, v = lin("q"), lin("k"), lin("v")
    if kind != "attention_2":
        q, k = rms(q, eps) * f64(w[p + ".q.norm"]), rms(k, eps) * f64(w[p + ".k.norm"])
    q, k, v = q.view(T, H, D), k.view(T, G, D), v.view(T, G, V)
    rot, pos, amplitude, layout = m["rot"], range(T), 1.0, "halves"
    freqs = base_frequencies(rot["dims"], rot["base"])
    sc = rot.get("scaling")
    if kind == "attention" and sc is not None:
        freqs = llama3_frequencies(freqs, sc["factor"], sc["low"], sc["high"], sc["original"])
    if kind == "attention_2":
        layout = "pairs"
        if sc is not None:
            freqs, amplitude = yarn_frequencies(freqs, rot["dims"], rot["base"], sc["factor"], sc["original"], sc["fast"], sc["slow"])
    q, k = rotate(q, pos, freqs, layout, amplitude), rotate(k, pos, freqs, layout, amplitude)
    vfreqs = base_frequencies(V, rot["base"])
    if kind == "attention":
        v = rotate(v, pos, vfreqs, "halves")
    if store is not None:
        k, v = store(k), store(v)
    mask = visible(T, m["mask"]["size"] if m.get("mask") is not None else None)
    o = torch.empty(T, H, V, dtype=F)
    for hd in range(H):
        g = hd // (H // G)
        s = q[:, hd] @ k[:, g].T * m["scale"]
        if m.get("softcap") is not None:
            s = soft_cap(s, m["softcap"])
        sink = {"attention": lambda: float(w[p + ".sink"][hd]), "attention_2": lambda: 0.0, "attention_3": lambda: None}[kind]()
        o[:, hd] = weights_with_sink(s, mask, sink) @ v[:, g]
    if kind == "attention":
        o = rotate(o, pos, vfreqs, "halves", sign=-1.0)
    return o.reshape(T, H * V) @ f64(w[p + ".o"]).T


# ---- feed-forwards ------------------------------------------------------------------------------------------------------

def gated(h, w, p):
    lin = lambda x, n: x @ f64(w[f"{p}.{n}"]).T
    return lin(silu(lin(h, "gate")) * lin(h, "up"), "down")


def route(h, w, p, r):
    """[T, E] weights: the ``top`` largest logits, softmax over those, zero elsewhere; also the chosen and the margin
    between the last chosen logit and the first left out."""
    z = h @ f64(w[p + ".router"]).T + f64(w[p + ".router.b"])
    E, top = r["experts"], r["top"]
    order = torch.sort(z, dim=-1, descending=True, stable=True).indices
    chosen = order[:, :top]
    out = torch.zeros_like(z)
    out.scatter_(1, chosen, torch.softmax(z.gather(1, chosen), -1))
    margin = torch.full((z.shape[0],), float("inf"), dtype=F)
    if top < E:
        margin = (z.gather(1, order[:, top - 1:top]) - z.gather(1, order[:, top:top + 1]))[:, 0]
    return out, chosen, margin


def moe(h, w, p, mlp):
    weights, chosen, _ = route(h, w, p, mlp["router"])
    y = torch.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        rows = torch.nonzero((chosen == e).any(-1))[:, 0]
        if rows.numel():
            y[rows] += weights[rows, e:e + 1] * gated(h[rows], w, f"{p}.e{e}")
    if mlp.get("shared") is not None:
        y = y + torch.sigmoid(h @ f64(w[p + ".shared.sg"]).T) * gated(h, w, p + ".shared")
    return y


def feed_forward(h, w, p, mlp):
    return gated(h, w, p) if mlp["kind"] == "dense" else moe(h, w, p, mlp)


# ---- the model ------------------------------------------------------------------------------------------------------------

def run_order(config):
    n, loop = len(config["layers"]), config.get("loop")
    if loop is None:
        return list(range(n))
    a, b = loop["start"], loop["stop"]
    return list(range(a)) + list(range(a, b)) * loop["times"] + list(range(b, n))


def layer(x, w, i, spec, config, round_inputs, store):
    p, eps = f"l{i}", config["norm"]["eps"]
    h = round_inputs(group_norm(x, w[p + ".norm1"], config["norm"]["groups"], eps))
    hm = round_inputs(h + causal_conv(h, w[p + ".canon1"])) if config.get("canon") is not None else h
    y = attention(hm, w, p + ".mix", spec["type"], spec["mixer"], eps, store)
    if spec.get("mlp") is not None:
        y = y + feed_forward(h, w, p + ".mlp", spec["mlp"])
    return x + config["residual_mult"] * y


def forward(config, w, tokens, round_inputs=None, store=None, return_layers=False):
    """Logits [T, vocab] (float64) for one sequence.  ``round_inputs``: applied to what a product reads (None: nothing);
    ``store``: how kept keys and values are rounded."""
    rin = round_inputs or (lambda t: t)
    x = embed(config, w, tokens)
    per_layer = []
    for i in run_order(config):
        x = layer(x, w, i, config["layers"][i], config, rin, store)
        per_layer.append(x.clone())
    logits = rin(group_norm(x, w["final.norm"], config["norm"]["groups"], config["norm"]["eps"])) @ f64(w["head"]).T
    if config.get("logit_softcap") is not None:
        logits = soft_cap(logits, config["logit_softcap"])
    return (logits, torch.stack(per_layer)) if return_layers else logits
