"""Small Kopalorn configurations and weights for tests.

The configurations differ from one another in every size and option: layer orders (each kind of mixer first, last, alone), repeated
runs of layers that start at the first layer, in the middle, reach the last layer, cover the whole model, run once, or are absent;
head counts and groupings (one key/value head for all, one a query head, groups of two and four); key and value sizes that differ,
that no vector width divides, and that the tensor-core kernels take; rotations of a whole map, of part of it, of two elements, and
none; windows of one token, shorter than a page, a page and one, several pages, none; decays from zero to one; caps that bite and
that hardly matter; routers with and without groups, one group kept and all of them, top = 1 and top = everything that can be chosen,
scales of one and others, with and without an expert for every token; layers without a feed-forward; widths and vocabularies that
are no multiples of 8; residual multipliers of one, below and above it.  Weights are drawn so that every mechanism matters to the
logits and stored in bfloat16 so that both compute paths and the plain implementation read the same numbers.
"""
import json
import os

import torch

import citlali_b200 as cb


def moe(experts, top, ff, shared=None, groups=None, scale=None):
    """``groups``: (count, keep)."""
    d = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if groups is not None:
        d["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
    if scale is not None:
        d["router"]["scale"] = scale
    if shared is not None:
        d["shared"] = {"ff": shared}
    return d


def attention(heads, kv_heads, dim, vdim, scale, diff, rot, window, mlp):
    """``rot``: (dims, base) or None; ``window`` None: every earlier key."""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff}
    if rot is not None:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
    if window is not None:
        m["mask"] = {"size": window}
    return {"type": "attention", "mixer": m, "mlp": mlp}


def mlstm(heads, dim, vdim, cap, mlp):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}, "mlp": mlp}


def parallel(left, right, mlp):
    """``left``: (heads, kv_heads, dim, vdim, scale); ``right``: (dim, vdim, decays)."""
    l = dict(zip(("heads", "kv_heads", "dim", "vdim", "scale"), left))
    r = {"heads": len(right[2]), "dim": right[0], "vdim": right[1], "decay": list(right[2])}
    return {"type": "parallel", "mixer": {"left": l, "right": r}, "mlp": mlp}


def model(vocab, width, eps, mult, loop, layers):
    d = {"architecture": "Kopalorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult, "layers": layers}
    if loop is not None:
        d["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return d


CONFIGS = {
    # the repeated run sits in the middle; a window shorter than a page; two groups of three of which one is kept
    "A": model(200, 64, 1e-5, 0.7, (1, 3, 2), [
        attention(4, 2, 16, 24, 0.3, 0.4, (8, 100.0), 9, moe(6, 2, 32, 24, (2, 1), 1.7)),
        mlstm(3, 24, 16, 6.0, moe(4, 1, 16)),
        parallel((6, 3, 16, 8, 0.25), (16, 24, (0.5, 0.9, 0.99)), None),
        attention(3, 3, 8, 32, 0.35, 0.8, (2, 50.0), 1, moe(8, 4, 24, 16, (4, 2), 0.6))]),
    # odd width and vocabulary, no repeated run, sizes no vector width divides, a window wider than any short request, everything
    # that can be chosen is, a head count that leaves rows unaligned
    "B": model(333, 60, 1e-6, 1.0, None, [
        mlstm(5, 12, 20, 15.0, moe(3, 3, 24, 40)),
        parallel((5, 5, 12, 20, 0.3), (20, 12, (0.0, 0.3, 0.7, 0.95, 1.0)), moe(9, 3, 20, 12, (3, 1), 2.0)),
        attention(4, 1, 10, 14, 0.3, 0.2, (6, 2000.0), 300, None)]),
    # the repeated run is the whole model and runs twice; maps of 64 with values of 128, where the widest prompt kernel serves; sixteen
    # experts; windows of several pages; a multiplier above one
    "C": model(512, 96, 1e-6, 1.25, (0, 3, 2), [
        parallel((8, 2, 64, 64, 0.125), (64, 64, (0.8, 0.97)), moe(16, 4, 16, 32, (4, 2), 2.5)),
        attention(4, 1, 64, 128, 0.15, 0.6, (32, 10000.0), 130, moe(8, 8, 24, 16)),
        mlstm(2, 128, 128, 12.0, moe(12, 3, 16, 8, (2, 2), 1.0))]),
    # the repeated run reaches the last layer and runs three times; no rotation; no window
    "D": model(130, 40, 1e-5, 0.3, (1, 3, 3), [
        attention(2, 2, 20, 16, 0.4, 0.5, None, None, moe(5, 5, 8)),
        mlstm(4, 8, 8, 3.0, None),
        parallel((2, 1, 16, 16, 0.3), (8, 16, (0.99, 0.999, 0.6, 0.2)), moe(10, 3, 16, 24, (5, 3), 1.3))]),
    # one layer that is run once by a loop; a window of a page
    "E": model(96, 72, 1e-4, 0.5, (0, 1, 1), [
        attention(6, 2, 24, 48, 0.25, 0.0, (24, 10.0), 64, moe(10, 3, 8, 64, (2, 1), 3.0))]),
    # the widest heads, a map of 128 among them
    "F": model(150, 56, 1e-5, 0.9, (0, 1, 2), [
        mlstm(1, 200, 72, 8.0, moe(4, 2, 16, 16, (2, 1))),
        attention(2, 1, 128, 136, 0.1, 0.7, (64, 500.0), 40, None),
        parallel((2, 2, 80, 80, 0.15), (256, 40, (0.97,)), moe(4, 2, 64, None, None, 0.8))]),
    # no router has a choice: bfloat16 can be held at every position
    "G": model(180, 48, 1e-5, 0.6, (1, 2, 2), [
        parallel((4, 2, 24, 16, 0.25), (16, 32, (0.9, 0.5, 0.98)), moe(4, 4, 16, 24, (2, 2), 1.5)),
        mlstm(2, 32, 40, 10.0, moe(3, 3, 16)),
        attention(4, 2, 24, 24, 0.25, 0.5, (12, 300.0), 65, moe(2, 2, 32, 16, None, 0.7))]),
}


def config(name):
    return cb.config_from_dict(json.loads(json.dumps(CONFIGS[name])))


def draw_tensor(n, shape, r):
    """A weight of the design from normal numbers ``r``, sized so that its mechanism matters."""
    last = n.split(".")[-1]
    if n.endswith("embed"):
        return 0.7 * r
    if n == "loop.step":
        return 0.5 * r
    if n.endswith(".i.b"):
        return 1.0 * r
    if n.endswith(".f.b"):
        return 2.0 + 1.5 * r
    if last == "b":
        return 0.4 * r
    if last in ("norm1", "norm2", "norm1b", "norm2b", "norm", "out"):
        return 1.0 + 0.3 * r                           # plain weights
    if last in ("lq1", "lk1", "lq2", "lk2"):
        return 0.8 * r / shape[0] ** 0.25
    if last == "correction":
        return 1.2 * r - 0.3                           # choice scores of either sign; most choices are no close calls
    if last == "router":
        return 1.5 * r / shape[1] ** 0.5
    if last in ("sg", "i", "f"):
        return 2.0 * r / shape[1] ** 0.5
    if last in ("q", "k"):
        return 1.5 * r / shape[1] ** 0.5               # scores of several units: the softmax is no average
    return r / shape[-1] ** 0.5                        # matrices [out, in]


def make_weights(cfg, seed):
    """{name: bfloat16 tensor} for every tensor the model reads."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for spec in cb.expected_tensors(cfg.to_model_spec()):
        if spec.optional:
            continue
        shape = tuple(spec.shape)
        out[spec.name] = draw_tensor(spec.name, shape, torch.randn(shape, generator=g)).to(torch.bfloat16)
    return out


def write_model(path, name, seed):
    cfg = config(name)
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg.to_dict(), f)
    w = make_weights(cfg, seed)
    cb.write_safetensors(os.path.join(path, "model.safetensors"), lambda: iter(w.items()), metadata={"format": "pt"})
    return cfg, w
