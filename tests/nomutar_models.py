"""Small Nomutar configurations and weights for tests.

The configurations differ from one another in every size and option: layer orders (each kind of mixer first, last, alone),
repeated runs of layers that start at the first layer, in the middle, reach the last layer, cover the whole model, run once,
or are absent; head counts and groupings (one key/value head for all, one a query head, groups of two and four); key and value
sizes that differ, that no vector width divides, and that the tensor-core kernels take; rotations of a whole head, of part of
it and of two elements, with and without scaled frequencies (scalings that leave all frequencies, stretch all of them, and blend
between); windows of one token, shorter than a page, a page and one, several pages, none; soft caps that bite and that hardly
matter; norms over one part, several parts, and parts of odd size; convolutions of one to six taps; dense and routed
feed-forwards, top = 1, top > 1 and top = experts, with and without an expert for every token, layers without a feed-forward;
widths and vocabularies that are no multiples of 8; residual multipliers of one, below and above it; bigram tables smaller and
larger than the vocabulary, and none.  Weights are drawn so that every mechanism matters to the logits and stored in bfloat16
so that both compute paths and the plain implementation read the same numbers.
"""
import json
import os

import torch

import citlali_b200 as cb


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, shared=None):
    d = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared is not None:
        d["shared"] = {"ff": shared}
    return d


def wavelength(factor, low, high, original):
    return {"factor": factor, "low": low, "high": high, "original": original}


def ramp(factor, original, fast, slow):
    return {"factor": factor, "original": original, "fast": fast, "slow": slow}


def mixer(kind, heads, kv_heads, dim, vdim, scale, rot, mlp, softcap=None, window=None, scaling=None):
    """``rot``: (dims, base)."""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": {"dims": rot[0], "base": rot[1]}}
    if scaling is not None:
        m["rot"]["scaling"] = scaling
    if softcap is not None:
        m["softcap"] = softcap
    if window is not None:
        m["mask"] = {"size": window}
    return {"type": kind, "mixer": m, "mlp": mlp}


def model(vocab, width, eps, groups, mult, scale, bigram, taps, cap, loop, layers):
    d = {"architecture": "Nomutar", "vocab": vocab, "width": width, "norm": {"eps": eps, "groups": groups}, "residual_mult": mult,
         "embedding": {"scale": scale}, "layers": layers}
    if bigram is not None:
        d["embedding"]["bigram"] = {"buckets": bigram[0], "mul_prev": bigram[1], "mul_cur": bigram[2]}
    if taps is not None:
        d["canon"] = {"taps": taps}
    if cap is not None:
        d["logit_softcap"] = cap
    if loop is not None:
        d["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return d


A, B, C = "attention", "attention_2", "attention_3"
CONFIGS = {
    # the repeated run sits in the middle; a window shorter than a page; values wider than keys, of sizes the tensor-core
    # kernels take; a rotation of part of a head; top = 2 of 6 with an expert for every token; a cap that bites
    "P": model(200, 64, 1e-5, 2, 0.7, 3.0, (61, 13, 7), 4, 12.0, (1, 3, 2), [
        mixer(A, 4, 2, 16, 24, 0.25, (8, 100.0), moe(6, 2, 32, 24), softcap=3.0, window=9, scaling=wavelength(8.0, 1.0, 4.0, 64)),
        mixer(B, 2, 1, 40, 8, 0.15, (40, 1000.0), dense(96), softcap=50.0, window=65, scaling=ramp(4.0, 128, 8.0, 1.0)),
        mixer(C, 6, 3, 24, 40, 0.2, (24, 10000.0), None),
        mixer(A, 3, 3, 32, 32, 0.18, (2, 50.0), moe(4, 1, 16), softcap=20.0, window=1)]),
    # odd width and vocabulary, no repeated run, every earlier key first, parts of odd size in the norm, sizes no vector width
    # divides, a window wider than any short request, top = experts, a convolution of two taps, no scaled frequencies
    "Q": model(333, 60, 1e-6, 4, 1.0, 1.5, (1000, 2, 3), 2, 40.0, None, [
        mixer(C, 5, 5, 12, 20, 0.3, (12, 100.0), moe(3, 3, 24, 40)),
        mixer(B, 4, 4, 20, 12, 0.25, (6, 500.0), None, softcap=4.0, window=300),
        mixer(A, 2, 1, 14, 18, 0.3, (10, 2000.0), dense(100), softcap=8.0, window=70)]),
    # the repeated run is the whole model and runs twice; heads of 64 and 128 with equal key and value sizes; windows of several
    # pages; sixteen experts; one part in the norm; a multiplier above one
    "R": model(512, 96, 1e-6, 1, 1.25, 4.0, (256, 1023, 31), 3, 25.0, (0, 3, 2), [
        mixer(B, 8, 2, 64, 64, 0.125, (64, 10000.0), moe(16, 4, 16, 32), softcap=10.0, window=130, scaling=ramp(16.0, 64, 32.0, 1.0)),
        mixer(C, 4, 1, 128, 128, 0.08, (128, 200000.0), dense(200)),
        mixer(A, 4, 4, 64, 64, 0.15, (32, 20.0), moe(8, 8, 24, 16), softcap=6.0, window=100, scaling=wavelength(2.0, 0.5, 16.0, 4096))]),
    # the repeated run reaches the last layer and runs three times; parts of five elements; no pair table; taps = 1; no window on
    # one capped layer; no experts for every token
    "S": model(130, 40, 1e-5, 8, 0.3, 2.0, None, 1, 30.0, (1, 3, 3), [
        mixer(B, 2, 2, 16, 16, 0.2, (4, 10000.0), dense(48), softcap=2.0, window=17, scaling=ramp(32.0, 4096, 32.0, 1.0)),
        mixer(A, 4, 1, 8, 16, 0.4, (8, 30.0), moe(5, 5, 8), softcap=6.0, scaling=wavelength(4.0, 1.0, 2.0, 16)),
        mixer(C, 6, 3, 12, 12, 0.4, (8, 64.0), dense(24))]),
    # no convolution, no cap on the logits; every token's expert wider than the routed ones; one layer
    "T": model(96, 72, 1e-4, 3, 0.5, 10.0, (7, 0, 1), None, None, None, [
        mixer(A, 6, 2, 24, 8, 0.3, (24, 10.0), moe(10, 3, 8, 64), softcap=5.0, window=64, scaling=wavelength(3.0, 2.0, 3.0, 10))]),
    # a long convolution
    "U": model(150, 56, 1e-5, 7, 0.9, 2.0, (149, 150, 1), 6, 20.0, (0, 1, 2), [
        mixer(C, 4, 2, 16, 16, 0.3, (16, 100.0), moe(4, 2, 16, 16)),
        mixer(B, 4, 2, 32, 48, 0.2, (32, 1000.0), dense(64), softcap=9.0, window=40)]),
}


def config(name):
    return cb.config_from_dict(json.loads(json.dumps(CONFIGS[name])))


def draw_tensor(n, shape, r):
    """A weight of the design from normal numbers ``r``, sized so that its mechanism matters."""
    if n.endswith("embed"):
        return 0.5 * r
    if n.endswith("bigram"):
        return 1.5 * r
    if n.endswith((".norm1", ".q.norm", ".k.norm")) or n == "final.norm":
        return 1.0 + 0.3 * r                           # plain weights
    if n.endswith(".router.b"):
        return 1.0 * r
    if n.endswith(".b"):
        return 0.4 * r
    if n.endswith(".sink"):
        return 1.0 + r
    if n.endswith(".canon1"):
        return 0.6 * r
    if n.endswith(".router") or n.endswith(".sg"):
        return 2.0 * r / shape[1] ** 0.5
    if n.endswith((".mix.q", ".mix.k", "m.q", "m.k")):
        return 1.5 * r / shape[1] ** 0.5               # scores of several units: the softmax is no average, the cap bites
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
