"""Configuration of the Nomutar decoder, read from its own config.json keys.

Nomutar is a decoder whose layers run mixer and feed-forward side by side on one norm, with a short convolution on what the
mixer reads: h = N(x), x <- x + m (mixer(h + C(h)) + ff(h)), with N an RMS norm over ``norm.groups`` equal parts of the
vector, C a causal convolution per channel (``canon.taps``) and m one number for the model (``residual_mult``).  To an
embedding row, times ``embedding.scale``, a row of a second table is added that the previous and the present token choose
(``embedding.bigram`` {buckets, mul_prev, mul_cur}).  The head is a matrix of its own, and the logits are capped softly:
``logit_softcap`` c makes them c tanh(logits / c).

config ``layers`` lists the layers in order, each with a ``type`` that names its mixer, the mixer's sizes (``mixer``) and
its feed-forward (``mlp``, or null for none).  All mixers are grouped-query softmax attention with key and value sizes of
their own, a rotation of the first ``rot.dims`` elements of a head and a ``scale``:

* ``attention``: q and k normed whole (ahead of the split into heads), rotation in halves with frequencies stretched by
  wavelength (``rot.scaling`` {factor, low, high, original}), values rotated too and the output turned back, a soft cap on the
  scores, a sliding window (``mask.size``), a learned sink a head;
* ``attention_2``: biases on q, k and v, rotation of neighbours with a ramp over the frequencies (``rot.scaling`` {factor,
  original, fast, slow}), a soft cap, a window, one added to the softmax's denominator;
* ``attention_3``: q and k normed whole, rotation in halves, every earlier key.

Feed-forwards: ``dense`` (SiLU-gated) or ``moe`` (``expert`` {ff}, ``router`` {experts, top}: the logits plus a bias choose,
the weights are the softmax over the chosen; ``shared`` {ff}: an expert for every token, times a sigmoid of one number).

``loop`` {start, stop, times}: layers start .. stop - 1 run ``times`` times in a row with the same weights and a cache of
their own every time.

The residual is kept divided by m: with y = x / m a layer is y <- y + (mixer + ff), an RMS norm of x is the same norm of y
with eps / m^2, and the embedding's two rows enter divided by m.  That is the same function, and the sums of a layer's two
products into the residual need no factor.

Tensor names: ``embed``, ``bigram``, ``final.norm``, ``head``; layer i's tensors start with ``l<i>.``: ``norm1``, ``canon1``,
``mix.{q,k,v,o}``, ``mix.{q.norm,k.norm,sink}`` or ``mix.{q.b,k.b,v.b}``, ``mlp.{gate,up,down}`` or ``mlp.router``,
``mlp.router.b``, ``mlp.e<j>.{gate,up,down}`` and ``mlp.shared.{gate,up,down,sg}``.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Dict, Optional, Tuple

from ..errors import require
from .lanizen import _int, _number
from .spec import LayerSpec, ModelSpec, PartSpec, ScheduleStep

ARCHITECTURE = "Nomutar"
MAX_POSITIONS = 1 << 24          # positions are exact as float32 up to here; the design itself sets no limit

_MLP_KINDS = ("dense", "moe")
# a layer type's fixed choices, and the keys of its rotation's scaling
_LAYER_TYPES = {
    "attention": dict(qk_norm=True, biases=False, rot_layout="halves", scaling=("wavelength", ("factor", "low", "high")),
                      rotated_values=True, sink="heads"),
    "attention_2": dict(qk_norm=False, biases=True, rot_layout="pairs", scaling=("ramp", ("factor", "fast", "slow")),
                        rotated_values=False, sink=0.0),
    "attention_3": dict(qk_norm=True, biases=False, rot_layout="halves", scaling=None, rotated_values=False, sink=None),
}


def _check_mixer(kind, m, mw):
    fixed = _LAYER_TYPES[kind]
    heads = _int(m, "heads", mw)
    kv = _int(m, "kv_heads", mw) if m.get("kv_heads") is not None else heads
    require(heads % kv == 0, f"config.json: {mw}.heads {heads} is not a multiple of kv_heads {kv}")
    dim = _int(m, "dim", mw)
    vdim = _int(m, "vdim", mw) if m.get("vdim") is not None else dim
    require(not fixed["rotated_values"] or vdim % 2 == 0, f"config.json: {mw}.vdim {vdim} must be even: its elements turn in pairs")
    _number(m, "scale", mw)
    if m.get("softcap") is not None:
        _number(m, "softcap", mw)
    if m.get("mask") is not None:
        _int(m["mask"], "size", mw + ".mask")
    rot = m.get("rot")
    dims = _int(rot, "dims", mw + ".rot", minimum=0)
    require(dims % 2 == 0 and dims <= dim, f"config.json: {mw}.rot.dims {dims} must be even and at most dim {dim}")
    _number(rot, "base", mw + ".rot")
    sc = rot.get("scaling")
    if sc is None:
        return
    sw = mw + ".rot.scaling"
    require(fixed["scaling"] is not None, f"config.json: {sw}: layers of type '{kind}' have no scaling of their rotation")
    for key in fixed["scaling"][1] + ("original",):
        _number(sc, key, sw)
    if "high" in fixed["scaling"][1]:
        require(sc["high"] > sc["low"], f"config.json: {sw}.high must be larger than low")
    else:
        require(rot["base"] != 1, f"config.json: {mw}.rot.base must not be 1 with a scaling")


def _check_mlp(mlp, lw):
    require(isinstance(mlp, dict) and mlp.get("kind") in _MLP_KINDS, f"config.json: {lw}.kind must be one of: {', '.join(_MLP_KINDS)}")
    if mlp["kind"] == "dense":
        _int(mlp, "ff", lw)
        return
    _int(mlp.get("expert"), "ff", lw + ".expert")
    r = mlp.get("router")
    experts, top = _int(r, "experts", lw + ".router"), _int(r, "top", lw + ".router")
    require(top <= experts, f"config.json: {lw}.router.top {top} exceeds experts {experts}")
    if mlp.get("shared") is not None:
        _int(mlp["shared"], "ff", lw + ".shared")


@dataclass(frozen=True)
class NomutarConfig:
    vocab: int
    width: int
    norm_eps: float
    norm_groups: int
    residual_mult: float
    embedding_scale: float
    bigram: Optional[Tuple[int, int, int]]      # (buckets, mul_prev, mul_cur)
    taps: Optional[int]
    logit_softcap: Optional[float]
    loop: Optional[Tuple[int, int, int]]        # (start, stop, times)
    layers: Tuple[Dict[str, Any], ...]          # as config.json lists them, validated

    # ---- reading -------------------------------------------------------------------------------------------------
    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "NomutarConfig":
        vocab = _int(d, "vocab", "the top level")
        width = _int(d, "width", "the top level")
        norm = d.get("norm")
        eps = _number(norm, "eps", "norm")
        groups = _int(norm, "groups", "norm") if norm.get("groups") is not None else 1
        require(width % groups == 0, f"config.json: norm.groups {groups} does not divide the width {width}")
        mult = _number(d, "residual_mult", "the top level") if d.get("residual_mult") is not None else 1.0
        emb = d.get("embedding") or {}
        scale = _number(emb, "scale", "embedding") if emb.get("scale") is not None else 1.0
        bigram = None
        if emb.get("bigram") is not None:
            b = emb["bigram"]
            bigram = (_int(b, "buckets", "embedding.bigram"), _int(b, "mul_prev", "embedding.bigram", minimum=0),
                      _int(b, "mul_cur", "embedding.bigram", minimum=0))
            require(max(bigram[1:]) <= 1 << 31, "config.json: embedding.bigram.mul_prev and mul_cur must fit in 32 bits")
        taps = None if d.get("canon") is None else _int(d["canon"], "taps", "canon")
        require(taps is None or taps <= 16, f"config.json: canon.taps {taps} exceeds the kernels' 16")
        cap = None if d.get("logit_softcap") is None else _number(d, "logit_softcap", "the top level")
        layers = d.get("layers")
        require(isinstance(layers, list) and len(layers) > 0, "config.json: 'layers' must be a non-empty list")
        checked = []
        for i, layer in enumerate(layers):
            where = f"layers[{i}]"
            require(isinstance(layer, dict), f"config.json: {where} must be an object")
            kind = layer.get("type")
            require(kind in _LAYER_TYPES, f"config.json: {where}.type '{kind}' is unknown; known: {', '.join(_LAYER_TYPES)}")
            require(isinstance(layer.get("mixer"), dict), f"config.json: {where}.mixer must be an object")
            _check_mixer(kind, layer["mixer"], where + ".mixer")
            if layer.get("mlp") is not None:
                _check_mlp(layer["mlp"], where + ".mlp")
            checked.append(copy.deepcopy(layer))
        loop = None
        if d.get("loop") is not None:
            lp = d["loop"]
            start, stop = _int(lp, "start", "loop", minimum=0), _int(lp, "stop", "loop", minimum=0)
            times = _int(lp, "times", "loop")
            require(start < stop <= len(layers), f"config.json: loop runs layers {start} .. {stop} - 1, the model has {len(layers)}")
            loop = (start, stop, times)
        return cls(vocab, width, eps, groups, mult, scale, bigram, taps, cap, loop, tuple(checked))

    def to_dict(self) -> Dict[str, Any]:
        """The config.json this configuration is read back from."""
        emb: Dict[str, Any] = {"scale": self.embedding_scale}
        if self.bigram is not None:
            emb["bigram"] = {"buckets": self.bigram[0], "mul_prev": self.bigram[1], "mul_cur": self.bigram[2]}
        d = {"architecture": ARCHITECTURE, "vocab": self.vocab, "width": self.width,
             "norm": {"eps": self.norm_eps, "groups": self.norm_groups}, "residual_mult": self.residual_mult, "embedding": emb,
             "layers": copy.deepcopy(list(self.layers))}
        if self.taps is not None:
            d["canon"] = {"taps": self.taps}
        if self.logit_softcap is not None:
            d["logit_softcap"] = self.logit_softcap
        if self.loop is not None:
            d["loop"] = {"start": self.loop[0], "stop": self.loop[1], "times": self.loop[2]}
        return d

    def describe(self) -> Dict[str, Any]:
        one = lambda l: l["type"] + (" + " + l["mlp"]["kind"] if l.get("mlp") else " (no feed-forward)")
        loop = "none" if self.loop is None else f"layers {self.loop[0]}..{self.loop[1] - 1} x {self.loop[2]}"
        return {"architecture": ARCHITECTURE, "vocab": self.vocab, "width": self.width, "norm_eps": self.norm_eps,
                "norm_groups": self.norm_groups, "residual_mult": self.residual_mult, "embedding_scale": self.embedding_scale,
                "bigram_buckets": None if self.bigram is None else self.bigram[0], "canon_taps": self.taps,
                "logit_softcap": self.logit_softcap, "loop": loop, "layers": ", ".join(one(l) for l in self.layers)}

    # ---- the architecture as data ----------------------------------------------------------------------------------
    def _norm(self, name: str) -> PartSpec:
        """A norm of the residual x = m y, given y: eps / m^2 inside the root."""
        return PartSpec("grouped_rms_norm", {"size": self.width, "eps": self.norm_eps / self.residual_mult ** 2,
                                             "groups": self.norm_groups, "tensor": name}, name)

    def _mixer(self, p: str, kind: str, m) -> PartSpec:
        fixed = _LAYER_TYPES[kind]
        rot = m["rot"]
        scaling = rot.get("scaling")
        if scaling is not None:
            scaling = dict(scaling, kind=fixed["scaling"][0])
        return PartSpec("window_attention", {
            "hidden_size": self.width, "heads": m["heads"], "kv_heads": m.get("kv_heads") or m["heads"], "dim": m["dim"],
            "vdim": m.get("vdim") or m["dim"], "conv": None, "qk_norm_eps": self.norm_eps if fixed["qk_norm"] else None,
            "qk_norm_over": "projection", "rot_dims": rot["dims"], "rot_base": rot["base"], "rot_layout": fixed["rot_layout"],
            "rot_scaling": scaling, "value_rot_base": rot["base"] if fixed["rotated_values"] else None, "scale": m["scale"],
            "window": None if m.get("mask") is None else m["mask"]["size"], "keep_first": 0, "softcap": m.get("softcap"),
            "biases": fixed["biases"], "sink": fixed["sink"],
            "names": {"q_norm": f"{p}.q.norm", "k_norm": f"{p}.k.norm"}}, p)

    def _feed_forward(self, p: str, mlp) -> PartSpec:
        if mlp["kind"] == "dense":
            return PartSpec("gated", {"hidden_size": self.width, "intermediate_size": mlp["ff"], "activation": "silu",
                                      "names": {"gate": f"{p}.gate", "up": f"{p}.up", "down": f"{p}.down"}}, p)
        r, shared = mlp["router"], mlp.get("shared")
        return PartSpec("routed_experts", {
            "hidden_size": self.width, "experts": r["experts"], "top": r["top"], "intermediate_size": mlp["expert"]["ff"],
            "groups": None, "keep_groups": None, "weight_scale": 1.0, "score": "softmax_chosen", "router_bias": True,
            "activation": "silu",
            "shared": None if shared is None else {"intermediate_size": shared["ff"], "weight": "sigmoid"}}, p)

    def to_model_spec(self) -> ModelSpec:
        layers = []
        for i, layer in enumerate(self.layers):
            p = f"l{i}"
            parts = {"norm": self._norm(f"{p}.norm1"), "mixer": self._mixer(f"{p}.mix", layer["type"], layer["mixer"])}
            if self.taps is not None:
                parts["mixer_input"] = PartSpec("residual_conv", {"hidden_size": self.width, "taps": self.taps}, f"{p}.canon1")
            if layer.get("mlp") is not None:
                parts["feed_forward"] = self._feed_forward(f"{p}.mlp", layer["mlp"])
            layers.append(LayerSpec(block="parallel_residual", parts=parts))
        n = len(layers)
        start, stop, times = self.loop or (0, 0, 0)
        order = list(range(start)) + list(range(start, stop)) * times + list(range(stop, n))
        addition = None
        if self.bigram is not None:
            addition = PartSpec("hashed_pairs", {"hidden_size": self.width, "buckets": self.bigram[0], "mul_prev": self.bigram[1],
                                                 "mul_cur": self.bigram[2], "pair_scale": 1.0 / self.residual_mult}, "bigram")
        spec = ModelSpec(
            architecture=ARCHITECTURE, vocab_size=self.vocab, hidden_size=self.width, max_positions=MAX_POSITIONS,
            embedding_name="embed", layers=tuple(layers), schedule=tuple(ScheduleStep(i) for i in order),
            final_norm=self._norm("final.norm"), head_name="head", tie_head_to_embedding=False, stop_token_ids=(),
            embedding_scale=self.embedding_scale / self.residual_mult, embedding_addition=addition,
            logit_softcap=self.logit_softcap)
        spec.validate()
        return spec
