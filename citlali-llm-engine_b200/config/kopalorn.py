"""Configuration of the Kopalorn decoder, read from its own config.json keys.

Kopalorn is a decoder with a layer norm (weight and bias) in front of every sub-layer and another on what it gives:
x <- x + m N1b(mixer(N1(x))), then x <- x + m N2b(ff(N2(x))), with m one number for the model (``residual_mult``).  The head is
a matrix of its own.  config ``layers`` lists the layers in order, each with a ``type`` that names its mixer, the mixer's sizes
(``mixer``) and its feed-forward (``mlp``, or null for none):

* ``attention``: differential attention over a sliding window (``mask.size``): two softmax maps a head with a key half of their
  own over the same values, the second one's result times a learned number (with the constant ``diff``) taken from the first
  one's, each head normed, a gate a head; the first ``rot.dims`` elements of a map turn in neighbouring pairs;
* ``mlstm``: the matrix memory of xLSTM with exponential gates (``gate_cap``) and a running maximum, each head normed, a gate an
  element;
* ``parallel``: two mixers on the same input, ``left`` grouped-query softmax attention over every earlier key (biases on q, k and
  v, no rotation, a gate an element), ``right`` a linear attention with a fixed decay a head (``decay``), SiLU on q, k and v, the
  heads normed together, a gate an element; the result is half the sum of both, each first RMS-normed.

Feed-forward: ``moe``: experts without a gate (``expert`` {ff}; the activation is relu squared), sigmoid scores, ``router`` {experts,
top, scale, groups {count, keep}}: a correction an expert takes part in every choice, a group's score is the sum of its two
largest, the weights are the chosen experts' scores over their sum, times ``scale``; ``shared`` {ff}: an expert for every token,
times a sigmoid of one number.

``loop`` {start, stop, times}: layers start .. stop - 1 run ``times`` times in a row with the same weights and a cache or state of
their own every time; ahead of every pass a vector of its own (row t of ``loop.step``) is added to the residual, ahead of every pass
but the first the embedding's rows as well.

The multiplier m is folded into the weight and the bias of the norms behind the sub-layers, in 32-bit.

Tensor names: ``embed``, ``loop.step``, ``final.norm``, ``final.norm.b``, ``head``; layer i's tensors start with ``l<i>.``:
``norm1``, ``norm1b``, ``norm2``, ``norm2b`` (each with ``.b``), ``mix.{q,k,v,g,o}``, ``mix.{lq1,lk1,lq2,lk2}`` or ``mix.{i,i.b,f,f.b,
norm}``, or ``mix.left.{q,q.b,k,k.b,v,v.b,g,o,out}`` and ``mix.right.{q,k,v,g,o,norm,out}``; ``mlp.router``, ``mlp.correction``,
``mlp.e<j>.{up,down}`` and ``mlp.shared.{up,down,sg}``.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Dict, Optional, Tuple

from ..errors import require
from .lanizen import _int, _number
from .spec import LayerSpec, ModelSpec, PartSpec, ScheduleStep

ARCHITECTURE = "Kopalorn"
MAX_POSITIONS = 1 << 24          # positions are exact as float32 up to here; the design itself sets no limit

_LAYER_TYPES = ("attention", "mlstm", "parallel")
_MLP_KINDS = ("moe",)


def _check_heads(m, mw):
    """Grouped heads with key and value sizes of their own."""
    heads = _int(m, "heads", mw)
    kv = _int(m, "kv_heads", mw) if m.get("kv_heads") is not None else heads
    require(heads % kv == 0, f"config.json: {mw}.heads {heads} is not a multiple of kv_heads {kv}")
    _int(m, "dim", mw)
    if m.get("vdim") is not None:
        _int(m, "vdim", mw)


def _check_mixer(kind, m, mw):
    if kind == "attention":
        _check_heads(m, mw)
        _number(m, "scale", mw)
        _number(m, "diff", mw, positive=False)
        if m.get("mask") is not None:
            _int(m["mask"], "size", mw + ".mask")
        if m.get("rot") is not None:
            dims = _int(m["rot"], "dims", mw + ".rot", minimum=0)
            require(dims % 2 == 0 and dims <= m["dim"], f"config.json: {mw}.rot.dims {dims} must be even and at most dim {m['dim']}")
            _number(m["rot"], "base", mw + ".rot")
    elif kind == "mlstm":
        _check_heads(m, mw)
        require(m.get("kv_heads") is None or m["kv_heads"] == m["heads"], f"config.json: {mw}: the matrix memory has a key a head")
        _number(m, "gate_cap", mw)
    else:
        for side in ("left", "right"):
            require(isinstance(m.get(side), dict), f"config.json: {mw}.{side} must be an object")
            _check_heads(m[side], f"{mw}.{side}")
        _number(m["left"], "scale", mw + ".left")
        decay = m["right"].get("decay")
        require(isinstance(decay, list) and len(decay) == m["right"]["heads"]
                and all(isinstance(v, (int, float)) and not isinstance(v, bool) and 0 <= v <= 1 for v in decay),
                f"config.json: {mw}.right.decay must list a number between 0 and 1 for each of the {m['right']['heads']} heads")


def _check_mlp(mlp, lw):
    require(isinstance(mlp, dict) and mlp.get("kind") in _MLP_KINDS, f"config.json: {lw}.kind must be one of: {', '.join(_MLP_KINDS)}")
    _int(mlp.get("expert"), "ff", lw + ".expert")
    r, rw = mlp.get("router"), lw + ".router"
    experts, top = _int(r, "experts", rw), _int(r, "top", rw)
    if r.get("scale") is not None:
        _number(r, "scale", rw, positive=False)
    reach = experts
    if r.get("groups") is not None:
        count, keep = _int(r["groups"], "count", rw + ".groups"), _int(r["groups"], "keep", rw + ".groups")
        require(experts % count == 0, f"config.json: {rw}.experts {experts} do not form {count} equal groups")
        require(keep <= count, f"config.json: {rw}.groups.keep {keep} exceeds count {count}")
        reach = keep * (experts // count)
    require(top <= reach, f"config.json: {rw}.top {top} exceeds the {reach} experts that can be chosen")
    if mlp.get("shared") is not None:
        _int(mlp["shared"], "ff", lw + ".shared")


@dataclass(frozen=True)
class KopalornConfig:
    vocab: int
    width: int
    norm_eps: float
    residual_mult: float
    loop: Optional[Tuple[int, int, int]]        # (start, stop, times)
    layers: Tuple[Dict[str, Any], ...]          # as config.json lists them, validated

    # ---- reading -------------------------------------------------------------------------------------------------
    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "KopalornConfig":
        vocab = _int(d, "vocab", "the top level")
        width = _int(d, "width", "the top level")
        eps = _number(d.get("norm"), "eps", "norm")
        mult = _number(d, "residual_mult", "the top level", positive=False) if d.get("residual_mult") is not None else 1.0
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
        return cls(vocab, width, eps, mult, loop, tuple(checked))

    def to_dict(self) -> Dict[str, Any]:
        """The config.json this configuration is read back from."""
        d = {"architecture": ARCHITECTURE, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
             "residual_mult": self.residual_mult, "layers": copy.deepcopy(list(self.layers))}
        if self.loop is not None:
            d["loop"] = {"start": self.loop[0], "stop": self.loop[1], "times": self.loop[2]}
        return d

    def describe(self) -> Dict[str, Any]:
        one = lambda l: l["type"] + (" + " + l["mlp"]["kind"] if l.get("mlp") else " (no feed-forward)")
        loop = "none" if self.loop is None else f"layers {self.loop[0]}..{self.loop[1] - 1} x {self.loop[2]}"
        return {"architecture": ARCHITECTURE, "vocab": self.vocab, "width": self.width, "norm_eps": self.norm_eps,
                "residual_mult": self.residual_mult, "loop": loop, "layers": ", ".join(one(l) for l in self.layers)}

    # ---- the architecture as data ----------------------------------------------------------------------------------
    def _norm(self, name: str, scale: float = 1.0) -> PartSpec:
        return PartSpec("layer_norm", {"size": self.width, "eps": self.norm_eps, "tensor": name, "bias": name + ".b", "scale": scale}, name)

    def _attention(self, p: str, m) -> PartSpec:
        rot = m.get("rot") or {}
        return PartSpec("differential_attention", {
            "hidden_size": self.width, "heads": m["heads"], "kv_heads": m.get("kv_heads"), "dim": m["dim"], "vdim": m.get("vdim"),
            "rot_dims": rot.get("dims", 0), "rot_base": rot.get("base", 1.0), "rot_layout": "pairs", "scale": m["scale"],
            "window": None if m.get("mask") is None else m["mask"]["size"], "diff": m["diff"], "eps": self.norm_eps, "gate": "heads"}, p)

    def _mlstm(self, p: str, m) -> PartSpec:
        return PartSpec("linear_memory", {
            "hidden_size": self.width, "heads": m["heads"], "dim": m["dim"], "vdim": m.get("vdim"), "gate_cap": m["gate_cap"], "act": None,
            "q_scale": m["dim"] ** -0.5, "norm_over": "head", "norm_eps": self.norm_eps}, p)

    def _parallel(self, p: str, m) -> PartSpec:
        l, r = m["left"], m["right"]
        left = PartSpec("window_attention", {
            "hidden_size": self.width, "heads": l["heads"], "kv_heads": l.get("kv_heads"), "dim": l["dim"], "vdim": l.get("vdim"), "conv": None,
            "qk_norm_eps": None, "rot_dims": 0, "scale": l["scale"], "window": None, "biases": True, "gate": "elements"}, p + ".left")
        right = PartSpec("linear_memory", {
            "hidden_size": self.width, "heads": r["heads"], "dim": r["dim"], "vdim": r.get("vdim"), "decay": list(r["decay"]), "act": "silu",
            "norm_over": "row", "norm_eps": self.norm_eps}, p + ".right")
        return PartSpec("parallel", {"left": left, "right": right, "left_scale": 0.5, "right_scale": 0.5,
                                     "out_norms": {"size": self.width, "eps": self.norm_eps, "left": p + ".left.out",
                                                   "right": p + ".right.out"}}, p)

    def _feed_forward(self, p: str, mlp) -> PartSpec:
        r, shared, groups = mlp["router"], mlp.get("shared"), mlp["router"].get("groups")
        return PartSpec("routed_experts", {
            "hidden_size": self.width, "experts": r["experts"], "top": r["top"], "intermediate_size": mlp["expert"]["ff"],
            "groups": None if groups is None else groups["count"], "keep_groups": None if groups is None else groups["keep"],
            "group_score": "top2_sum", "weight_scale": r.get("scale"), "score": "sigmoid", "correction": True, "renormalise": True,
            "activation": "relu_squared",
            "shared": None if shared is None else {"intermediate_size": shared["ff"], "weight": "sigmoid"}}, p)

    def to_model_spec(self) -> ModelSpec:
        mixers = {"attention": self._attention, "mlstm": self._mlstm, "parallel": self._parallel}
        layers = []
        for i, layer in enumerate(self.layers):
            p = f"l{i}"
            parts = {"mixer_norm": self._norm(f"{p}.norm1"), "mixer": mixers[layer["type"]](f"{p}.mix", layer["mixer"]),
                     "mixer_out_norm": self._norm(f"{p}.norm1b", self.residual_mult)}
            if layer.get("mlp") is not None:
                parts.update({"feed_forward_norm": self._norm(f"{p}.norm2"), "feed_forward": self._feed_forward(f"{p}.mlp", layer["mlp"]),
                              "feed_forward_out_norm": self._norm(f"{p}.norm2b", self.residual_mult)})
            layers.append(LayerSpec(block="sandwich_norm", parts=parts))
        n = len(layers)
        order = list(range(n))
        if self.loop is not None:
            start, stop, times = self.loop
            layers.append(LayerSpec(block="input_addition", parts={},
                                    block_params={"hidden_size": self.width, "passes": times, "steps": "loop.step"}))
            order = list(range(start)) + ([n] + list(range(start, stop))) * times + list(range(stop, n))
        spec = ModelSpec(
            architecture=ARCHITECTURE, vocab_size=self.vocab, hidden_size=self.width, max_positions=MAX_POSITIONS,
            embedding_name="embed", layers=tuple(layers), schedule=tuple(ScheduleStep(i) for i in order),
            final_norm=self._norm("final.norm"), head_name="head", tie_head_to_embedding=False, stop_token_ids=())
        spec.validate()
        return spec
