"""Grouped-query attention over a sliding window that also keeps a sequence's first tokens, with a short causal
convolution in front and heads whose keys and values may differ in size.

For a token with input h:  q (``heads`` of ``dim``), k (``kv_heads`` of ``dim``) and v (``kv_heads`` of ``vdim``) are
projections of h, without biases unless ``biases`` says otherwise (a bias a channel, added to what the convolution gives;
with no convolution: to the projection); each channel then passes a causal convolution over time (``conv`` taps, no bias, zeros before
the sequence's start; None: none).  q and k heads pass an RMS norm over ``dim`` with a weight shared by the heads
(``qk_norm_eps`` None: none; ``qk_norm_over`` "projection": over all of q and over all of k at once, ahead of the split into
heads, with weights of those sizes), then the rotation of the first ``rot_dims`` elements of a head in neighbouring pairs
(2i, 2i+1), or with ``rot_layout`` "halves" in pairs (i, i + rot_dims/2), by position * ``rot_base``^(-2i/rot_dims), the
frequencies stretched by ``rot_scaling`` (see :func:`~.rotary.rotation_table`) if given; the rest of a head passes unchanged,
and so does v, unless ``value_rot_base`` b is given: then v is rotated over its whole length, pair m by position *
b^(-2m/vdim), before it is cached, and a head's output is turned back by the same angles of the row's own position (ahead of
the gate), so that a value is seen rotated by its distance.  Query head j reads key
head j // (heads / kv_heads).  Position p sees key j if j <= p and (p - j < ``window`` or j < ``keep_first``); ``window``
None: every earlier key.  Kept tokens keep their own positions.  Scores times ``scale``, then with ``softcap`` c the
score s becomes c tanh(s / c); a softmax over the visible keys (``sink``: its denominator also counts exp(z), with z a
learned number a head ("heads") or the given number; z is not scaled, not capped, and has no value), the weighted sum of values; with ``gate``
"elements" the heads side by side are multiplied element by element by sigmoid(W_g h), a projection of the same input
without a bias that rides in the q | k | v product; then the output matrix.

The convolution (or the norms over the whole projections), head norm, rotations and the cache write are one kernel; scores and softmax are float32.  The cache holds
keys and values in pages (``KVRequirement`` with the window and the kept tokens: pages that hold neither are given back);
beside it a sequence keeps the last ``conv - 1`` projected rows in a float32 region, so the mixer asks for two caches.

Parameters: hidden_size, heads, kv_heads, dim, vdim, conv, qk_norm_eps, rot_dims, rot_base, scale, window, keep_first,
softcap, biases, gate, qk_norm_over, rot_layout, rot_scaling, value_rot_base, value_rot_layout (default: rot_layout), sink;
``names``: full tensor names by role (q, k, v, q_conv, k_conv, v_conv, q_norm, k_norm, o, gate, sink,
q_bias, k_bias, v_bias; the biases default to the matrix's name with ``.b``, the gate to ``<prefix>.g``).
"""
from __future__ import annotations

import torch

from .. import ops
from ..cache import KVRequirement, StateRequirement
from ..errors import require
from ..weights.loader import TensorSpec
from .base import bind_vector, register_part
from .delta import bind_float32
from .linear import DenseLinear
from .rotary import rotation_table

_ROLES = ("q", "k", "v", "q_conv", "k_conv", "v_conv", "q_norm", "k_norm", "o", "sink")
_LAYOUTS = ("pairs", "halves")


class WindowAttention:
    graph_safe = True            # slots and positions are read on the device; the launch depends on the row count alone
    can_overwrite = True

    def __init__(self, params, prefix: str):
        self.hidden = int(params["hidden_size"])
        self.nq, self.nkv = int(params["heads"]), int(params.get("kv_heads") or params["heads"])
        self.d = int(params["dim"])
        self.vd = int(params.get("vdim") or self.d)
        self.has_conv = params.get("conv") is not None
        self.taps = int(params.get("conv") or 1)
        self.eps = params.get("qk_norm_eps")
        self.rot_dims = int(params.get("rot_dims") or 0)
        self.rot_base = float(params.get("rot_base") or 1.0)
        self.scale = float(params["scale"])
        self.window = None if params.get("window") is None else int(params["window"])
        self.keep_first = int(params.get("keep_first") or 0) if self.window is not None else 0
        self.softcap = float(params.get("softcap") or 0.0)
        self.has_biases = bool(params.get("biases", False))
        self.has_gate = params.get("gate") is not None
        require(params.get("gate") in (None, "elements"), f"{prefix}: gate must be 'elements' or None")
        require(self.softcap >= 0.0, f"{prefix}: softcap must be positive or None")
        self.norm_whole = {"head": False, "projection": True}.get(str(params.get("qk_norm_over") or "head"))
        require(self.norm_whole is not None, f"{prefix}: qk_norm_over must be 'head' or 'projection'")
        self.rot_layout = str(params.get("rot_layout") or "pairs")
        self.rot_scaling = params.get("rot_scaling")
        self.v_base = None if params.get("value_rot_base") is None else float(params["value_rot_base"])
        self.v_layout = str(params.get("value_rot_layout") or self.rot_layout)
        require(self.rot_layout in _LAYOUTS and self.v_layout in _LAYOUTS, f"{prefix}: a rotation's layout is 'pairs' or 'halves'")
        require(self.v_base is None or self.vd % 2 == 0, f"{prefix}: rotated values need an even size, not {self.vd}")
        self.sink = params.get("sink")
        require(self.sink is None or self.sink == "heads" or isinstance(self.sink, (int, float)),
                f"{prefix}: sink must be 'heads', a number or None")
        # one kernel prepares heads behind a convolution or with a norm a head, another everything else
        self.plain_heads = not self.has_conv and (self.eps is None or self.norm_whole)
        require(self.plain_heads or (not self.norm_whole and self.rot_layout == "pairs" and self.v_base is None
                                     and (self.rot_scaling is None or self.rot_scaling["kind"] != "ramp")),
                f"{prefix}: a convolution or a norm a head goes with the 'pairs' rotation of q and k only")
        require(self.nq % self.nkv == 0, f"{prefix}: {self.nq} query heads are not a multiple of {self.nkv} key/value heads")
        require(self.rot_dims % 2 == 0 and self.rot_dims <= self.d,
                f"{prefix}: {self.rot_dims} rotated elements must be even and at most the head size {self.d}")
        require(self.window is None or self.window > 0, f"{prefix}: window must be positive or None")
        require(self.d <= 256 and self.vd <= 256, f"{prefix}: heads of {self.d} / {self.vd} exceed the kernels' 256")
        n = dict(params.get("names") or {})
        self.names = {r: str(n.get(r) or f"{prefix}.{r}") for r in _ROLES}
        self.names["gate"] = str(n.get("gate") or f"{prefix}.g")
        for r in ("q", "k", "v"):
            self.names[r + "_bias"] = str(n.get(r + "_bias") or self.names[r] + ".b")
        self.prefix = prefix
        self.C = (self.nq + self.nkv) * self.d + self.nkv * self.vd
        nm = self.names
        self.sizes = [self.nq * self.d, self.nkv * self.d, self.nkv * self.vd]
        self.qkv = DenseLinear([nm["q"], nm["k"], nm["v"]] + ([nm["gate"]] if self.has_gate else []),
                               self.sizes + ([self.nq * self.vd] if self.has_gate else []), self.hidden)
        self.o = DenseLinear([nm["o"]], [self.hidden], self.nq * self.vd)

    def tensor_specs(self):
        nm = self.names
        specs = self.qkv.tensor_specs() + self.o.tensor_specs()
        if self.has_conv:
            specs += [TensorSpec(nm["q_conv"], (self.nq * self.d, self.taps), "state"),
                      TensorSpec(nm["k_conv"], (self.nkv * self.d, self.taps), "state"),
                      TensorSpec(nm["v_conv"], (self.nkv * self.vd, self.taps), "state")]
        if self.eps is not None:
            specs += [TensorSpec(nm["q_norm"], (self.norm_sizes()[0],), "gain"), TensorSpec(nm["k_norm"], (self.norm_sizes()[1],), "gain")]
        if self.sink == "heads":
            specs.append(TensorSpec(nm["sink"], (self.nq,), "state"))
        if self.has_biases:
            specs += [TensorSpec(nm[r + "_bias"], (size,), "state") for r, size in zip(("q", "k", "v"), self.sizes)]
        return specs

    def kernel_sources(self, dtype):
        prepared = ("heads_prepare",) if self.plain_heads else ("window_attention",)
        kept = ("recurrent",) if self.taps > 1 else ()
        if dtype == torch.float32 or self.d % 8 or self.vd % 8 or self.keep_first:
            return prepared + kept + ("window_attention",)
        return prepared + kept + ("attention_decode", "attention_prefill") + (("attention_prefill_tc",) if self.d == self.vd == 128 else ())

    def norm_sizes(self):
        return (self.nq * self.d, self.nkv * self.d) if self.norm_whole else (self.d, self.d)

    def cache_requirement(self):
        kv = KVRequirement(self.nkv, self.d, self.window, value_dim=self.vd, keep_first=self.keep_first)
        if self.taps > 1:
            return (kv, StateRequirement(((self.taps - 1) * self.C,), torch.float32))
        return (kv,)

    def bind(self, weights, ctx):
        nm = self.names
        self.qkv.bind(weights, ctx)
        self.o.bind(weights, ctx)
        if self.has_conv:
            self.conv_w = torch.cat([bind_float32(weights, nm["q_conv"], (self.nq * self.d, self.taps), ctx),
                                     bind_float32(weights, nm["k_conv"], (self.nkv * self.d, self.taps), ctx),
                                     bind_float32(weights, nm["v_conv"], (self.nkv * self.vd, self.taps), ctx)], 0).contiguous()
        else:
            self.conv_w = torch.ones((self.C, 1), dtype=torch.float32, device=ctx.device)
        self.q_gain = self.k_gain = None
        if self.eps is not None:
            self.q_gain = bind_float32(weights, nm["q_norm"], (self.norm_sizes()[0],), ctx)
            self.k_gain = bind_float32(weights, nm["k_norm"], (self.norm_sizes()[1],), ctx)
        self.bias = None
        if self.has_biases:
            self.bias = torch.cat([bind_vector(weights, nm[r + "_bias"], size, ctx)
                                   for r, size in zip(("q", "k", "v"), self.sizes)]).contiguous()
        freq, self.amplitude = rotation_table(self.rot_dims, self.rot_base, self.rot_scaling)
        self.inv_freq = freq.to(ctx.device)
        self.v_freq = None if self.v_base is None else rotation_table(self.vd, self.v_base)[0].to(ctx.device)
        self.sinks = None
        if self.sink == "heads":
            self.sinks = bind_vector(weights, nm["sink"], self.nq, ctx)
        elif self.sink is not None:
            self.sinks = torch.full((self.nq,), float(self.sink), dtype=torch.float32, device=ctx.device)
        self.dtype = ctx.dtype
        self.error_flag = ctx.error_flag

    def forward(self, h, batch, cache_view, residual, write_cache=True, overwrite=False):
        require(isinstance(cache_view, tuple) and len(cache_view) == (2 if self.taps > 1 else 1),
                f"{self.prefix}: attention behind a convolution needs a key/value cache and a region for its last inputs")
        require(write_cache, f"{self.prefix}: this attention always keeps its own keys and values")
        kv = cache_view[0]
        state = cache_view[1].storage if self.taps > 1 else None
        rows = batch.rows
        proj = self.qkv.forward(h, out_dtype=torch.float32)
        q = torch.empty((rows, self.nq * self.d), dtype=self.dtype, device=proj.device)
        turns = None
        if self.plain_heads:
            if self.v_freq is not None:
                turns = torch.empty((rows, self.vd // 2, 2), dtype=torch.float32, device=proj.device)
            ops.heads_prepare(proj, batch, kv, q, self.nq, self.nkv, self.d, self.vd, bias=self.bias, q_gain=self.q_gain,
                              k_gain=self.k_gain, eps=float(self.eps or 0.0), inv_freq=self.inv_freq, rot_dims=self.rot_dims,
                              rot_pairs=self.rot_layout == "pairs", amplitude=self.amplitude, v_freq=self.v_freq,
                              v_pairs=self.v_layout == "pairs", turns=turns)
        else:
            ops.conv_heads_prepare(proj, self.conv_w, state, 0, self.q_gain, self.k_gain, self.inv_freq, self.rot_dims, batch, kv,
                                   q, self.nq, self.nkv, self.d, self.vd, float(self.eps or 0.0), bias=self.bias)
        if self.taps > 1:
            ops.conv_keep(proj, proj.shape[1], self.taps, self.C, state, 0, batch)
        out = torch.empty((rows, self.nq * self.vd), dtype=self.dtype, device=proj.device)
        ops.attention_window(q, kv, batch, out, self.nq, self.nkv, self.d, self.vd, self.window, self.keep_first, self.scale,
                             softcap=self.softcap, gate=proj[:, self.C:] if self.has_gate else None, sink=self.sinks,
                             turns=turns, turn_pairs=self.v_layout == "pairs", error_flag=self.error_flag)
        if overwrite:
            self.o.forward(out, out=residual)
        else:
            self.o.forward(out, accumulate_into=residual)
        return residual


register_part("mixer", "window_attention", WindowAttention)
