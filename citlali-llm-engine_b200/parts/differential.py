"""Differential attention: every head has two softmax maps over the same values, and the second one's result, times one
number of the layer, is taken from the first one's.

For a token with input h:  q (``heads`` times two maps of ``dim``), k (``kv_heads`` times two maps of ``dim``) and v
(``kv_heads`` of ``vdim``) are projections of h without biases, laid out head by head as [map 1, map 2]; query head j reads
key/value head j // (heads / kv_heads).  The first ``rot_dims`` elements of every map of q and k turn by position *
``rot_base``^(-2i/rot_dims), in neighbouring pairs or (``rot_layout`` "halves") in halves.  Each map is a softmax of its own over
the keys j <= p with p - j < ``window`` (None: every earlier key), scores times ``scale``.  With the maps' results a1, a2 and

    lambda = exp(sum lq1 lk1) - exp(sum lq2 lk2) + diff:      o = a1 - lambda a2;   o <- (1 - diff) o / sqrt(mean(o^2) + eps)

over a head's ``vdim`` elements, and with ``gate`` "heads" o <- sigmoid(W_g h)_head o (a row of the same product as q, k, v); then
the output matrix.

How it runs: a cached key holds both maps side by side (2 dim elements), and a query head becomes two heads of 2 dim elements, each
with one map and zeros in the other's place.  The attention kernels then see 2 heads query heads over kv_heads key/value heads of
(2 dim, vdim): keys and values are read once for both maps of all heads that share them.  The maps' results stay float32 until
they have been combined, normed and gated by one kernel.

Parameters: hidden_size, heads, kv_heads, dim, vdim, rot_dims, rot_base, rot_layout, scale, window, diff, eps, gate; ``names``: full
tensor names by role (q, k, v, o, gate, lq1, lk1, lq2, lk2; the gate defaults to ``<prefix>.g``).
"""
from __future__ import annotations

import math

import torch

from .. import ops
from ..cache import KVRequirement
from ..errors import require
from ..weights.loader import TensorSpec
from .base import register_part
from .linear import DenseLinear
from .rotary import rotation_table

MAPS = 2
_LAMBDA = ("lq1", "lk1", "lq2", "lk2")


class DifferentialAttention:
    graph_safe = True
    can_overwrite = True

    def __init__(self, params, prefix: str):
        self.hidden = int(params["hidden_size"])
        self.H, self.G = int(params["heads"]), int(params.get("kv_heads") or params["heads"])
        self.d = int(params["dim"])
        self.vd = int(params.get("vdim") or self.d)
        self.rot_dims = int(params.get("rot_dims") or 0)
        self.rot_base = float(params.get("rot_base") or 1.0)
        self.rot_layout = str(params.get("rot_layout") or "pairs")
        self.scale = float(params["scale"])
        self.window = None if params.get("window") is None else int(params["window"])
        self.diff = float(params["diff"])
        self.eps = float(params["eps"])
        self.has_gate = params.get("gate") is not None
        require(params.get("gate") in (None, "heads"), f"{prefix}: gate must be 'heads' or None")
        require(self.rot_layout in ("pairs", "halves"), f"{prefix}: a rotation's layout is 'pairs' or 'halves'")
        require(self.H % self.G == 0, f"{prefix}: {self.H} query heads are not a multiple of {self.G} key/value heads")
        require(self.rot_dims % 2 == 0 and self.rot_dims <= self.d,
                f"{prefix}: {self.rot_dims} rotated elements must be even and at most a map's size {self.d}")
        require(self.window is None or self.window > 0, f"{prefix}: window must be positive or None")
        require(MAPS * self.d <= 256 and self.vd <= 256, f"{prefix}: two maps of {self.d} or values of {self.vd} exceed the kernels' 256")
        n = dict(params.get("names") or {})
        self.names = {r: str(n.get(r) or f"{prefix}.{r}") for r in ("q", "k", "v", "o") + _LAMBDA}
        self.names["gate"] = str(n.get("gate") or f"{prefix}.g")
        self.prefix = prefix
        nm, key = self.names, MAPS * self.d
        sizes = [self.H * key, self.G * key, self.G * self.vd]
        self.C = sum(sizes)
        self.qkv = DenseLinear([nm["q"], nm["k"], nm["v"]] + ([nm["gate"]] if self.has_gate else []),
                               sizes + ([self.H] if self.has_gate else []), self.hidden)
        self.o = DenseLinear([nm["o"]], [self.hidden], self.H * self.vd)

    def tensor_specs(self):
        return (self.qkv.tensor_specs() + self.o.tensor_specs()
                + [TensorSpec(self.names[r], (self.d,), "state") for r in _LAMBDA])

    def kernel_sources(self, dtype):
        own = ("heads_prepare", "differential")
        if dtype == torch.float32 or self.d % 4 or self.vd % 8:
            return own + ("window_attention",)
        return own + ("attention_decode", "attention_prefill") + (("attention_prefill_tc",) if MAPS * self.d == self.vd == 128 else ())

    def cache_requirement(self):
        return (KVRequirement(self.G, MAPS * self.d, self.window, value_dim=self.vd),)

    def bind(self, weights, ctx):
        self.qkv.bind(weights, ctx)
        self.o.bind(weights, ctx)
        vectors = []
        for r in _LAMBDA:
            h = weights[self.names[r]]
            require(tuple(h.shape) == (self.d,), f"unexpected tensor shape for {self.names[r]}: got {list(h.shape)}, expected {[self.d]}")
            vectors.append(h.tensor.to(device="cpu", dtype=torch.float64))
        lq1, lk1, lq2, lk2 = vectors
        self.lam = math.exp(float((lq1 * lk1).sum())) - math.exp(float((lq2 * lk2).sum())) + self.diff
        self.inv_freq = rotation_table(self.rot_dims, self.rot_base)[0].to(ctx.device)
        self.dtype = ctx.dtype
        self.error_flag = ctx.error_flag

    def forward(self, h, batch, cache_view, residual, write_cache=True, overwrite=False):
        require(isinstance(cache_view, tuple) and len(cache_view) == 1, f"{self.prefix}: differential attention needs its key/value cache")
        require(write_cache, f"{self.prefix}: this attention always keeps its own keys and values")
        kv, rows, key = cache_view[0], batch.rows, MAPS * self.d
        proj = self.qkv.forward(h, out_dtype=torch.float32)
        q = torch.empty((rows, self.H * MAPS * key), dtype=self.dtype, device=proj.device)
        ops.heads_prepare(proj, batch, kv, q, self.H, self.G, key, self.vd, inv_freq=self.inv_freq, rot_dims=self.rot_dims,
                          rot_pairs=self.rot_layout == "pairs", maps=MAPS)
        maps = torch.empty((rows, self.H * MAPS * self.vd), dtype=torch.float32, device=proj.device)
        ops.attention_window(q, kv, batch, maps, self.H * MAPS, self.G, key, self.vd, self.window, 0, self.scale,
                             error_flag=self.error_flag)
        out = torch.empty((rows, self.H * self.vd), dtype=self.dtype, device=proj.device)
        ops.differential_output(maps, self.lam, 1.0 - self.diff, self.eps, proj[:, self.C:] if self.has_gate else None, out, self.H, self.vd)
        if overwrite:
            self.o.forward(out, out=residual)
        else:
            self.o.forward(out, accumulate_into=residual)
        return residual


register_part("mixer", "differential_attention", DifferentialAttention)
