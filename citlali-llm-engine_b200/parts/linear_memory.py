"""A mixer whose memory of a sequence is a matrix per head, a decayed sum of outer products of keys and values.

For a token with input h:  q, k (``heads`` of ``dim``), v (``heads`` of ``vdim``) and a gate (``heads`` of ``vdim``) are
projections of h without biases; ``act`` "silu": q, k and v pass SiLU; q times ``q_scale``.  Per head S [dim, vdim], zero at a
sequence's start:

* with ``decay`` (a number a head):  S <- decay S + k v^T;   o = S^T q;
* with ``gate_cap`` c (the matrix memory of xLSTM):  i = c tanh((W_i h + b_i) / c),  f = logsigmoid(c tanh((W_f h + b_f) / c)), a
  running maximum m (zero at the start):  m' = max(f + m, i);  S <- exp(f + m - m') S + exp(i - m') k v^T;  n likewise with k
  alone;  o = S^T q / (max(|n . q|, exp(-m')) + 1e-6).

The heads' results are divided by their root mean square, each by its own (``norm_over`` "head") or all together ("row"),
multiplied by a weight of heads * vdim and by sigmoid(gate), and pass the output matrix.

Everything behind the projections is float32 in the 32-bit path, and in bfloat16 for few new tokens a sequence; long runs in
bfloat16 take 64 tokens at a time through the tensor cores, with q, k, v as bfloat16 operands and state, exponents and sums in
float32.  A sequence keeps, in one float32 region: S of every head, then with a gate n of every head and m of every head.

Parameters: hidden_size, heads, dim, vdim, decay or gate_cap, act, q_scale, norm_over, norm_eps; ``names``: full tensor names by
role (q, k, v, gate, o, norm, i, f, i_bias, f_bias; the gate defaults to ``<prefix>.g``, a bias to its matrix's name with ``.b``).
"""
from __future__ import annotations

import torch

from .. import ops
from ..cache import StateRequirement
from ..errors import require
from ..weights.loader import TensorSpec
from .base import bind_vector, register_part
from .linear import DenseLinear

_CHUNK_ROWS = 32            # runs of new tokens from here on go through the tensor cores (bfloat16)


class LinearMemoryMixer:
    graph_safe = True        # slots and row ranges are read on the device; the launches depend on the counts alone
    can_overwrite = True
    kernel_sources = ("linear_memory",)

    def __init__(self, params, prefix: str):
        self.hidden = int(params["hidden_size"])
        self.H, self.D = int(params["heads"]), int(params["dim"])
        self.V = int(params.get("vdim") or self.D)
        self.eps = float(params["norm_eps"])
        self.act = params.get("act")
        require(self.act in (None, "silu"), f"{prefix}: act is 'silu' or None")
        self.q_scale = 1.0 if params.get("q_scale") is None else float(params["q_scale"])
        self.groups = {"head": self.H, "row": 1}.get(str(params.get("norm_over") or "head"))
        require(self.groups is not None, f"{prefix}: norm_over must be 'head' or 'row'")
        self.gate_cap = None if params.get("gate_cap") is None else float(params["gate_cap"])
        self.decays = None if params.get("decay") is None else [float(v) for v in params["decay"]]
        require((self.gate_cap is None) != (self.decays is None), f"{prefix}: a memory has either fixed decays or gates")
        require(self.decays is None or (len(self.decays) == self.H and all(0.0 <= v <= 1.0 for v in self.decays)),
                f"{prefix}: {self.H} heads need as many decays between 0 and 1")
        require(self.gate_cap is None or self.gate_cap > 0.0, f"{prefix}: the gates' cap must be positive")
        require(self.D <= 256, f"{prefix}: a head size of {self.D} exceeds the recurrence kernel's 256")
        n = dict(params.get("names") or {})
        self.names = {r: str(n.get(r) or f"{prefix}.{r}") for r in ("q", "k", "v", "o", "norm", "i", "f")}
        self.names["gate"] = str(n.get("gate") or f"{prefix}.g")
        for r in ("i", "f"):
            self.names[r + "_bias"] = str(n.get(r + "_bias") or self.names[r] + ".b")
        self.prefix = prefix
        nm, hd, hv = self.names, self.H * self.D, self.H * self.V
        gated = self.gate_cap is not None
        self.proj = DenseLinear([nm["q"], nm["k"], nm["v"], nm["gate"]] + ([nm["i"], nm["f"]] if gated else []),
                                [hd, hd, hv, hv] + ([self.H, self.H] if gated else []), self.hidden)
        self.o = DenseLinear([nm["o"]], [self.hidden], hv)
        self.sum_off = self.H * self.D * self.V
        self.max_off = self.sum_off + hd
        self.state_floats = self.max_off + self.H if gated else self.sum_off

    def tensor_specs(self):
        nm = self.names
        gates = [TensorSpec(nm["i_bias"], (self.H,), "state"), TensorSpec(nm["f_bias"], (self.H,), "state")] if self.gate_cap is not None else []
        return self.proj.tensor_specs() + self.o.tensor_specs() + [TensorSpec(nm["norm"], (self.H * self.V,), "gain")] + gates

    def cache_requirement(self):
        return StateRequirement((self.state_floats,), torch.float32)

    def bind(self, weights, ctx):
        self.proj.bind(weights, ctx)
        self.o.bind(weights, ctx)
        self.norm_w = bind_vector(weights, self.names["norm"], self.H * self.V, ctx)
        self.decay = self.i_bias = self.f_bias = None
        if self.decays is not None:
            self.decay = torch.tensor(self.decays, dtype=torch.float64).to(device=ctx.device, dtype=torch.float32)
        else:
            self.i_bias = bind_vector(weights, self.names["i_bias"], self.H, ctx)
            self.f_bias = bind_vector(weights, self.names["f_bias"], self.H, ctx)
        self.dtype = ctx.dtype

    def forward(self, h, batch, cache_view, residual, write_cache=True, overwrite=False):
        require(cache_view is not None and tuple(cache_view.requirement.shape) == (self.state_floats,),
                f"{self.prefix}: the memory needs its state region of {self.state_floats} floats a sequence")
        require(write_cache, f"{self.prefix}: a recurrent mixer cannot run without carrying its state")
        state, rows, H, hd, hv = cache_view.storage, batch.rows, self.H, self.H * self.D, self.H * self.V
        proj = self.proj.forward(h, out_dtype=torch.float32)
        new = lambda *shape: torch.empty(shape, dtype=torch.float32, device=proj.device)
        logs = sums = floors = None
        if self.gate_cap is not None:
            logs, sums, floors = new(rows, H, 2), new(rows, H), new(rows, H)
            at = 2 * hd + 2 * hv
            ops.memory_gates(proj[:, at:at + H], proj[:, at + H:at + 2 * H], self.i_bias, self.f_bias, self.gate_cap, state, self.max_off,
                             batch, logs, floors)
        o = new(rows, hv)
        form = ops.MEMORY_SINGLE if batch.max_new == 1 else ops.MEMORY_SCAN
        if self.dtype == torch.bfloat16 and batch.max_new >= _CHUNK_ROWS:
            form = ops.MEMORY_CHUNKS
        ops.linear_memory(proj[:, :hd], proj[:, hd:2 * hd], proj[:, 2 * hd:2 * hd + hv], state, batch, H, self.D, self.V, o, decay=self.decay,
                          logs=logs, sums=sums, sum_off=self.sum_off, act=self.act, q_scale=self.q_scale, form=form)
        y = torch.empty((rows, hv), dtype=self.dtype, device=proj.device)
        ops.linear_memory_output(o, sums, floors, proj[:, 2 * hd + hv:2 * hd + 2 * hv], self.norm_w, y, H, self.V, self.groups, self.eps)
        if overwrite:
            self.o.forward(y, out=residual)
        else:
            self.o.forward(y, accumulate_into=residual)
        return residual


register_part("mixer", "linear_memory", LinearMemoryMixer)
