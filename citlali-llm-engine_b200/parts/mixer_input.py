"""What a mixer reads instead of the normed rows themselves.

Interface of a part in the role ``mixer_input``: ``__init__(params, prefix)``, ``tensor_specs()``, ``bind(weights, ctx)``,
``cache_requirement()`` and ``forward(norm, x, batch, cache_view) -> (h, m)``: the normed rows of the residual ``x``, which
the feed-forward reads, and the rows the mixer reads.

``residual_conv``: m = h + conv(h), a causal convolution over time on each channel, conv(h)_t = sum_j w[:, j] h_(t - taps + 1 +
j), zeros ahead of the first token, no bias.  The norm in front (an RMS norm over the row or over equal parts of it) and the
convolution are one kernel; a sequence keeps its last ``taps - 1`` rows h, unrounded.  Parameters: hidden_size, taps,
``tensor`` (the weights' full name, [hidden, taps]).
"""
from __future__ import annotations

import torch

from .. import ops
from ..cache import StateRequirement
from ..errors import require
from ..weights.loader import TensorSpec
from .base import register_part
from .delta import bind_float32


class ResidualConv:
    graph_safe = True
    kernel_sources = ("group_norm",)

    def __init__(self, params, prefix: str):
        self.hidden, self.taps = int(params["hidden_size"]), int(params["taps"])
        self.name = str(params.get("tensor") or prefix)
        require(1 <= self.taps <= 16, f"{prefix}: a convolution of {self.taps} taps (1 to 16)")

    def tensor_specs(self):
        return [TensorSpec(self.name, (self.hidden, self.taps), "state")]

    def cache_requirement(self):
        return StateRequirement(((self.taps - 1) * self.hidden,), torch.float32) if self.taps > 1 else None

    def bind(self, weights, ctx):
        self.taps_w = bind_float32(weights, self.name, (self.hidden, self.taps), ctx)
        self.dtype = ctx.dtype

    def forward(self, norm, x, batch, cache_view):
        require(callable(getattr(norm, "group_terms", None)), "the norm ahead of a residual convolution must be an RMS norm")
        gain, groups, eps = norm.group_terms()
        h = torch.empty(x.shape, dtype=self.dtype, device=x.device)
        m = torch.empty_like(h)
        ops.group_norm_conv(x, gain, groups, eps, self.taps_w, cache_view.storage if self.taps > 1 else None, batch, h, m)
        return h, m


register_part("mixer_input", "residual_conv", ResidualConv)
