"""Embeddings that add to a token's row something that depends on more than the token.

Interface of an embedding part (role ``embedding``): ``__init__(params, prefix)``, ``tensor_specs()``, ``bind(weights, ctx)``,
``cache_requirement()`` -> what it keeps per sequence between steps (or None), and
``forward(table, batch, x, cache_view, error_flag, scale)``, which fills the float32 rows ``x`` with
``table[token] * scale`` plus its own addition.

``hashed_pairs``: a row of a second table, chosen by the token before and the token: row
``(previous * mul_prev + token * mul_cur) mod buckets`` and, for a sequence's first token, row ``buckets`` (the last one).
The rows are multiplied by ``pair_scale`` (default 1) as they are added; gather, scales and sum are one kernel.  A sequence
keeps its last token (one int32).  Parameters: hidden_size, buckets, mul_prev, mul_cur, pair_scale, ``tensor`` (the table's
full name).
"""
from __future__ import annotations

import torch

from .. import ops
from ..cache import StateRequirement
from ..errors import require
from ..weights.loader import TensorSpec
from .base import register_part


class HashedPairEmbedding:
    graph_safe = True

    def __init__(self, params, prefix: str):
        self.hidden, self.buckets = int(params["hidden_size"]), int(params["buckets"])
        self.mul_prev, self.mul_cur = int(params["mul_prev"]), int(params["mul_cur"])
        self.pair_scale = float(params.get("pair_scale", 1.0))
        self.name = str(params.get("tensor") or prefix)
        require(self.buckets > 0, f"{prefix}: {self.buckets} buckets")
        require(max(abs(self.mul_prev), abs(self.mul_cur)) <= 1 << 31, f"{prefix}: multipliers of more than 32 bits")

    def tensor_specs(self):
        return [TensorSpec(self.name, (self.buckets + 1, self.hidden), "matrix")]

    def cache_requirement(self):
        return StateRequirement((1,), torch.int32)

    def bind(self, weights, ctx):
        h = weights[self.name]
        shape = (self.buckets + 1, self.hidden)
        require(tuple(h.shape) == shape, f"unexpected tensor shape for {self.name}: got {list(h.shape)}, expected {list(shape)}")
        self.table = torch.empty(shape, dtype=ctx.dtype, device=ctx.device)
        h.copy_into(self.table)

    def forward(self, table, batch, x, cache_view, error_flag, scale: float):
        require(cache_view is not None and tuple(cache_view.requirement.shape) == (1,),
                "an embedding of pairs needs the sequences' last tokens")
        ops.embed_rows_paired(table, self.table, batch, cache_view.storage, x, error_flag, self.mul_prev, self.mul_cur, scale,
                              self.pair_scale)
        return x


register_part("embedding", "hashed_pairs", HashedPairEmbedding)
