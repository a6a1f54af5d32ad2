"""What a part is, and the registries parts are chosen from.

A layer is put together from parts: a *mixer* (mixes information between positions;
attention here), a *feed-forward* (acts on each position alone), *norms*, a *position
encoding* inside the mixer, and a *block* that arranges them around the residual stream.
A configuration names each part by ``kind`` and gives its sizes and constants as
``params``; a part never looks at the model it is in.

Interfaces (all tensors are on the model's device; ``x`` is the float32 residual stream
``[rows, hidden]``; ``h`` is a normed copy in the compute dtype):

* every part: ``__init__(params, prefix)`` (no device work), ``tensor_specs()`` -> the
  checkpoint tensors it needs, ``bind(weights, ctx)`` -> take them from a ``{name: WeightHandle}``
  map onto the device.
* any part may name the kernel sources (``csrc/<name>.cu``) it is going to call, so that a first load compiles them side by
  side: ``kernel_sources``, a tuple, or a function of the compute dtype that gives one.  What is not named is compiled when
  it is first called.
* norm: ``forward(x, row_index=None) -> h`` (``row_index`` int32 picks and orders rows).
* mixer: ``cache_requirement()`` -> KVRequirement | StateRequirement | None;
  ``forward(h, batch, cache_view, residual, write_cache)`` adds its output into ``residual``
  in place.  ``batch`` is a :class:`StepBatch`: the rows of one sequence are consecutive and in
  position order, ``batch.row_slot`` / ``batch.row_pos`` say whose they are and where.
* feed-forward: ``forward(h, batch, residual)`` adds its output into ``residual`` in place.
* position encoding: ``__init__(params, head_dim)``; see :mod:`.rotary`.
* mixer input: what a mixer reads instead of the normed rows; see :mod:`.mixer_input`.
* embedding: what is added to a token's embedding row; see :mod:`.embedding`.
* block: ``__init__(layer_spec)`` builds the parts it knows by name from ``layer_spec.parts``
  (:func:`build_part`); ``parts()``, ``tensor_specs()``, ``cache_requirement()``, ``bind``;
  ``forward(x, batch, cache_view, write_cache)`` updates ``x`` in place.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List, Optional

import torch

from ..errors import require

_REGISTRIES: Dict[str, Dict[str, type]] = {
    "mixer": {}, "feed_forward": {}, "norm": {}, "position": {}, "block": {}, "mixer_input": {}, "embedding": {},
}


def register_part(role: str, kind: str, cls: type, replace: bool = False) -> None:
    require(role in _REGISTRIES, f"unknown part role '{role}'; roles: {', '.join(_REGISTRIES)}")
    require(replace or kind not in _REGISTRIES[role], f"{role} kind '{kind}' is already registered")
    _REGISTRIES[role][kind] = cls


def unregister_part(role: str, kind: str) -> None:
    _REGISTRIES[role].pop(kind, None)


def part_class(role: str, kind: str) -> type:
    require(role in _REGISTRIES, f"unknown part role '{role}'")
    table = _REGISTRIES[role]
    require(kind in table, f"unknown {role} kind '{kind}'; registered: {', '.join(sorted(table)) or '(none)'}")
    return table[kind]


def registered_parts(role: str) -> List[str]:
    return sorted(_REGISTRIES[role])


def build_part(role: str, spec):
    """The part a :class:`PartSpec` describes, from the registry of ``role``."""
    return part_class(role, spec.kind)(spec.params, spec.prefix)


def named_sources(part, dtype) -> tuple:
    """The kernel sources a part (or a block) names, see the module's head."""
    named = getattr(part, "kernel_sources", ())
    return tuple(named(dtype) if callable(named) else named)


@dataclass
class BuildContext:
    """Where and how a model is built: device, compute dtype (bfloat16: the serving kernels and
    precisions; float32: everything in true 32-bit) and the device word kernels raise on a
    fault they detect themselves."""
    device: torch.device
    dtype: torch.dtype
    error_flag: Optional[torch.Tensor] = None

    @property
    def is_float32(self) -> bool:
        return self.dtype == torch.float32


@dataclass
class NormedRows:
    """Rows that stand for ``rms_norm(x)`` without having been normalised: ``rows`` is bfloat16(x), ``sumsq[r, g]``
    the sum of squares of x[r]'s g-th group of 32 features.  A product whose weights carry the norm's gain reads
    ``rows`` and multiplies its result rows by ``rsqrt(sum(sumsq[r]) / dim + eps)``: the same numbers as the product
    of the normalised rows, with the norm's kernel saved."""
    rows: torch.Tensor
    sumsq: torch.Tensor
    dim: int
    eps: float = 0.0

    def with_eps(self, eps: float) -> "NormedRows":
        return NormedRows(self.rows, self.sumsq, self.dim, float(eps))

    @property
    def scale(self):
        return (self.sumsq, self.dim, self.eps)


@dataclass
class StepBatch:
    """One step's rows.  Sequence ``b`` owns rows ``seq_start[b] .. seq_start[b+1]-1``, which are
    its new tokens in order, at positions ``past[b] .. past[b]+n_new[b]-1`` of slot ``slots[b]``."""
    tokens: torch.Tensor          # [rows] int32
    row_slot: torch.Tensor        # [rows] int32
    row_pos: torch.Tensor         # [rows] int32
    seq_start: torch.Tensor       # [sequences + 1] int32
    seq_slot: torch.Tensor        # [sequences] int32
    seq_past: torch.Tensor        # [sequences] int32
    want_rows: torch.Tensor       # [wanted] int32, rows whose logits are asked for
    slots: List[int]
    past: List[int]
    n_new: List[int]
    # A block that ends with a product which emitted what the next norm needs of the residual rows leaves it here
    # (``norm_carry``); the model hands it to the next layer as ``norm_carry_in`` and clears it, so a layer that does
    # not know of it breaks the chain instead of passing on something stale.
    norm_carry: Optional["NormedRows"] = None
    norm_carry_in: Optional["NormedRows"] = None
    # A block on several residual streams may leave its last write-back undone, as (y, mix, out), for the next such
    # block to do together with its first read (one pass over the streams instead of two); the model does what is left
    # after the last layer.
    stream_write: Optional[tuple] = None
    # A block whose last kernel also left the residual rows in the compute dtype hands them to the next block here
    # (``rows_carry`` -> ``rows_carry_in``, moved by the model like ``norm_carry``).
    rows_carry: Optional[torch.Tensor] = None
    rows_carry_in: Optional[torch.Tensor] = None
    # The model tells every block which norm the block that runs next begins with (``next_first_norm``, the part itself;
    # None if that block names none).  A block whose last kernel can run that norm too leaves (normed rows, the norm) as
    # ``normed_carry``; the next block gets it as ``normed_carry_in`` and uses the rows if the norm is its own first one.
    normed_carry: Optional[tuple] = None
    normed_carry_in: Optional[tuple] = None
    next_first_norm: Optional[object] = None
    # For blocks that say ``needs_embedding_output``: the rows as the embedding (and its norm, if the model has one) left
    # them, float32 [rows, hidden], untouched by the layers; and how often the layer that runs now has run before in
    # this step (a layer the schedule names several times: 0, 1, 2, ...).
    embedding_output: Optional[torch.Tensor] = None
    visit: int = 0

    @property
    def rows(self) -> int:
        return int(self.tokens.shape[0])

    @property
    def sequences(self) -> int:
        return len(self.slots)

    @property
    def is_decode(self) -> bool:
        """Every sequence brings exactly one token."""
        return all(n == 1 for n in self.n_new)

    @property
    def max_keys(self) -> int:
        return max(p + n for p, n in zip(self.past, self.n_new))

    @property
    def max_new(self) -> int:
        return max(self.n_new)


def bind_gain(weights, name: str, size: int, ctx: BuildContext) -> torch.Tensor:
    """A norm's gain on the device: float32 on the 32-bit path and when it is stored in 32-bit (a tensor
    stored so stays so), else bfloat16 (a float16 gain is rounded once)."""
    h = weights[name]
    require(tuple(h.shape) == (size,), f"unexpected tensor shape for {name}: got {list(h.shape)}, expected {[size]}")
    dtype = torch.float32 if (ctx.is_float32 or h.dtype == torch.float32) else torch.bfloat16
    return h.tensor.to(device=ctx.device, dtype=dtype).contiguous()


def bind_vector(weights, name: str, size: int, ctx: BuildContext) -> torch.Tensor:
    """A vector that enters 32-bit arithmetic (a bias added to a product's float32 result, a norm's bias, a number per
    head): float32 on the device in both paths, whatever it is stored in."""
    h = weights[name]
    require(tuple(h.shape) == (size,), f"unexpected tensor shape for {name}: got {list(h.shape)}, expected {[size]}")
    return h.tensor.to(device=ctx.device, dtype=torch.float32).contiguous()
