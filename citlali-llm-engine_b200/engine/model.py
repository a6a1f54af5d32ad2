"""A decoder built from a ModelSpec: embedding, the schedule of layers, final norm, head.

The forward pass follows QwenModel::forward_token (src/model/qwen_model.cpp:239-419) for a
batch of rows instead of one token: embedding rows, each scheduled layer on all rows, and
only for the rows whose logits are wanted the final norm and the output matrix (the
reference skips both for prompt tokens that are not the last, :378-380).  Which layers
exist, what they are made of, and in which order they run is the spec's data.
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from .. import ops
from ..config.spec import ModelSpec
from ..errors import require
from ..parts.base import BuildContext, StepBatch, build_part, named_sources, part_class
from ..parts.linear import DenseLinear
from ..weights.loader import TensorSpec, WeightHandle


def _numel(shape) -> int:
    n = 1
    for d in shape:
        n *= int(d)
    return n


def _build_layers(spec: ModelSpec):
    return [part_class("block", l.block)(l) for l in spec.layers]


def expected_tensors(spec: ModelSpec) -> List[TensorSpec]:
    """Every checkpoint tensor the model reads, in a fixed order.  No device is touched."""
    specs = [TensorSpec(spec.embedding_name, (spec.vocab_size, spec.hidden_size), "matrix")]
    if spec.embedding_addition is not None:
        specs.extend(build_part("embedding", spec.embedding_addition).tensor_specs())
    if spec.embedding_norm is not None:
        specs.extend(build_part("norm", spec.embedding_norm).tensor_specs())
    for block in _build_layers(spec):
        specs.extend(block.tensor_specs())
    specs.extend(build_part("norm", spec.final_norm).tensor_specs())
    # tied: the head is the embedding and a stored head is ignored; undecided: used if present
    specs.append(TensorSpec(spec.head_name, (spec.vocab_size, spec.hidden_size), "matrix",
                            optional=spec.tie_head_to_embedding is not False))
    seen = set()
    for s in specs:
        require(s.name not in seen, f"two parts of the model claim the tensor '{s.name}'")
        seen.add(s.name)
    return specs


def cache_requirements_of(spec: ModelSpec, layers=None) -> List[object]:
    """Per schedule step: what it keeps (a KVRequirement, a StateRequirement, or None for a step that keeps
    nothing or reads another step's cache).  An addition to the embedding's rows has one more entry behind the schedule's.
    No device is touched."""
    layers = layers if layers is not None else _build_layers(spec)
    out = [None if step.cache_of is not None else layers[step.layer].cache_requirement() for step in spec.schedule]
    if spec.embedding_addition is not None:
        out.append(build_part("embedding", spec.embedding_addition).cache_requirement())
    return out


class DecoderModel:
    def __init__(self, spec: ModelSpec, ctx: BuildContext):
        spec.validate()
        self.spec = spec
        self.ctx = ctx
        self.layers = _build_layers(spec)
        self.final_norm = build_part("norm", spec.final_norm)
        self.embedding_norm = build_part("norm", spec.embedding_norm) if spec.embedding_norm is not None else None
        self.embedding_addition = build_part("embedding", spec.embedding_addition) if spec.embedding_addition is not None else None
        require(spec.residual_streams is None or self.embedding_addition is None,
                "an addition to the embedding's rows works on one residual stream")
        self.keeps_embedding_output = any(getattr(block, "needs_embedding_output", False) for block in self.layers)
        require(spec.residual_streams is None or (self.embedding_norm is None and not self.keeps_embedding_output),
                "a norm on the embedding's rows and blocks that read them again work on one residual stream")
        seen: Dict[int, int] = {}
        self.visits = []                       # per schedule step: how often its layer has run before it
        for step in spec.schedule:
            self.visits.append(seen.get(step.layer, 0))
            seen[step.layer] = self.visits[-1] + 1
        self.head = DenseLinear([spec.head_name], [spec.vocab_size], spec.hidden_size)
        self.embedding: Optional[torch.Tensor] = None
        self.tied = None
        streams = spec.residual_streams
        for i, block in enumerate(self.layers):
            takes = getattr(block, "residual_streams", None)
            require(takes == streams, f"layer {i}'s block works on {takes or 'one'} residual stream(s), the model has "
                                      f"{streams or 'one'}")

    def tensor_specs(self) -> List[TensorSpec]:
        return expected_tensors(self.spec)

    def cache_requirements(self) -> List[object]:
        return cache_requirements_of(self.spec, self.layers)

    def bind(self, weights: Dict[str, WeightHandle]) -> None:
        ctx, spec = self.ctx, self.spec
        emb = weights[spec.embedding_name]
        require(tuple(emb.shape) == (spec.vocab_size, spec.hidden_size),
                f"unexpected tensor shape for {spec.embedding_name}: got {list(emb.shape)}, "
                f"expected {[spec.vocab_size, spec.hidden_size]}")
        self.embedding = torch.empty((spec.vocab_size, spec.hidden_size), dtype=ctx.dtype, device=ctx.device)
        emb.copy_into(self.embedding)
        for block in self.layers:
            block.bind(weights, ctx)
        self.final_norm.bind(weights, ctx)
        if self.embedding_norm is not None:
            self.embedding_norm.bind(weights, ctx)
        if self.embedding_addition is not None:
            self.embedding_addition.bind(weights, ctx)
        tie = spec.tie_head_to_embedding
        if tie is None:
            tie = spec.head_name not in weights      # absent head: reuse the embedding (qwen_model.cpp:71-75)
        self.tied = bool(tie)
        if self.tied:
            self.head.bind_shared(self.embedding, ctx)
        else:
            require(spec.head_name in weights, f"missing required tensor: {spec.head_name}")
            self.head.bind(weights, ctx)

    def kernel_sources(self) -> List[str]:
        """The kernel sources the model's steps call, as far as its parts name them (``csrc/<name>.cu``)."""
        dtype = self.ctx.dtype
        out = {"elementwise", "gemm_simt" if dtype == torch.float32 else "gemm_tcgen05"}
        if self.spec.residual_streams is not None:
            out.add("hyper_connection")
        for owner in [self.final_norm, self.embedding_norm, self.embedding_addition] + [p for b in self.layers for p in [b] + list(b.parts())]:
            if owner is not None:
                out.update(named_sources(owner, dtype))
        return sorted(out)

    def weight_bytes_read_per_step(self) -> int:
        """Bytes of weights one step reads when each matrix it uses is read once: every tensor the layers
        declare as a matrix (``tensor_specs()``, so lists of matrices inside a part count too), once per
        schedule step that runs the layer, plus the output matrix.  The embedding's rows and the norm
        gains are left out: they are thousands of times smaller."""
        size = torch.tensor([], dtype=self.ctx.dtype).element_size()
        per_layer = [sum(_numel(t.shape) for t in block.tensor_specs() if t.role == "matrix") * size
                     for block in self.layers]
        return self.head.nbytes + sum(per_layer[step.layer] for step in self.spec.schedule)

    def forward(self, batch: StepBatch, cache) -> torch.Tensor:
        """Logits ``[wanted, vocab]`` float32 for ``batch.want_rows``, in that order."""
        ctx, spec = self.ctx, self.spec
        streams = spec.residual_streams
        emb_scale = 1.0 if spec.embedding_scale is None else float(spec.embedding_scale)
        if streams is None:
            x = torch.empty((batch.rows, spec.hidden_size), dtype=torch.float32, device=ctx.device)
            if self.embedding_addition is not None:
                at = len(spec.schedule)
                self.embedding_addition.forward(self.embedding, batch, x, cache.view(at) if cache.has_view(at) else None,
                                                ctx.error_flag, emb_scale)
            else:
                ops.embed_rows(self.embedding, batch.tokens, x, ctx.error_flag, emb_scale)
            if self.embedding_norm is not None:
                x = self.embedding_norm.forward(x, out_dtype=torch.float32)
            # blocks that read the embedding's rows again get them apart from the residual, which the layers change in place
            batch.embedding_output = x.clone() if self.keeps_embedding_output else None
        else:                       # every stream starts as the embedding's rows
            x = torch.empty((streams, batch.rows, spec.hidden_size), dtype=torch.float32, device=ctx.device)
            ops.embed_rows_streams(self.embedding, batch.tokens, x, ctx.error_flag, emb_scale)
        batch.norm_carry = None
        batch.rows_carry = None
        batch.normed_carry = None
        batch.stream_write = None
        first_norms = [getattr(block, "first_norm", lambda: None)() for block in self.layers]
        for i, step in enumerate(spec.schedule):
            source = i if step.cache_of is None else step.cache_of
            view = cache.view(source) if cache.has_view(source) else None
            # what the layer before left for this layer's first norm, if it left anything (parts/block.py)
            batch.norm_carry_in, batch.norm_carry = batch.norm_carry, None
            batch.rows_carry_in, batch.rows_carry = batch.rows_carry, None
            batch.normed_carry_in, batch.normed_carry = batch.normed_carry, None
            batch.next_first_norm = first_norms[spec.schedule[i + 1].layer] if i + 1 < len(spec.schedule) else None
            batch.visit = self.visits[i]
            if batch.stream_write is not None and not getattr(self.layers[step.layer], "takes_stream_write", False):
                ops.hyper_write(x, *batch.stream_write)      # the block ahead left a write-back that this one would not do
                batch.stream_write = None
            self.layers[step.layer].forward(x, batch, view, write_cache=step.cache_of is None)
        batch.norm_carry_in = batch.norm_carry = None
        batch.rows_carry_in = batch.rows_carry = None
        batch.normed_carry_in = batch.normed_carry = batch.next_first_norm = None
        batch.embedding_output = None
        if batch.stream_write is not None:              # the last layer's last write-back into the streams
            ops.hyper_write(x, *batch.stream_write)
            batch.stream_write = None
        wanted = int(batch.want_rows.numel())
        if wanted == 0:
            return torch.empty((0, spec.vocab_size), dtype=torch.float32, device=ctx.device)
        if streams is None:
            h = self.final_norm.forward(x, row_index=batch.want_rows)
        else:
            summed = torch.empty((wanted, spec.hidden_size), dtype=torch.float32, device=ctx.device)
            ops.stream_sum(x, summed, batch.want_rows)
            h = self.final_norm.forward(summed)
        logits = self.head.forward(h, out_dtype=torch.float32)
        if spec.logit_scale is not None:
            ops.scale_(logits, float(spec.logit_scale))
        if spec.logit_softcap is not None:
            ops.soft_cap_(logits, float(spec.logit_softcap))
        return logits
