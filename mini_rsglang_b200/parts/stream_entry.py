"""Parts that stand before a run of a layer and act on the whole residual stream.

"rejoin_embedding": x <- W [x ; x0], one product over the stream joined with the embedding's output (W [width, 2 width],
the stream's columns first).  It stands where a group of layers is entered again and again with the same weights: every
pass starts from the stream so far and is shown the embedding anew.  The operand is the float32 stream and embedding
rounded once to the engine's dtype; the result is the product's float32 sums and becomes the stream.

"add_embedding_and_step": x <- x (+ x0) + step[t], t the number of the pass: every pass but the first is shown the embedding
anew, and every pass is told its number by a vector of its own (row t of one table).  Nothing is launched for it: the norm that
opens the layer adds both terms together with the branch before (`StreamEntry.join`)."""
from __future__ import annotations

import torch

from .. import kernels
from ..errors import InvalidRequest
from ..weights.spec import WeightSpec
from .base import STREAM_ENTRIES, BranchSum, StreamEntry
from .linear import linear


@STREAM_ENTRIES.register("rejoin_embedding")
class RejoinEmbedding(StreamEntry):
    def __init__(self, prefix: str, width: int, leaf: str = "weight"):
        super().__init__(prefix)
        self.width, self.leaf = int(width), leaf
        self.weight = None

    def weight_specs(self):
        return [WeightSpec(self.name(self.leaf), (self.width, 2 * self.width))]

    def bind(self, tensors, runtime):
        super().bind(tensors, runtime)
        self.weight = tensors[self.name(self.leaf)].contiguous()

    def forward(self, stream, origin, ctx):
        joined = torch.empty((stream.shape[0], 2 * self.width), dtype=self.runtime.dtype, device=stream.device)
        kernels.concat_rows(stream, origin, joined)
        return linear(joined, self.weight, out_dtype=torch.float32)


@STREAM_ENTRIES.register("add_embedding_and_step")
class AddEmbeddingAndStep(StreamEntry):
    adds_only = True

    def __init__(self, prefix: str, width: int, times: int, number: int, with_embedding: bool, leaf: str = "weight"):
        """Pass `number` of `times`; the table [times, width] is one tensor that the entries of all passes name."""
        super().__init__(prefix)
        self.width, self.times, self.number, self.leaf = int(width), int(times), int(number), leaf
        if not 0 <= self.number < self.times:
            raise InvalidRequest(f"{prefix}: pass {number} of {times}")
        self.reads_origin = bool(with_embedding)
        self.step = None

    def weight_specs(self):
        # one table for all passes: the first pass asks for it
        return [WeightSpec(self.name(self.leaf), (self.times, self.width), "bias")] if self.number == 0 else []

    def bind(self, tensors, runtime):
        super().bind(tensors, runtime)
        self.step = tensors[self.name(self.leaf)].float()[self.number].contiguous()

    def join(self, pending, origin):
        terms = list(pending.terms) if isinstance(pending, BranchSum) else ([(pending, 1.0)] if pending is not None else [])
        row = self.step
        if isinstance(pending, BranchSum) and pending.row is not None:
            row = row + pending.row
        return BranchSum(terms + ([(origin, 1.0)] if self.reads_origin else []), row)

    def forward(self, stream, origin, ctx):
        return self.join(None, origin).add_to(stream)
