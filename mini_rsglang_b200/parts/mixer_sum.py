"""Several mixers side by side on one input: y = sum of factor_j * mixer_j(h), each with tensors of its own below a name.

The layer's one cache entry serves all of them: at most one keeps keys and values in pages, at most one keeps a state in the
request's slot.  Where every mixer allows it (`Mixer.projection`), one product over the row-concatenated matrices reads h for
all; each goes on from its columns.  The factors multiply the mixers' float32 outputs; a block that adds several branches to the
stream at once takes the terms as they are (`gives_terms`)."""
from __future__ import annotations

import torch

from .. import kernels
from ..errors import InvalidRequest
from .base import MIXERS, BranchSum, Mixer, PartSpec
from .linear import linear


@MIXERS.register("mixer_sum")
class MixerSum(Mixer):
    gives_terms = True

    def __init__(self, prefix: str, width: int, branches: list[tuple[str, PartSpec, float]]):
        """`branches`: (name below the part's root, mixer, factor) of every mixer; a mixer with pages comes first."""
        super().__init__(prefix)
        self.width = int(width)
        self.mixers = [MIXERS.build(spec, self.name(name)) for name, spec, _ in branches]
        self.factors = [float(factor) for _, _, factor in branches]
        if not self.mixers:
            raise InvalidRequest(f"{prefix}: a sum of mixers needs at least one")
        for what in ("cache_need", "state_need"):
            if sum(getattr(m, what)() is not None for m in self.mixers) > 1:
                raise InvalidRequest(f"{prefix}: at most one mixer with pages and one with a state share a layer")
        self.replayable = all(m.replayable for m in self.mixers)
        self.fused, self.offsets = None, []

    def weight_specs(self):
        return [spec for m in self.mixers for spec in m.weight_specs()]

    def cache_need(self):
        return next((need for need in (m.cache_need() for m in self.mixers) if need is not None), None)

    def state_need(self):
        return next((need for need in (m.state_need() for m in self.mixers) if need is not None), None)

    def step_signature(self, facts):
        signatures = tuple(m.step_signature(facts) for m in self.mixers)
        return signatures if any(s is not None for s in signatures) else None

    def bind(self, tensors, runtime):
        super().bind(tensors, runtime)
        for m in self.mixers:
            m.bind(tensors, runtime)
        rows = [m.projection() for m in self.mixers]
        if len(rows) < 2 or any(r is None for r in rows):
            return
        self.offsets, at, padded = [], 0, []
        for r in rows:                                       # every mixer's columns begin on a 16-byte boundary
            self.offsets.append(at)
            padding = -r.shape[0] % 8
            padded += [r] + ([r.new_zeros((padding, self.width))] if padding else [])
            at += r.shape[0] + padding
        self.fused = torch.cat(padded, dim=0).contiguous()
        for m in self.mixers:                                # the product reads the joined rows; the mixers' own copies go
            m.fused = None

    def forward(self, h, ctx, cache, write_cache=True, as_terms=False):
        if self.fused is not None:
            proj = linear(h, self.fused, out_dtype=torch.float32)
            outs = [m.forward_projected(proj, at, ctx, cache, write_cache) for m, at in zip(self.mixers, self.offsets)]
        else:
            outs = [m.forward(h, ctx, cache, write_cache) for m in self.mixers]
        terms = [(o if o.dtype is torch.float32 else o.float(), factor) for o, factor in zip(outs, self.factors)]
        if as_terms:
            return BranchSum(terms)
        total = torch.zeros_like(terms[0][0])
        for at in range(0, len(terms), kernels.MAX_BRANCHES):
            kernels.add_scaled_branches_norms(total, terms[at:at + kernels.MAX_BRANCHES], [], 0.0)
        return total
