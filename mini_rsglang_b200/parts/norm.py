"""RMSNorm: y = x * rsqrt(mean(x^2) + eps) * weight, statistics in float32
(reference: crates/kernels/src/ops.cu:66-78).  The weight multiplies plainly unless the checkpoint stores it as its
distance from one (`weight_offset`): it is then held as offset + w in float32.
LayerNorm: y = (x - mean) / sqrt(var + eps) * weight + bias, var the mean of the squared deviations."""
from __future__ import annotations

import torch

from .. import kernels
from ..errors import InvalidRequest
from ..weights.spec import WeightSpec
from .base import NORMS, BranchSum, Norm, Normed, Prenormed


def _settle(residual: torch.Tensor, delta: BranchSum, write_back: bool) -> torch.Tensor:
    """The stream with the sum's terms added (in place when `write_back`), for norms whose own kernel adds one branch."""
    residual = residual if write_back else residual.clone()
    terms = [(x if x.dtype is torch.float32 else x.float(), factor) for x, factor in delta.terms]
    for at in range(0, len(terms), kernels.MAX_BRANCHES):
        kernels.add_scaled_branches_norms(residual, terms[at:at + kernels.MAX_BRANCHES], [], 0.0)
    if delta.row is not None:
        residual.add_(delta.row)
    return residual


@NORMS.register("rmsnorm")
class RMSNorm(Norm):
    rides_on_products = True

    def __init__(self, prefix: str, width: int, eps: float, leaf: str = "weight", weight_offset: float = 0.0):
        super().__init__(prefix)
        self.width, self.eps = int(width), float(eps)
        self.weight_offset = float(weight_offset)
        self.leaf = leaf                   # the weights' name below the part's root ("": the root itself)
        self.weight: torch.Tensor | None = None

    def weight_specs(self):
        return [WeightSpec(self.name(self.leaf), (self.width,), "offset_vector" if self.weight_offset else "vector")]

    def bind(self, tensors, runtime):
        super().bind(tensors, runtime)
        self.weight = tensors[self.name(self.leaf)]
        if self.weight_offset:
            self.weight = (self.weight + self.weight_offset).contiguous()

    def forward(self, x):
        out = torch.empty_like(x)
        kernels.rmsnorm(x, self.weight, self.eps, out)
        return out

    def add_norm(self, residual, delta, rows=None, write_back=True):
        if isinstance(delta, Prenormed):          # the stream holds the sum already
            if delta.norm is self and rows is None:
                return delta                      # and the product after this norm finishes it
            delta = None
        if isinstance(delta, Normed):             # the stream holds the sum, and this norm of it may be there already
            if delta.norm is self and rows is None:
                return delta.rows
            delta = None
        if isinstance(delta, BranchSum):
            residual = _settle(residual, delta, write_back)
            delta = None
        n = residual.shape[0] if rows is None else rows.shape[0]
        out = torch.empty((n, self.width), dtype=self.runtime.dtype, device=residual.device)
        kernels.add_rmsnorm(residual, delta, self.weight, self.eps, out, rows, write_back)
        return out


class NormPair(Norm):
    """Two RMS norms of one stream, read side by side: `add_norm` returns the rows of both.  They share their statistic, so
    one kernel makes both (and adds the branches that came before); it is what a block with two entry norms hands to the
    block before it as the norm that follows."""

    def __init__(self, first: RMSNorm, second: RMSNorm):
        super().__init__(first.prefix)
        if not first.rides_on_products or not second.rides_on_products or (first.width, first.eps) != (second.width, second.eps):
            raise InvalidRequest(f"norms at {first.prefix!r} and {second.prefix!r}: a pair is two RMS norms of one width and epsilon")
        self.first, self.second = first, second
        self.width, self.eps = first.width, first.eps

    def outputs(self, stream, dtype) -> list:
        """[(weight, rows to fill)] of both norms."""
        return [(norm.weight, torch.empty(stream.shape, dtype=dtype, device=stream.device)) for norm in (self.first, self.second)]

    def add_norm(self, residual, delta, rows=None, write_back=True):
        if isinstance(delta, Normed) and delta.norm is self:
            return delta.rows
        if isinstance(delta, (Prenormed, Normed)):       # the stream holds the sum already
            delta = None
        if rows is not None or not write_back:
            raise InvalidRequest("a pair of norms reads whole streams")
        outs = self.outputs(residual, self.first.runtime.dtype)
        if isinstance(delta, BranchSum):
            residual, delta = _settle(residual, delta, True), None
        kernels.add_scaled_branches_norms(residual, [(delta.float(), 1.0)] if delta is not None else [], outs, self.eps)
        return tuple(out for _, out in outs)


@NORMS.register("layernorm")
class LayerNorm(Norm):
    """Layer norm with weight and bias, statistics in float32.  `leaf` and `bias_leaf` name the two tensors below the
    part's root ("": the root itself)."""

    def __init__(self, prefix: str, width: int, eps: float, leaf: str = "weight", bias_leaf: str = "bias"):
        super().__init__(prefix)
        self.width, self.eps = int(width), float(eps)
        self.leaf, self.bias_leaf = leaf, bias_leaf
        self.weight: torch.Tensor | None = None
        self.bias: torch.Tensor | None = None

    def weight_specs(self):
        return [WeightSpec(self.name(self.leaf), (self.width,), "vector"), WeightSpec(self.name(self.bias_leaf), (self.width,), "bias")]

    def bind(self, tensors, runtime):
        super().bind(tensors, runtime)
        self.weight, self.bias = tensors[self.name(self.leaf)], tensors[self.name(self.bias_leaf)]

    def forward(self, x):
        """Rows of the engine's dtype, normed (no residual)."""
        out = torch.empty_like(x)
        kernels.add_layernorm(x.float(), None, self.weight, self.bias, self.eps, out)
        return out

    def add_norm(self, residual, delta, rows=None, write_back=True):
        if isinstance(delta, (Prenormed, Normed)):       # the stream holds the sum already
            delta = None
        factor, extra, row = 1.0, None, None
        if isinstance(delta, BranchSum):
            # the kernel adds a branch times a factor, a second branch as it is and a vector; anything beyond is added before
            terms, row = list(delta.terms), delta.row
            plain_one = next((i for i in reversed(range(len(terms))) if terms[i][1] == 1.0 and terms[i][0].dtype is torch.float32), None)
            if len(terms) > 1 and plain_one is not None:
                extra = terms.pop(plain_one)[0]
            if len(terms) > 1:
                residual = _settle(residual, BranchSum(terms[1:]), write_back)
            delta, factor = terms[0] if terms else (None, 1.0)
        n = residual.shape[0] if rows is None else rows.shape[0]
        out = torch.empty((n, self.width), dtype=self.runtime.dtype, device=residual.device)
        kernels.add_layernorm(residual, delta, self.weight, self.bias, self.eps, out, rows, write_back, factor=factor, extra=extra, row=row)
        return out
