"""RMSNorm: y = x * 1/sqrt(mean(x^2) + eps) * w, sum and scale in float32
(src/model.zig:1166-1181; plain weight, no 1 + w); and the layer norm with weight and bias that other designs use."""
from __future__ import annotations

from typing import Optional

import torch

from .. import kernels
from .base import NORMS, Norm, WeightSpec
from .linear import NormedRows, ResidualSink


class RMSNorm(Norm):
    """`one_plus`: the weight is stored around zero and 1 + w multiplies (the kernels are handed 1 + w, made at load)."""

    def __init__(self, dim: int, eps: float, weight_name: str, one_plus: bool = False):
        self.dim, self.eps, self.weight_name, self.one_plus = dim, float(eps), weight_name, bool(one_plus)
        self.weight: Optional[torch.Tensor] = None

    def weight_specs(self):
        return [WeightSpec(self.weight_name, (self.dim,), role="vector", init="normal" if self.one_plus else "norm")]

    def load(self, weights, dtype, device):
        w = weights[self.weight_name]
        self.weight = w + 1.0 if self.one_plus else w

    def forward(self, ctx, x, rows=None):
        return kernels.rmsnorm(x, self.weight, self.eps, ctx.dtype, rows)

    def add_normed(self, ctx, m, x):
        """x += norm(m), row by row in float32: the form a block needs that normalises what a sublayer
        RETURNS instead of what it reads."""
        return kernels.rmsnorm_add(m, self.weight, self.eps, x)

    def pending(self, ctx, x, prepared=None):
        """All rows, not yet normalised: `linear` and the fused kernels resolve a `NormedRows`.
        `prepared` is what `ahead` returned for these rows, after the contraction that got it ran."""
        emit = None
        if (isinstance(prepared, ResidualSink) and prepared.emit is not None and prepared.rows is x
                and prepared.norm_weight is self.weight):
            emit = prepared.emit
        return NormedRows(x, self.weight, self.eps, ctx.dtype, scaled=emit)

    def ahead(self, ctx, x):
        """For the few rows of a single-token step in bfloat16: the contraction that sums into `x`
        can write this norm's inputs along (see `linear`)."""
        if ctx.dtype != torch.bfloat16 or x.shape[0] > kernels.GEMM_TC_SWAPPED_MAX_M:
            return None
        return ResidualSink(x, self.weight)


class LayerNorm(Norm):
    """y = (x - mean) / sqrt(var + eps) * w + b over a row, var the mean of the squared deviations; sums and scale in
    float32.  `bias_name` None: no bias.  It has no pending form: every consumer gets the normalised tensor."""

    def __init__(self, dim: int, eps: float, weight_name: str, bias_name: Optional[str] = None):
        self.dim, self.eps, self.weight_name, self.bias_name = dim, float(eps), weight_name, bias_name
        self.weight: Optional[torch.Tensor] = None
        self.bias: Optional[torch.Tensor] = None

    def weight_specs(self):
        specs = [WeightSpec(self.weight_name, (self.dim,), role="vector", init="norm")]
        if self.bias_name is not None:
            specs.append(WeightSpec(self.bias_name, (self.dim,), role="vector"))
        return specs

    def load(self, weights, dtype, device):
        self.weight = weights[self.weight_name]
        self.bias = weights[self.bias_name] if self.bias_name is not None else None

    def forward(self, ctx, x, rows=None):
        return kernels.layernorm(x, self.weight, self.bias, self.eps, ctx.dtype, rows)


NORMS.register("rmsnorm", RMSNorm)
NORMS.register("layernorm", LayerNorm)
