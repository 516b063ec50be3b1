"""Layer norm with a weight and, optionally, a bias.

``y_c = (x_c - mean) / sqrt(mean((x - mean)^2) + eps) * w_c + b_c`` over the fp32 residual stream, mean,
deviations and their square in fp32.  ``bias_name`` (``None``: no bias) names the bias tensor.  This norm is
not folded into the products around it: the product before it would have to leave ``bf16(x * w)`` of a
row whose mean is still inside, and the mean taken off after the next product's sums; where the mean is large
beside the deviations that loses bits that the norm as a kernel keeps.
"""
from __future__ import annotations

from ..registry import NORMS
from .base import Norm, WeightSpec


@NORMS.register("layer_norm")
class LayerNorm(Norm):
    def __init__(self, params, rt):
        super().__init__(params, rt)
        self.size = int(params["size"])
        self.eps = float(params["eps"])
        self.name = params.get("name", "weight")
        self.bias_name = params.get("bias_name")
        self.weight = self.bias = None

    def weight_specs(self):
        specs = [WeightSpec(self.name, (self.size,), role="norm", std=0.1)]
        if self.bias_name:
            specs.append(WeightSpec(self.bias_name, (self.size,), role="vector", std=0.1))
        return specs

    def load(self, tensors):
        self.weight = tensors[self.name]
        self.bias = tensors[self.bias_name] if self.bias_name else None
        if self.bias is not None and self.bias.dtype != self.weight.dtype:      # one of them stored in 32 bits
            self.weight, self.bias = self.weight.float().contiguous(), self.bias.float().contiguous()

    def forward(self, ctx, hidden, rows=None, out_name="normed", dtype=None):
        """``dtype``: of the result (default: the run dtype; fp32 for a consumer that goes on in fp32)."""
        n = hidden.shape[0] if rows is None else rows.shape[0]
        out = self.rt.buffer(out_name, n, self.size, dtype or self.rt.dtype)
        self.rt.ops.layer_norm(hidden, self.weight, self.bias, out, self.eps, rows)
        return out
