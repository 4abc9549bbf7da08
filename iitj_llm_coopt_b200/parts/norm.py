"""Norms over the float32 residual stream: RMSNorm and its gains, and a norm without statistics.

y = x * rsqrt(mean(x^2) + eps) * weight  (engine/model.py:85-89), statistics in float32.
The reference's fused form `residual += x; x = norm(residual)` (engine/model.py:236, 249, 254)
is the `delta` argument here.  An option `branch_factor` of an RMSNorm's spec multiplies the delta on its way into the residual,
residual += branch_factor * delta; the delta may then also be a routed feed-forward whose weighted sum is still to be taken.
"""
from __future__ import annotations

from .base import ParamSpec, Part


class RMSNorm(Part):
    graph_safe = True
    takes_partial_sums = True     # `delta` may be the k-split parts of a matrix product: added while they are read

    def __init__(self, spec, kernels, dtype):
        self.spec, self.k, self.dtype = spec, kernels, dtype
        self.width, self.eps = spec.width, spec.eps
        self.factor = dict(spec.options).get("branch_factor")
        self.takes_routed_sums = self.factor is not None
        self.weight = None

    @classmethod
    def parameters(cls, spec) -> dict:
        return {"weight": ParamSpec((spec.width,), kind="vector")}

    def load(self, tensors: dict) -> None:
        self.weight = tensors["weight"] if self.factor is None else tensors["weight"].float().contiguous()

    def forward(self, ctx, residual, delta=None, rows=None):
        n = rows.shape[0] if rows is not None else residual.shape[0]
        out = ctx.buffer(f"norm.{self.part_name}.out" if rows is None else f"norm.{self.part_name}.rows", (n, self.width), self.dtype)
        if self.factor is not None and delta is not None:
            return self.k.add_branch_rmsnorm(residual, delta, float(self.factor), self.weight, self.eps, out, rows=rows)
        return self.k.add_rmsnorm(residual, delta, self.weight, self.eps, out, rows=rows)


class DynamicTanh(Part):
    """y = tanh(alpha * x) * weight + bias, number by number, alpha one number: no mean and no variance is taken.  The spec's
    option `branch_factor` (1) multiplies the delta on its way into the residual: residual += branch_factor * delta.  A delta may be
    the k-split parts of a product, or a routed feed-forward whose weighted sum is still to be taken: the kernel adds either as it
    reads, so a sub-layer's last sum, the residual sum and the norm of the next sub-layer are one kernel."""
    graph_safe = True
    takes_partial_sums = True
    takes_routed_sums = True

    def __init__(self, spec, kernels, dtype):
        self.spec, self.k, self.dtype, self.width = spec, kernels, dtype, spec.width
        self.factor = float(dict(spec.options).get("branch_factor", 1.0))
        self.weight = self.bias = self.alpha = None

    @classmethod
    def parameters(cls, spec) -> dict:
        return {"weight": ParamSpec((spec.width,), kind="vector"), "bias": ParamSpec((spec.width,), kind="vector"),
                "alpha": ParamSpec((), kind="vector")}

    def load(self, tensors: dict) -> None:
        self.weight, self.bias = tensors["weight"].float().contiguous(), tensors["bias"].float().contiguous()
        self.alpha = tensors["alpha"].float().reshape(1).contiguous()

    def forward(self, ctx, residual, delta=None, rows=None):
        n = rows.shape[0] if rows is not None else residual.shape[0]
        out = ctx.buffer(f"norm.{self.part_name}.out" if rows is None else f"norm.{self.part_name}.rows", (n, self.width), self.dtype)
        return self.k.add_dynamic_tanh(residual, delta, self.factor, (self.alpha, self.weight, self.bias), out, rows=rows)


class ScalarGainRMSNorm(RMSNorm):
    """RMSNorm whose gain is one number for the whole width: y = x * rsqrt(mean(x^2) + eps) * g.  The
    checkpoint holds g as a tensor without dimensions; it is spread over the width once, at loading, so the
    kernel of `RMSNorm` serves both."""

    @classmethod
    def parameters(cls, spec) -> dict:
        return {"weight": ParamSpec((), kind="vector")}

    def load(self, tensors: dict) -> None:
        self.weight = tensors["weight"].float().reshape(1).expand(self.width).contiguous()


class OnePlusRMSNorm(RMSNorm):
    """RMSNorm whose gain is stored around zero: y = x * rsqrt(mean(x^2) + eps) * (1 + w).  One is added once, at loading, in
    float32, so the kernels of `RMSNorm` serve it."""

    def load(self, tensors: dict) -> None:
        self.weight = (tensors["weight"].float() + 1.0).contiguous()
