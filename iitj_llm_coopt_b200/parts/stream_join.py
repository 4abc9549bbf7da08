"""`StreamJoin`: what the stream becomes where a run of layers starts over.

    x <- [x; x0] W^T           x0 the embedding's output of the same tokens, x first

x and x0 lie side by side as the engine's type in one matrix [T, 2 * width]: the x0 half is written once a step (by the embedding's
own kernel where it knows how: it finds the half under `ORIGIN` in `ctx.shared`; else by `keep`), the x half before every pass by the
kernel that adds the pending branch (times the spec's option `branch_factor`) to the stream.  The product writes the new float32
stream in place of the old one.
"""
from __future__ import annotations

from .base import ParamSpec, Part

ORIGIN = "stream_join.origin"      # ctx.shared: where the embedding may leave its rows as the engine's type


class StreamJoin(Part):
    graph_safe = True
    takes_partial_sums = True
    takes_routed_sums = True

    def __init__(self, spec, kernels, dtype):
        self.spec, self.k, self.dtype, self.width = spec, kernels, dtype, spec.width
        self.factor = float(dict(spec.options).get("branch_factor", 1.0))
        self.weight = None

    @classmethod
    def parameters(cls, spec) -> dict:
        return {"weight": ParamSpec((spec.width, 2 * spec.width))}

    def _rows(self, ctx):
        return ctx.buffer("stream_join.rows", (ctx.num_tokens, 2 * self.width), self.dtype)

    def origin(self, ctx):
        """The place of x0 in this step's joined rows."""
        return self._rows(ctx)[:, self.width:]

    def keep(self, ctx, residual) -> None:
        """Copies the embedding's output there, for an embedding that did not."""
        self.k.add_dynamic_tanh(residual, None, 1.0, None, self.origin(ctx))

    def forward(self, ctx, residual, delta=None):
        rows = self._rows(ctx)
        self.k.add_dynamic_tanh(residual, delta, self.factor, None, rows[:, :self.width], store=False)
        return self.k.linear(rows, self.weight, residual)
