"""`GatedDelta`: a recurrent mixer with a matrix state per head that is corrected towards each token's value (a gated delta rule) behind
short causal convolutions.

    [q, k, v, z] = x W^T                       (one product, no biases; q, k kv_heads x head_dim, v, z heads x value_dim)
    q, k, v = silu(sum_j taps[:, j] * u_(t - n + 1 + j))      per channel of the projection u, n = `conv_taps`, the last tap the current
                                                             token's, zeros before the first
    q, k divided by sqrt(sum of squares + unit_tiny) per head;   q scaled by head_dim^(-1/2)
    beta = sigmoid(x Wb^T),   g = exp(-exp(A_log) * softplus(x Wa^T + dt_bias))          one number per head each
    S <- g S;   S <- S + k (beta (v - S^T k))^T;   o = S^T q          head h uses q and k of head h // (heads / kv_heads)
    out = (each head of o divided by its root mean square * gain [value_dim] * silu(z)) Wo^T

The state is one cache entry (kind "state"): a record of `record(...)` float32 numbers per request: per head the columns of S (each
padded to a multiple of four numbers), then `conv_taps` rows of the projection's q, k and v channels; the row of position p is row
p % conv_taps, so a decoded token writes a row that no convolution of the step reads.  The cache manager clears the record when it
admits a request, so a portion of a prompt simply continues from what the slot holds.  Everything behind the convolutions is float32.
"""
from __future__ import annotations

import torch

from ..config.specs import CacheNeed
from .base import ParamSpec, Part
from .matrix_memory import padded
from .state_plan import KEY, plan_state_chunks


def record(heads: int, kv_heads: int, dim: int, vdim: int, taps: int) -> int:
    return padded(heads * vdim * padded(dim) + taps * (2 * kv_heads * dim + heads * vdim))


class GatedDelta(Part):
    graph_safe = True
    prepare_key = KEY

    def __init__(self, spec, kernels, dtype, position=None):
        self.spec, self.k, self.dtype = spec, kernels, dtype
        self.width, self.heads, self.kv_heads = spec.width, spec.heads, spec.kv_heads
        self.head_dim, self.value_dim = spec.head_dim, spec.value_dim or spec.head_dim
        if self.heads % self.kv_heads:
            raise ValueError(f"gated delta: heads {self.heads} is not a multiple of kv_heads {self.kv_heads}")
        self.eps, self.tiny = float(spec.option("eps", 1e-6)), float(spec.option("unit_tiny", 1e-6))
        self.cols = 2 * self.kv_heads * self.head_dim + 2 * self.heads * self.value_dim
        self.qkvg = self.conv = self.gates = self.A_log = self.dt_bias = self.norm = self.o = self.rate = None

    @classmethod
    def parameters(cls, spec) -> dict:
        h, qk, v = spec.heads, spec.kv_heads * spec.head_dim, spec.heads * (spec.value_dim or spec.head_dim)
        rows = (("q", qk), ("k", qk), ("v", v))
        return {"qkvg": ParamSpec((2 * qk + 2 * v, spec.width), pieces=rows + (("g", v),)),
                "conv": ParamSpec((2 * qk + v, int(spec.option("conv_taps"))), kind="vector", pieces=rows),
                "gates": ParamSpec((2 * h, spec.width), pieces=(("b", h), ("a", h))),
                "A_log": ParamSpec((h,), kind="vector"),
                "dt_bias": ParamSpec((h,), kind="vector"),
                "norm": ParamSpec((spec.value_dim or spec.head_dim,), kind="vector"),
                "o": ParamSpec((spec.width, v))}

    @classmethod
    def cache_need(cls, spec) -> CacheNeed:
        n = record(spec.heads, spec.kv_heads, spec.head_dim, spec.value_dim or spec.head_dim, int(spec.option("conv_taps")))
        return CacheNeed(kind="state", state_shape=(n,), state_dtype="float32")

    def prepare_step(self, shape):
        return plan_state_chunks(self.k, shape)

    def load(self, tensors: dict) -> None:
        super().load(tensors)
        for name in ("conv", "A_log", "dt_bias", "norm"):        # they enter float32 arithmetic: kept in float32
            setattr(self, name, getattr(self, name).float().contiguous())
        self.rate = torch.exp(self.A_log)

    def forward(self, ctx, x, call):
        t = x.shape[0]
        _, state = ctx.cache.view(call.cache)
        proj = ctx.buffer("state.proj", (t, self.cols), self.dtype)
        self.k.linear(x, self.qkvg, proj)
        gates = ctx.buffer("state.gates", (t, 2 * self.heads), torch.float32)
        self.k.linear(x, self.gates, gates)
        gated = ctx.buffer("state.gated", (t, self.heads * self.value_dim), self.dtype)
        self.k.gated_delta(proj, gates, self.conv, self.rate, self.dt_bias, self.norm, self.eps, self.tiny, state, ctx.state_slots,
                           ctx.positions, ctx.token_request, ctx.cu_seqlens, gated, self.heads, self.kv_heads, self.head_dim,
                           self.value_dim, longest=max(ctx.query_lens, default=0), plan=ctx.prepared.get(self.prepare_key),
                           write=call.write)
        out = ctx.buffer("state.out", (t, self.width), self.dtype)
        return self.k.linear(gated, self.o, out)
