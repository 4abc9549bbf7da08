"""`MatrixMemory`: a recurrent mixer with a matrix state per head, exponential input gates and a normaliser beside it (the matrix
memory of xLSTM).

    [q, k, v, z] = x W^T                       (one product, no biases; q, k heads x head_dim, v, z heads x value_dim)
    i = c tanh((x Wi^T + bi) / c),   f = log sigmoid(c tanh((x Wf^T + bf) / c))          per head, c = `gate_cap`
    m_t = max(f_t + m_(t-1), i_t)
    S_t = e^(f_t + m_(t-1) - m_t) S_(t-1) + e^(i_t - m_t) k_t v_t^T,     n_t the same with k_t alone
    o_t = S_t^T q_t / (max(|n_t . q_t|, e^(-m_t)) + tiny)                q scaled by head_dim^(-1/2)
    out = (each head of o divided by its root mean square * gain * sigmoid(z)) Wo^T

S [head_dim, value_dim], n and m are zero for a new request; m starts at zero, so early gates below zero do not blow the state up.
The gates' rows are a product of their own with float32 results: they enter exponentials that compound over the whole sequence.

The state is the layer's cache entry (kind "state"): one record of `record(...)` float32 numbers per request, per head the columns
of S and then n (each padded to a multiple of four numbers), then every head's m.  The cache manager clears it when it admits a
request, so a portion of a prompt simply continues from what the slot holds.
"""
from __future__ import annotations

import torch

from ..config.specs import CacheNeed
from .base import ParamSpec, Part
from .state_plan import KEY, plan_state_chunks


def padded(n: int) -> int:
    return -(-n // 4) * 4


def record(heads: int, dim: int, vdim: int) -> int:
    return padded(heads * (vdim + 1) * padded(dim) + heads)


class MatrixMemory(Part):
    graph_safe = True
    prepare_key = KEY

    def __init__(self, spec, kernels, dtype, position=None):
        self.spec, self.k, self.dtype = spec, kernels, dtype
        self.width, self.heads = spec.width, spec.heads
        self.head_dim, self.value_dim = spec.head_dim, spec.value_dim or spec.head_dim
        self.eps, self.cap, self.tiny = float(spec.option("eps", 1e-6)), float(spec.option("gate_cap")), float(spec.option("tiny", 1e-6))
        self.cols = 2 * self.heads * (self.head_dim + self.value_dim)
        self.qkvg = self.gates = self.gate_bias = self.norm = self.o = None

    @classmethod
    def parameters(cls, spec) -> dict:
        h, qk, v = spec.heads, spec.heads * spec.head_dim, spec.heads * (spec.value_dim or spec.head_dim)
        return {"qkvg": ParamSpec((2 * qk + 2 * v, spec.width), pieces=(("q", qk), ("k", qk), ("v", v), ("g", v))),
                "gates": ParamSpec((2 * h, spec.width), pieces=(("i", h), ("f", h))),
                "gate_bias": ParamSpec((2 * h,), kind="vector", pieces=(("i", h), ("f", h))),
                "norm": ParamSpec((v,), kind="vector"),
                "o": ParamSpec((spec.width, v))}

    @classmethod
    def cache_need(cls, spec) -> CacheNeed:
        return CacheNeed(kind="state", state_shape=(record(spec.heads, spec.head_dim, spec.value_dim or spec.head_dim),),
                         state_dtype="float32")

    def prepare_step(self, shape):
        return plan_state_chunks(self.k, shape)

    def load(self, tensors: dict) -> None:
        super().load(tensors)
        self.gate_bias, self.norm = self.gate_bias.float().contiguous(), self.norm.float().contiguous()

    def forward(self, ctx, x, call):
        t = x.shape[0]
        _, state = ctx.cache.view(call.cache)
        proj = ctx.buffer("state.proj", (t, self.cols), self.dtype)
        self.k.linear(x, self.qkvg, proj)
        gates = ctx.buffer("state.gates", (t, 2 * self.heads), torch.float32)
        self.k.linear(x, self.gates, gates)
        gated = ctx.buffer("state.gated", (t, self.heads * self.value_dim), self.dtype)
        self.k.matrix_memory(proj, gates, self.gate_bias, self.cap, self.norm, self.eps, self.tiny, state, ctx.state_slots, ctx.cu_seqlens,
                             gated, self.heads, self.head_dim, self.value_dim, longest=max(ctx.query_lens, default=0),
                             plan=ctx.prepared.get(self.prepare_key), write=call.write)
        out = ctx.buffer("attn.out", (t, self.width), self.dtype)
        return self.k.linear(gated, self.o, out, defer=True)
