// Mixers with a matrix state per head, kept between steps in one float32 record per request: what their kernels share.
//
// A record holds, per head, `columns` columns of the state, each of `dim` numbers padded with zeros to a multiple of four (`dp`), and
// behind all heads what else the mixer remembers.  Column c of S [dim, vdim] needs value c of a token only, so columns can be dealt out
// to blocks and threads at will.
#pragma once
#include "common.cuh"

constexpr int kMemory = 0;       // matrix memory: columns = vdim + 1 (the normaliser n is the column whose value is always 1), then m
constexpr int kDelta = 1;        // gated delta rule: columns = vdim, then the convolution's rows

__host__ __device__ __forceinline__ int state_dp(int dim) { return (dim + 3) & ~3; }

// log(sigmoid(x)) and log(1 + e^x) without overflow at either end
__device__ __forceinline__ float log_sigmoid(float x) { return fminf(x, 0.f) - log1pf(expf(-fabsf(x))); }
__device__ __forceinline__ float soft_plus(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }
__device__ __forceinline__ float sigmoid_f(float x) { return 1.0f / (1.0f + expf(-x)); }

// the matrix memory's gates of one token and head: (log forget gate, log input gate)
__device__ __forceinline__ float2 memory_gates(const float* __restrict__ gates, const float* __restrict__ bias, int heads, int h, float cap) {
    const float gi = cap * tanhf((gates[h] + bias[h]) / cap);
    const float gf = log_sigmoid(cap * tanhf((gates[heads + h] + bias[heads + h]) / cap));
    return make_float2(gf, gi);
}
