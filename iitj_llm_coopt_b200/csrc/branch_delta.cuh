// Where a branch that joins the residual stream comes from, and how a kernel that adds it reads four neighbouring columns of it:
//   form 0  nothing;
//   form 1  rows of the engine's type or float32;
//   form 2  float32 partial sums of a k-split product, added in split order;
//   form 3  the sorted rows of a routed feed-forward with their weights, summed in the order of the token's choices (so the weighted
//           sum is never stored), plus one more row per token where a shared expert's result stands beside them (`extra`: rows of the
//           same type, or partial sums).
#pragma once
#include "common.cuh"

struct BranchDelta {
    const void* data;            // null: none
    int splits;                  // > 0: float32 partial sums, `split_stride` numbers apart
    size_t split_stride;
    const int* place;            // given: `data` holds sorted rows, a token's `top` choices lie at place[token * top + j] (-1: none)
    const float* weights;        // [token * top + j]; null: 1
    int top;
    const void* extra;           // one more row per token beside sorted rows; null: none
    int extra_splits;            // > 0: `extra` is float32 partial sums, `extra_stride` numbers apart
    size_t extra_stride;

    int form() const { return !data ? 0 : place ? 3 : splits > 0 ? 2 : 1; }
};

template <typename T> __device__ __forceinline__ float4 load4(const T* p);
template <> __device__ __forceinline__ float4 load4<float>(const float* p) { return *reinterpret_cast<const float4*>(p); }
template <> __device__ __forceinline__ float4 load4<__nv_bfloat16>(const __nv_bfloat16* p) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
    return make_float4(a.x, a.y, b.x, b.y);
}
template <typename T> __device__ __forceinline__ void store4(T* p, float4 v);
template <> __device__ __forceinline__ void store4<float>(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
template <> __device__ __forceinline__ void store4<__nv_bfloat16>(__nv_bfloat16* p, float4 v) {
    __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    uint2 raw;
    raw.x = *reinterpret_cast<uint32_t*>(&a);
    raw.y = *reinterpret_cast<uint32_t*>(&b);
    *reinterpret_cast<uint2*>(p) = raw;
}

// columns i .. i + 3 of the branch's row s (16-byte aligned pieces: the launcher has checked)
template <typename TD, int FORM>
__device__ __forceinline__ float4 branch4(const BranchDelta& d, size_t s, int width, int i) {
    float4 e = make_float4(0.f, 0.f, 0.f, 0.f);
    if (FORM == 1) {
        e = load4(static_cast<const TD*>(d.data) + s * width + i);
    } else if (FORM == 2) {
        e = sum_parts4(static_cast<const float*>(d.data) + s * width + i, d.splits, d.split_stride);
    } else if (FORM == 3) {
        for (int j0 = 0; j0 < d.top; j0 += 4) {           // four rows' reads side by side, summed in the order of the choices
            float4 y[4];
            float w[4];
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const bool live = j0 + j < d.top;
                const int at = live ? d.place[s * d.top + j0 + j] : -1;
                w[j] = live ? (d.weights ? d.weights[s * d.top + j0 + j] : 1.0f) : 0.f;
                y[j] = at >= 0 ? load4(static_cast<const TD*>(d.data) + (size_t)at * width + i) : make_float4(0.f, 0.f, 0.f, 0.f);
            }
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                e.x = fmaf(w[j], y[j].x, e.x); e.y = fmaf(w[j], y[j].y, e.y);
                e.z = fmaf(w[j], y[j].z, e.z); e.w = fmaf(w[j], y[j].w, e.w);
            }
        }
        if (d.extra) {
            const float4 x = d.extra_splits > 0
                ? sum_parts4(static_cast<const float*>(d.extra) + s * width + i, d.extra_splits, d.extra_stride)
                : load4(static_cast<const TD*>(d.extra) + s * width + i);
            e.x += x.x; e.y += x.y; e.z += x.z; e.w += x.w;
        }
    }
    return e;
}

// column i of the branch's row s
template <typename TD, int FORM>
__device__ __forceinline__ float branch1(const BranchDelta& d, size_t s, int width, int i) {
    float e = 0.f;
    if (FORM == 1) {
        e = to_f32(static_cast<const TD*>(d.data)[s * width + i]);
    } else if (FORM == 2) {
        for (int k = 0; k < d.splits; ++k) e += static_cast<const float*>(d.data)[(size_t)k * d.split_stride + s * width + i];
    } else if (FORM == 3) {
        for (int j = 0; j < d.top; ++j) {
            const int at = d.place[s * d.top + j];
            const float w = d.weights ? d.weights[s * d.top + j] : 1.0f;
            if (at >= 0) e = fmaf(w, to_f32(static_cast<const TD*>(d.data)[(size_t)at * width + i]), e);
        }
        if (d.extra) {
            if (d.extra_splits > 0) {
                float x = 0.f;
                for (int k = 0; k < d.extra_splits; ++k) x += static_cast<const float*>(d.extra)[(size_t)k * d.extra_stride + s * width + i];
                e += x;
            } else {
                e += to_f32(static_cast<const TD*>(d.extra)[s * width + i]);
            }
        }
    }
    return e;
}
