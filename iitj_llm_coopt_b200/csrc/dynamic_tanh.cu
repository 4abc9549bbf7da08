// A norm without statistics, y = tanh(alpha * x) * gain + shift with one alpha for the whole row, on the float32 residual stream;
// the entry of a repeated run of layers; the tanh cap of logits.
//
// llm_add_dynamic_tanh:    v = residual[s] + factor * delta[s]  (delta optional);  out[r] = tanh(alpha v) * gain + shift, or v itself
//                          as the engine's type when no gain is given (what a product that reads the stream wants).  s = rows ? rows[r]
//                          : r.  The new stream is stored only on request.  delta comes in one of three forms: rows of the engine's
//                          type or float32; float32 partial sums of a k-split product, added in split order; or the sorted rows of a
//                          routed feed-forward with their weights, summed here in the order of the token's choices, so the weighted
//                          sum is never stored.
// llm_embed_dynamic_tanh:  x = tanh(alpha * scale * table[id]) * gain + shift as float32, and as the engine's type beside it.
// llm_softcap_f32:         x = cap * tanh(x / cap) in place.
//
// Nothing is summed over a row, so a row is cut into blocks of columns: four columns a thread where the width allows, else one.
#include "branch_delta.cuh"

namespace {

constexpr int kThreads = 256;

__device__ __forceinline__ float4 squash4(float4 v, float alpha, float4 g, float4 b) {
    return make_float4(fmaf(tanhf(alpha * v.x), g.x, b.x), fmaf(tanhf(alpha * v.y), g.y, b.y), fmaf(tanhf(alpha * v.z), g.z, b.z),
                       fmaf(tanhf(alpha * v.w), g.w, b.w));
}

// FORM: 0 no delta, 1 rows, 2 partial sums, 3 weighted sorted rows
template <typename TD, typename TO, int FORM>
__global__ void __launch_bounds__(kThreads)
add_tanh_vec_kernel(float* __restrict__ residual, BranchDelta d, float factor, const int* __restrict__ rows, const float* __restrict__ alpha,
                    const float* __restrict__ gain, const float* __restrict__ shift, TO* __restrict__ out, long long ld_out, int width,
                    int store) {
    pdl_trigger();
    const int i = (blockIdx.y * blockDim.x + threadIdx.x) * 4;
    const bool mine = i < width;
    float a = 0.f;
    float4 g = make_float4(0.f, 0.f, 0.f, 0.f), b = g;
    if (gain && mine) {                    // parameters: nothing before this kernel writes them
        a = alpha[0];
        g = load4(gain + i);
        b = load4(shift + i);
    }
    pdl_wait();
    if (!mine) return;
    const int r = blockIdx.x;
    const size_t s = rows ? (size_t)rows[r] : (size_t)r;
    float* res = residual + s * width + i;
    float4 v = load4(res);
    if (FORM) {
        const float4 e = branch4<TD, FORM>(d, s, width, i);
        v.x = fmaf(factor, e.x, v.x); v.y = fmaf(factor, e.y, v.y); v.z = fmaf(factor, e.z, v.z); v.w = fmaf(factor, e.w, v.w);
        if (store) store4(res, v);
    }
    store4(out + (size_t)r * ld_out + i, gain ? squash4(v, a, g, b) : v);
}

template <typename TD, typename TO, int FORM>
__global__ void __launch_bounds__(kThreads)
add_tanh_kernel(float* __restrict__ residual, BranchDelta d, float factor, const int* __restrict__ rows, const float* __restrict__ alpha,
                const float* __restrict__ gain, const float* __restrict__ shift, TO* __restrict__ out, long long ld_out, int width,
                int store) {
    pdl_trigger();
    pdl_wait();
    const int i = blockIdx.y * blockDim.x + threadIdx.x;
    if (i >= width) return;
    const int r = blockIdx.x;
    const size_t s = rows ? (size_t)rows[r] : (size_t)r;
    float v = residual[s * width + i];
    if (FORM) {
        const float e = branch1<TD, FORM>(d, s, width, i);
        v = fmaf(factor, e, v);
        if (store) residual[s * width + i] = v;
    }
    out[(size_t)r * ld_out + i] = from_f32<TO>(gain ? fmaf(tanhf(alpha[0] * v), gain[i], shift[i]) : v);
}

template <typename TW, typename TO>
__global__ void __launch_bounds__(kThreads)
embed_tanh_kernel(const int* __restrict__ ids, const TW* __restrict__ table, float scale, const float* __restrict__ alpha,
                  const float* __restrict__ gain, const float* __restrict__ shift, float* __restrict__ out, TO* __restrict__ cast,
                  long long ld_cast, int width, int vocab) {
    pdl_trigger();
    pdl_wait();
    const int i = blockIdx.y * blockDim.x + threadIdx.x;
    if (i >= width) return;
    const int t = blockIdx.x, id = ids[t];
    const bool ok = id >= 0 && id < vocab;             // the host refuses such ids; never read out of range
    const float x = ok ? scale * to_f32(table[(size_t)id * width + i]) : 0.f;
    const float y = fmaf(tanhf(alpha[0] * x), gain[i], shift[i]);
    out[(size_t)t * width + i] = y;
    if (cast) cast[(size_t)t * ld_cast + i] = from_f32<TO>(y);
}

template <typename TW, typename TO>
__global__ void __launch_bounds__(kThreads)
embed_tanh_vec_kernel(const int* __restrict__ ids, const TW* __restrict__ table, float scale, const float* __restrict__ alpha,
                      const float* __restrict__ gain, const float* __restrict__ shift, float* __restrict__ out, TO* __restrict__ cast,
                      long long ld_cast, int width, int vocab) {
    pdl_trigger();
    const int i = (blockIdx.y * blockDim.x + threadIdx.x) * 4;
    if (i >= width) return;
    const float a = alpha[0];                              // parameters: nothing before this kernel writes them
    const float4 g = load4(gain + i), b = load4(shift + i);
    pdl_wait();
    const int t = blockIdx.x, id = ids[t];
    float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
    if (id >= 0 && id < vocab) x = load4(table + (size_t)id * width + i);
    const float4 y = squash4(make_float4(scale * x.x, scale * x.y, scale * x.z, scale * x.w), a, g, b);
    store4(out + (size_t)t * width + i, y);
    if (cast) store4(cast + (size_t)t * ld_cast + i, y);
}

__global__ void softcap_kernel(float* __restrict__ x, float cap, size_t n) {
    pdl_trigger();
    pdl_wait();
    const float inv = 1.0f / cap;
    const size_t n4 = ((uintptr_t)x & 15) ? 0 : n / 4;
    for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n4; i += (size_t)gridDim.x * blockDim.x) {
        float4 v = reinterpret_cast<float4*>(x)[i];
        v.x = cap * tanhf(v.x * inv); v.y = cap * tanhf(v.y * inv); v.z = cap * tanhf(v.z * inv); v.w = cap * tanhf(v.w * inv);
        reinterpret_cast<float4*>(x)[i] = v;
    }
    for (size_t i = 4 * n4 + (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (size_t)gridDim.x * blockDim.x)
        x[i] = cap * tanhf(x[i] * inv);
}

}  // namespace

// residual float32 [*, width].  delta: null; rows of `delta_dtype`; with splits > 0 float32 partial sums; with `place` the sorted rows
// of a routed feed-forward.  gain / shift float32 [width] and alpha float32 [1]: all three, or none for the plain stream.  out: rows of
// `out_dtype`, `ld_out` numbers apart.  store: whether the new stream is written back (not with `rows`).
LLM_API int llm_add_dynamic_tanh(float* residual, const void* delta, int delta_dtype, int splits, long long split_stride, const int* place,
                                 const float* weights, int top, float factor, const int* rows, const float* alpha, const float* gain,
                                 const float* shift, void* out, int out_dtype, long long ld_out, int out_rows, int width, int store,
                                 cudaStream_t stream) {
    if (out_rows == 0) return 0;
    if (width <= 0) LLM_FAIL(-1, "add_dynamic_tanh: width %d", width);
    if ((gain == nullptr) != (shift == nullptr) || (gain == nullptr) != (alpha == nullptr))
        LLM_FAIL(-1, "add_dynamic_tanh: alpha, gain and shift come together or not at all");
    if (splits < 0 || splits > kMaxParts || (splits > 0 && (!delta || place))) LLM_FAIL(-1, "add_dynamic_tanh: %d partial sums", splits);
    if (place && (!delta || top < 1)) LLM_FAIL(-1, "add_dynamic_tanh: sorted rows need rows and at least one choice a token");
    if (store && rows) LLM_FAIL(-1, "add_dynamic_tanh: chosen rows of the stream are read only");
    const BranchDelta d{delta, splits, (size_t)split_stride, place, weights, top, nullptr, 0, 0};
    const int form = d.form();
    const bool vec = !(width % 4) && !(ld_out % 4) && !(split_stride % 4) && !((uintptr_t)residual & 15) && !((uintptr_t)delta & 15) &&
                     !((uintptr_t)out & 15) && !((uintptr_t)gain & 15) && !((uintptr_t)shift & 15);
    const int cols = vec ? width / 4 : width;
    const int threads = cols >= kThreads ? kThreads : (cols + 31) / 32 * 32;
    const dim3 grid((unsigned)out_rows, (unsigned)((cols + threads - 1) / threads));
    return llm_dispatch_dtype(delta ? delta_dtype : out_dtype, [&](auto td) {
        using TD = decltype(td);
        return llm_dispatch_dtype(out_dtype, [&](auto to) {
            using TO = decltype(to);
            auto go = [&](auto kern) {
                llm_launch(kern, grid, threads, 0, stream, residual, d, factor, rows, alpha, gain, shift, (TO*)out, ld_out, width, store);
            };
            if (vec) {
                if (form == 0) go(add_tanh_vec_kernel<TD, TO, 0>);
                else if (form == 1) go(add_tanh_vec_kernel<TD, TO, 1>);
                else if (form == 2) go(add_tanh_vec_kernel<TD, TO, 2>);
                else go(add_tanh_vec_kernel<TD, TO, 3>);
            } else {
                if (form == 0) go(add_tanh_kernel<TD, TO, 0>);
                else if (form == 1) go(add_tanh_kernel<TD, TO, 1>);
                else if (form == 2) go(add_tanh_kernel<TD, TO, 2>);
                else go(add_tanh_kernel<TD, TO, 3>);
            }
            LLM_CHECK_LAUNCH("add_dynamic_tanh");
            return 0;
        });
    });
}

// out float32 [tokens, width]; cast: null or rows of `cast_dtype`, `ld_cast` numbers apart.
LLM_API int llm_embed_dynamic_tanh(const int* ids, const void* table, int table_dtype, float scale, const float* alpha, const float* gain,
                                   const float* shift, float* out, void* cast, int cast_dtype, long long ld_cast, int tokens, int width,
                                   int vocab, cudaStream_t stream) {
    if (tokens == 0) return 0;
    const bool vec = !(width % 4) && !(cast && ld_cast % 4) && !((uintptr_t)table & 15) && !((uintptr_t)out & 15) && !((uintptr_t)cast & 15) &&
                     !((uintptr_t)gain & 15) && !((uintptr_t)shift & 15);
    const int cols = vec ? width / 4 : width;
    const int threads = cols >= kThreads ? kThreads : (cols + 31) / 32 * 32;
    const dim3 grid((unsigned)tokens, (unsigned)((cols + threads - 1) / threads));
    return llm_dispatch_dtype(table_dtype, [&](auto tw) {
        using TW = decltype(tw);
        return llm_dispatch_dtype(cast ? cast_dtype : LLM_BF16, [&](auto to) {
            using TO = decltype(to);
            auto go = [&](auto kern) {
                llm_launch(kern, grid, threads, 0, stream, ids, (const TW*)table, scale, alpha, gain, shift, out, (TO*)cast, ld_cast, width, vocab);
            };
            if (vec) go(embed_tanh_vec_kernel<TW, TO>);
            else go(embed_tanh_kernel<TW, TO>);
            LLM_CHECK_LAUNCH("embed_dynamic_tanh");
            return 0;
        });
    });
}

LLM_API int llm_softcap_f32(float* x, float cap, long long n, cudaStream_t stream) {
    if (n <= 0) return 0;
    if (!(cap > 0.f)) LLM_FAIL(-1, "softcap: the cap %g must be positive", (double)cap);
    const long long want = (n / 4 + 255) / 256 + 1;
    llm_launch(softcap_kernel, (unsigned)(want < 148 * 8 ? want : 148 * 8), 256, 0, stream, x, cap, (size_t)n);
    LLM_CHECK_LAUNCH("softcap");
    return 0;
}

LLM_TRACE_EXPORT(dynamic_tanh)
