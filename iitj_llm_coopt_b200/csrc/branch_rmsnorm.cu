// residual += factor * branch; out = residual / sqrt(mean(residual^2) + eps) * gain, on the float32 residual stream: a sub-layer's last
// sum (k-split parts, or a routed feed-forward's weighted rows with a shared expert's row), its factor, the residual sum and the norm in
// front of the next sub-layer in one kernel.  The branch's forms: branch_delta.cuh.
//
// Few rows (a decode step): a row is shared by a cluster of blocks, each with width / cluster columns, that exchange their sums of
// squares through each other's shared memory.  Many rows: a block a row.  Odd widths: a block a row, a number a thread.
#include "branch_delta.cuh"

#include <type_traits>

namespace {

template <typename TD, typename TO, int FORM, int PER>
__global__ void __launch_bounds__(256)
branch_rmsnorm_vec_kernel(float* __restrict__ residual, BranchDelta d, float factor, const int* __restrict__ rows,
                          const float* __restrict__ gain, TO* __restrict__ out, int width, float eps, int cluster) {
    pdl_trigger();
    __shared__ float red[32];
    __shared__ float all_ss[8];               // the sums of squares of the cluster's blocks, pushed here by each of them
    const int c = cluster > 1 ? (int)llm_cluster_rank() : 0;
    const int r = blockIdx.x / cluster;
    const int cols = width / cluster, col0 = c * cols;       // this block's columns (a multiple of 4)
    float4 v[PER], w[PER];
#pragma unroll
    for (int j = 0; j < PER; ++j) {           // parameters: nothing before this kernel writes them
        const int i = (threadIdx.x + j * blockDim.x) * 4;
        if (PER <= 4 && i < cols) w[j] = load4(gain + col0 + i);
    }
    pdl_wait();
    const size_t s = rows ? (size_t)rows[r] : (size_t)r;
    float* res = residual + s * width + col0;
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < PER; ++j) {
        const int i = (threadIdx.x + j * blockDim.x) * 4;
        v[j] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (i < cols) {
            v[j] = load4(res + i);
            const float4 e = branch4<TD, FORM>(d, s, width, col0 + i);
            v[j].x = fmaf(factor, e.x, v[j].x); v[j].y = fmaf(factor, e.y, v[j].y);
            v[j].z = fmaf(factor, e.z, v[j].z); v[j].w = fmaf(factor, e.w, v[j].w);
        }
    }
#pragma unroll
    for (int j = 0; j < PER; ++j) {
        const int i = (threadIdx.x + j * blockDim.x) * 4;
        if (i < cols) {
            if (!rows) store4(res + i, v[j]);
            ss += v[j].x * v[j].x + v[j].y * v[j].y + v[j].z * v[j].z + v[j].w * v[j].w;
        }
    }
    float total = block_sum(ss, red);
    if (cluster > 1) {
        if ((int)threadIdx.x < cluster) llm_cluster_write(&all_ss[c], (uint32_t)threadIdx.x, total);
        llm_cluster_sync();                   // every block's sum has arrived in every block; no remote access after this
        total = 0.f;
#pragma unroll
        for (int k = 0; k < 8; ++k)
            if (k < cluster) total += all_ss[k];     // in block order in every block: the same total everywhere
    }
    const float inv = 1.0f / sqrtf(total / (float)width + eps);
    TO* o = out + (size_t)r * width + col0;
#pragma unroll
    for (int j = 0; j < PER; ++j) {
        const int i = (threadIdx.x + j * blockDim.x) * 4;
        if (i < cols) {
            if (PER > 4) w[j] = load4(gain + col0 + i);
            store4(o + i, make_float4(v[j].x * inv * w[j].x, v[j].y * inv * w[j].y, v[j].z * inv * w[j].z, v[j].w * inv * w[j].w));
        }
    }
}

template <typename TD, typename TO, int FORM>
__global__ void __launch_bounds__(256)
branch_rmsnorm_kernel(float* __restrict__ residual, BranchDelta d, float factor, const int* __restrict__ rows,
                      const float* __restrict__ gain, TO* __restrict__ out, int width, float eps) {
    pdl_trigger();
    pdl_wait();
    extern __shared__ float row_buf[];        // width floats
    __shared__ float red[32];
    const int r = blockIdx.x;
    const size_t s = rows ? (size_t)rows[r] : (size_t)r;
    float ss = 0.f;
    for (int i = threadIdx.x; i < width; i += blockDim.x) {
        const float v = fmaf(factor, branch1<TD, FORM>(d, s, width, i), residual[s * width + i]);
        if (!rows) residual[s * width + i] = v;
        row_buf[i] = v;
        ss += v * v;
    }
    const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)width + eps);
    for (int i = threadIdx.x; i < width; i += blockDim.x) out[(size_t)r * width + i] = from_f32<TO>(row_buf[i] * inv * gain[i]);
}

}  // namespace

// residual float32 [*, width].  The branch: rows of `delta_dtype`; with splits > 0 float32 partial sums; with `place` the sorted rows of
// a routed feed-forward, and `extra` beside them.  rows: null, or the rows of the stream that are normed (the stream is then read only).
LLM_API int llm_add_branch_rmsnorm(float* residual, const void* delta, int delta_dtype, int splits, long long split_stride, const int* place,
                                   const float* weights, int top, const void* extra, int extra_splits, long long extra_stride,
                                   float factor, const int* rows, const float* gain, void* out, int out_dtype, int out_rows, int width,
                                   float eps, cudaStream_t stream) {
    if (out_rows == 0) return 0;
    if (width <= 0 || !delta) LLM_FAIL(-1, "add_branch_rmsnorm: width %d, branch %p", width, delta);
    if (splits < 0 || splits > kMaxParts || (splits > 0 && place) || extra_splits < 0 || extra_splits > kMaxParts)
        LLM_FAIL(-1, "add_branch_rmsnorm: %d and %d partial sums (at most %d)", splits, extra_splits, kMaxParts);
    if ((place && top < 1) || (extra && !place)) LLM_FAIL(-1, "add_branch_rmsnorm: sorted rows need a choice a token, and a row beside them needs sorted rows");
    const size_t smem = (size_t)width * sizeof(float);
    if (smem > 200 * 1024) LLM_FAIL(-1, "add_branch_rmsnorm: width %d is larger than 51200", width);
    const BranchDelta d{delta, splits, (size_t)split_stride, place, weights, top, extra, extra_splits, (size_t)extra_stride};
    const int form = d.form();
    const bool vec = !(width % 4) && !(split_stride % 4) && !(extra_stride % 4) && !((uintptr_t)residual & 15) && !((uintptr_t)delta & 15) &&
                     !((uintptr_t)extra & 15) && !((uintptr_t)out & 15) && !((uintptr_t)gain & 15) && width <= 4 * 256 * 16;
    return llm_dispatch_dtype(delta_dtype, [&](auto td) {
        using TD = decltype(td);
        return llm_dispatch_dtype(out_dtype, [&](auto to) {
            using TO = decltype(to);
            auto pick = [&](auto form_tag) {
                constexpr int F = decltype(form_tag)::value;
                if (!vec) {
                    auto kern = branch_rmsnorm_kernel<TD, TO, F>;
                    if (smem > 48 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
                    llm_launch(kern, (unsigned)out_rows, 256, smem, stream, residual, d, factor, rows, gain, (TO*)out, width, eps);
                    return;
                }
                int cluster = out_rows < 512 ? 8 : 1;
                while (cluster > 1 && (width % (4 * cluster) || width / (4 * cluster) < 32)) cluster >>= 1;
                const int vecs = width / (4 * cluster);
                int threads = (vecs + 31) / 32 * 32;
                if (threads > 256) threads = 256;
                const int per = (vecs + threads - 1) / threads;
                auto go = [&](auto kern) {
                    if (cluster > 1)
                        llm_launch_cluster(kern, (unsigned)(out_rows * cluster), threads, 0, stream, (unsigned)cluster, residual, d, factor,
                                           rows, gain, (TO*)out, width, eps, cluster);
                    else
                        llm_launch(kern, (unsigned)out_rows, threads, 0, stream, residual, d, factor, rows, gain, (TO*)out, width, eps, cluster);
                };
                if (per <= 1) go(branch_rmsnorm_vec_kernel<TD, TO, F, 1>);
                else if (per <= 2) go(branch_rmsnorm_vec_kernel<TD, TO, F, 2>);
                else if (per <= 4) go(branch_rmsnorm_vec_kernel<TD, TO, F, 4>);
                else go(branch_rmsnorm_vec_kernel<TD, TO, F, 16>);
            };
            if (form == 1) pick(std::integral_constant<int, 1>{});
            else if (form == 2) pick(std::integral_constant<int, 2>{});
            else pick(std::integral_constant<int, 3>{});
            LLM_CHECK_LAUNCH("add_branch_rmsnorm");
            return 0;
        });
    });
}

LLM_TRACE_EXPORT(branch_rmsnorm)
