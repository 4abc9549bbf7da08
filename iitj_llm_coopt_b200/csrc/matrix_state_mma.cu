// Long portions of prompts through the mixers of matrix_state.cu in bfloat16: a portion is cut into chunks of 64 tokens, and what the
// token-by-token walk does inside a chunk is restated as small matrix products on the tensor cores (mma.sync, float32 accumulation).
//
// Precision.  The rows of q, k and v are bfloat16 as their producers left them and enter the products exactly; their float32 factors
// (scales, unit lengths, decays) are applied to the products' float32 results.  Every float32 operand (the state, the weights between
// tokens, what the delta rule writes) is split into a high and a low bfloat16 half, x = hi + lo up to 2^-17 of x, and multiplied twice
// (three times where both sides are split; lo * lo is left out).  The state itself is carried in float32.
//
// Matrix memory, per head, F_t the sum of the log forget gates from the chunk's start up to t, 0 the state before the chunk:
//     weight of token s in what t sees   D_ts = exp(F_t - F_s + i_s - m_t)  (s <= t),   of the state  e_t = exp(F_t + m_0 - m_t)
//     o_t = e_t S_0^T q_t + sum_s D_ts (q_t . k_s) v_s,       S_end = e_end S_0 + sum_s D_end,s k_s v_s^T
//   llm_memory_chunk_gather   the chunks' own sums, all chunks side by side;
//   llm_memory_chunk_scan     the state at every chunk's start (the running sum along each request), and the state it leaves;
//   llm_memory_chunk_out      every chunk's outputs, all chunks side by side.
//
// Gated delta rule, G_t the sum of the log decays from the chunk's start up to t, k and q unit vectors:
//     A_ts = beta_t exp(G_t - G_s) k_t . k_s  (s < t),   P_ts = exp(G_t - G_s) q_t . k_s  (s <= t)
//     U = (I + A)^-1 diag(beta) (V - diag(e^G) K S_0),    O = diag(e^G) Q S_0 + P U,    S_end = e^(G_end) S_0 + (diag(e^(G_end - G)) K)^T U
//   llm_delta_chunk_tri       (I + A)^-1 diag(beta) and P of every chunk and head, and the factors of its rows, all side by side: the
//                             16 x 16 diagonal blocks are inverted by forward substitution, the blocks below from them;
//   llm_delta_chunk_walk      the chunks of a request in order, a block per head and 32 columns of the state, which stays in its
//                             accumulators; the next chunk's rows and matrices travel (cp.async) while one is worked on.
#include "matrix_state.cuh"

namespace {

constexpr int kC = 64;                 // tokens of a chunk
constexpr int kThreads = 128;
typedef __nv_bfloat16 bf16;

__device__ __forceinline__ uint32_t smem_u32(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void cp_async16(void* dst, const void* src, bool live) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(live ? 16 : 0) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], const void* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void ldsm4t(uint32_t (&r)[4], const void* p) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(p)));
}
__device__ __forceinline__ void mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// Fragment addresses in a row-major shared array of `ld` numbers a row (16-byte aligned rows), for this lane.
// A rows x k, as stored;  A from an array stored k x rows;  B (two n-tiles of 8) stored n x k;  B stored k x n.
__device__ __forceinline__ const bf16* at_a(const bf16* p, int ld, int row, int k) {
    const int l = threadIdx.x & 31;
    return p + (size_t)(row + (l & 15)) * ld + k + (l >> 4) * 8;
}
__device__ __forceinline__ const bf16* at_a_t(const bf16* p, int ld, int row, int k) {
    const int l = threadIdx.x & 31, m = l >> 3;
    return p + (size_t)(k + (m >> 1) * 8 + (l & 7)) * ld + row + (m & 1) * 8;
}
__device__ __forceinline__ const bf16* at_b_nk(const bf16* p, int ld, int n, int k) {
    const int l = threadIdx.x & 31, m = l >> 3;
    return p + (size_t)(n + (m >> 1) * 8 + (l & 7)) * ld + k + (m & 1) * 8;
}
__device__ __forceinline__ const bf16* at_b_kn(const bf16* p, int ld, int n, int k) {
    const int l = threadIdx.x & 31, m = l >> 3;
    return p + (size_t)(k + (m & 1) * 8 + (l & 7)) * ld + n + (m >> 1) * 8;
}

__device__ __forceinline__ uint32_t pack2(float a, float b) {
    __nv_bfloat162 v = __floats2bfloat162_rn(a, b);
    return *reinterpret_cast<uint32_t*>(&v);
}
// (a, b) as high halves and what they leave
__device__ __forceinline__ void split2(float a, float b, uint32_t& hi, uint32_t& lo) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
    const float2 f = __bfloat1622float2(h);
    hi = *reinterpret_cast<const uint32_t*>(&h);
    lo = pack2(a - f.x, b - f.y);
}

// rows [t0, t0 + n) of `cols` numbers (a multiple of 8) from column `col` on into a [kC, ld] array, zeros behind
__device__ __forceinline__ void load_rows(bf16* dst, int ld, const bf16* __restrict__ src, size_t src_ld, int t0, int n, int col, int cols,
                                          int live_cols) {
    const int pieces = cols / 8;
    for (int x = threadIdx.x; x < kC * pieces; x += kThreads) {
        const int r = x / pieces, c = (x % pieces) * 8;
        const bool live = r < n && c < live_cols;
        cp_async16(dst + (size_t)r * ld + c, live ? src + (size_t)(t0 + r) * src_ld + col + c : src, live);
    }
}

// inclusive sums over 64 numbers, two a lane (2 * lane, 2 * lane + 1), by one warp
__device__ __forceinline__ void scan64(float& a, float& b) {
    const int lane = threadIdx.x & 31;
    float s = a + b;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
        const float x = __shfl_up_sync(0xffffffffu, s, o);
        if (lane >= o) s += x;
    }
    float prev = __shfl_up_sync(0xffffffffu, s, 1);
    if (lane == 0) prev = 0.f;
    a += prev;
    b += a;
}

// ---- matrix memory --------------------------------------------------------------------------------------------------
struct MemoryArgs {
    const bf16* proj;
    int ld;
    const float4* gates;               // (f, i, m, m before) [tokens, heads]
    const int4* chunks;                // (request, first token, tokens, index in its request)
    float* own;                        // [chunks, heads, vdim + 1, dim]: what a chunk gathers by itself
    float* decay;                      // [chunks, heads]
    bf16* start_hi;                    // the state at a chunk's start, in two halves
    bf16* start_lo;
    float* o;                          // [tokens, heads, o_ld]
    int heads, dim, vdim, o_ld;
    float q_scale;
};

// F (sums of f), i, m of the chunk's tokens into shared memory; tokens behind its end weigh nothing
__device__ __forceinline__ void chunk_gates(const MemoryArgs& a, int4 ch, int h, float* F, float* I, float* M) {
    if (threadIdx.x < 32) {
        const int lane = threadIdx.x;
        float f[2], i[2], m[2];
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const int t = 2 * lane + e;
            const float4 g = t < ch.z ? a.gates[(size_t)(ch.y + t) * a.heads + h] : make_float4(0.f, -INFINITY, 0.f, 0.f);
            f[e] = g.x; i[e] = g.y; m[e] = g.z;
        }
        scan64(f[0], f[1]);
#pragma unroll
        for (int e = 0; e < 2; ++e) { F[2 * lane + e] = f[e]; I[2 * lane + e] = i[e]; M[2 * lane + e] = m[e]; }
    }
}

__global__ void __launch_bounds__(kThreads)
memory_gather_kernel(MemoryArgs a) {
    pdl_trigger();
    pdl_wait();
    extern __shared__ __align__(16) unsigned char sm_raw[];
    __shared__ float F[kC], I[kC], M[kC];
    const int D = a.dim, kld = D + 8, vld = 72;
    bf16* sv = reinterpret_cast<bf16*>(sm_raw);            // [kC][72]
    bf16* khi = sv + kC * vld;                             // [kC][D + 8]
    bf16* klo = khi + kC * kld;
    const int4 ch = a.chunks[blockIdx.x];
    const int h = blockIdx.y, c0 = blockIdx.z * 64, qk = a.heads * D;
    load_rows(sv, vld, a.proj, a.ld, ch.y, ch.z, 2 * qk + h * a.vdim + c0, 64, a.vdim - c0);
    load_rows(khi, kld, a.proj, a.ld, ch.y, ch.z, qk + h * D, D, D);
    cp_async_commit();
    chunk_gates(a, ch, h, F, I, M);
    cp_async_wait<0>();
    __syncthreads();
    const float f_end = F[ch.z - 1], m_end = M[ch.z - 1];
    for (int x = threadIdx.x; x < kC * (D / 2); x += kThreads) {        // k times its weight, in two halves
        const int s = x / (D / 2), i = (x % (D / 2)) * 2;
        const float w = s < ch.z ? expf(f_end - F[s] + I[s] - m_end) : 0.f;
        uint32_t* at = reinterpret_cast<uint32_t*>(khi + s * kld + i);
        const float2 k = __bfloat1622float2(*reinterpret_cast<__nv_bfloat162*>(at));
        split2(k.x * w, k.y * w, *at, *reinterpret_cast<uint32_t*>(klo + s * kld + i));
    }
    __syncthreads();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    float* own = a.own + ((size_t)blockIdx.x * a.heads + h) * (a.vdim + 1) * D;
    uint32_t va[kC / 16][4];
#pragma unroll
    for (int ks = 0; ks < kC / 16; ++ks) ldsm4t(va[ks], at_a_t(sv, vld, warp * 16, ks * 16));
    const int c = c0 + warp * 16 + (lane >> 2);
    for (int d0 = 0; d0 < D; d0 += 16) {
        float acc[2][4] = {};
#pragma unroll
        for (int ks = 0; ks < kC / 16; ++ks) {
            uint32_t b[4];
            ldsm4t(b, at_b_kn(khi, kld, d0, ks * 16));
            mma(acc[0], va[ks], b[0], b[1]);
            mma(acc[1], va[ks], b[2], b[3]);
            ldsm4t(b, at_b_kn(klo, kld, d0, ks * 16));
            mma(acc[0], va[ks], b[0], b[1]);
            mma(acc[1], va[ks], b[2], b[3]);
        }
#pragma unroll
        for (int n = 0; n < 2; ++n) {
            float* at = own + (size_t)c * D + d0 + n * 8 + 2 * (lane & 3);
            if (c < a.vdim) *reinterpret_cast<float2*>(at) = make_float2(acc[n][0], acc[n][1]);
            if (c + 8 < a.vdim) *reinterpret_cast<float2*>(at + 8 * (size_t)D) = make_float2(acc[n][2], acc[n][3]);
        }
    }
    if (blockIdx.z == 0) {             // the normaliser's column, and the decay over the chunk
        for (int i = threadIdx.x; i < D; i += kThreads) {
            float n = 0.f;
            for (int s = 0; s < kC; ++s) n += __bfloat162float(khi[s * kld + i]) + __bfloat162float(klo[s * kld + i]);
            own[(size_t)a.vdim * D + i] = n;
        }
        if (threadIdx.x == 0) a.decay[(size_t)blockIdx.x * a.heads + h] = expf(f_end + a.gates[(size_t)ch.y * a.heads + h].w - m_end);
    }
}

// per_head = (vdim + 1) * dim; four numbers a thread
__global__ void __launch_bounds__(256)
memory_scan_kernel(const float* __restrict__ own, const float* __restrict__ decay, bf16* __restrict__ start_hi, bf16* __restrict__ start_lo,
                   const int* __restrict__ longs, float* __restrict__ state, long long slot_stride, const int* __restrict__ state_slots,
                   int heads, int per_head, int write) {
    pdl_trigger();
    pdl_wait();
    const int b = longs[3 * blockIdx.y], first = longs[3 * blockIdx.y + 1], n = longs[3 * blockIdx.y + 2];
    const size_t x = 4 * ((size_t)blockIdx.x * blockDim.x + threadIdx.x), all = (size_t)heads * per_head;
    if (x >= all) return;
    const int h = (int)(x / per_head);
    float* at = state + (size_t)state_slots[b] * slot_stride + x;
    float4 S = *reinterpret_cast<const float4*>(at);
    constexpr int kAhead = 8;
    for (int j0 = 0; j0 < n; j0 += kAhead) {
        float4 add[kAhead];
        float dec[kAhead];
#pragma unroll
        for (int e = 0; e < kAhead; ++e)
            if (j0 + e < n) {
                add[e] = *reinterpret_cast<const float4*>(own + (size_t)(first + j0 + e) * all + x);
                dec[e] = decay[(size_t)(first + j0 + e) * heads + h];
            }
#pragma unroll
        for (int e = 0; e < kAhead; ++e)
            if (j0 + e < n) {
                uint2 hi, lo;
                split2(S.x, S.y, hi.x, lo.x);
                split2(S.z, S.w, hi.y, lo.y);
                const size_t to = (size_t)(first + j0 + e) * all + x;
                *reinterpret_cast<uint2*>(start_hi + to) = hi;
                *reinterpret_cast<uint2*>(start_lo + to) = lo;
                S = make_float4(fmaf(dec[e], S.x, add[e].x), fmaf(dec[e], S.y, add[e].y), fmaf(dec[e], S.z, add[e].z), fmaf(dec[e], S.w, add[e].w));
            }
    }
    if (write) *reinterpret_cast<float4*>(at) = S;
}

__global__ void __launch_bounds__(kThreads)
memory_out_kernel(MemoryArgs a) {
    pdl_trigger();
    pdl_wait();
    extern __shared__ __align__(16) unsigned char sm_raw[];
    __shared__ float F[kC], I[kC], M[kC];
    const int D = a.dim, ld = D + 8, vld = 72;
    bf16* sq = reinterpret_cast<bf16*>(sm_raw);
    bf16* sk = sq + kC * ld;
    bf16* shi = sk + kC * ld;          // [64 columns][D + 8]
    bf16* slo = shi + 64 * ld;
    bf16* sv = slo + 64 * ld;          // [kC][72]
    const int4 ch = a.chunks[blockIdx.x];
    const int h = blockIdx.y, c0 = blockIdx.z * 64, qk = a.heads * D;
    load_rows(sq, ld, a.proj, a.ld, ch.y, ch.z, h * D, D, D);
    load_rows(sk, ld, a.proj, a.ld, ch.y, ch.z, qk + h * D, D, D);
    load_rows(sv, vld, a.proj, a.ld, ch.y, ch.z, 2 * qk + h * a.vdim + c0, 64, a.vdim - c0);
    const size_t base = ((size_t)blockIdx.x * a.heads + h) * (a.vdim + 1) * D;
    load_rows(shi, ld, a.start_hi + base, D, c0, min(64, a.vdim - c0), 0, D, D);
    load_rows(slo, ld, a.start_lo + base, D, c0, min(64, a.vdim - c0), 0, D, D);
    cp_async_commit();
    chunk_gates(a, ch, h, F, I, M);
    const float m0 = a.gates[(size_t)ch.y * a.heads + h].w;
    cp_async_wait<0>();
    __syncthreads();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, row = warp * 16;
    if (row >= ch.z) return;           // (no barrier follows)
    float o[8][4] = {}, s[8][4] = {};
    for (int k0 = 0; k0 < D; k0 += 16) {
        uint32_t q[4], b[4];
        ldsm4(q, at_a(sq, ld, row, k0));
#pragma unroll
        for (int n = 0; n < 4; ++n) {
            ldsm4(b, at_b_nk(shi, ld, n * 16, k0));
            mma(o[2 * n], q, b[0], b[1]);
            mma(o[2 * n + 1], q, b[2], b[3]);
            ldsm4(b, at_b_nk(slo, ld, n * 16, k0));
            mma(o[2 * n], q, b[0], b[1]);
            mma(o[2 * n + 1], q, b[2], b[3]);
            if (n <= warp) {           // keys behind the warp's last token weigh nothing
                ldsm4(b, at_b_nk(sk, ld, n * 16, k0));
                mma(s[2 * n], q, b[0], b[1]);
                mma(s[2 * n + 1], q, b[2], b[3]);
            }
        }
    }
    const int t[2] = {row + (lane >> 2), row + (lane >> 2) + 8};
    float norm[2] = {0.f, 0.f}, e[2], ft[2], mt[2];
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        ft[r] = F[t[r]];
        mt[r] = M[t[r]];
        e[r] = t[r] < ch.z ? expf(ft[r] + (m0 - mt[r])) : 0.f;
    }
#pragma unroll
    for (int n = 0; n < 8; ++n)
#pragma unroll
        for (int x = 0; x < 4; ++x) o[n][x] *= e[x >> 1];
#pragma unroll
    for (int n = 0; n < 4; ++n) {
        if (n > warp) continue;
        uint32_t hi[4], lo[4], b[4];
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            float* p = s[2 * n + half];
#pragma unroll
            for (int x = 0; x < 4; ++x) {
                const int key = n * 16 + half * 8 + 2 * (lane & 3) + (x & 1), r = x >> 1;
                p[x] = key <= t[r] && t[r] < ch.z ? p[x] * expf((ft[r] - F[key]) + (I[key] - mt[r])) : 0.f;     // near keys first: long sums cancel
                norm[r] += p[x];
            }
            split2(p[0], p[1], hi[2 * half], lo[2 * half]);
            split2(p[2], p[3], hi[2 * half + 1], lo[2 * half + 1]);
        }
#pragma unroll
        for (int v = 0; v < 4; ++v) {
            ldsm4t(b, at_b_kn(sv, vld, v * 16, n * 16));
            mma(o[2 * v], hi, b[0], b[1]);
            mma(o[2 * v + 1], hi, b[2], b[3]);
            mma(o[2 * v], lo, b[0], b[1]);
            mma(o[2 * v + 1], lo, b[2], b[3]);
        }
    }
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        if (t[r] >= ch.z) continue;
        float* at = a.o + ((size_t)(ch.y + t[r]) * a.heads + h) * a.o_ld + c0;
#pragma unroll
        for (int n = 0; n < 8; ++n) {
            const int c = n * 8 + 2 * (lane & 3);
            if (c0 + c < a.vdim) *reinterpret_cast<float2*>(at + c) = make_float2(o[n][2 * r] * a.q_scale, o[n][2 * r + 1] * a.q_scale);
        }
    }
    if (blockIdx.z == 0) {             // n . q: the chunk's own keys, and the normaliser at its start
        const bf16* nh = a.start_hi + base + (size_t)a.vdim * D;
        const bf16* nl = a.start_lo + base + (size_t)a.vdim * D;
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            float far = 0.f;
            for (int i = lane & 3; i < D; i += 4)
                far = fmaf(__bfloat162float(nh[i]) + __bfloat162float(nl[i]), __bfloat162float(sq[(size_t)t[r] * ld + i]), far);
            float n = fmaf(e[r], far, norm[r]);
            n += __shfl_xor_sync(0xffffffffu, n, 1);
            n += __shfl_xor_sync(0xffffffffu, n, 2);
            if ((lane & 3) == 0 && t[r] < ch.z) a.o[((size_t)(ch.y + t[r]) * a.heads + h) * a.o_ld + a.vdim] = n * a.q_scale;
        }
    }
}

// ---- gated delta rule -----------------------------------------------------------------------------------------------
constexpr int kTri = 4 * kC * kC;      // numbers of a chunk's matrices: the inverse in two halves, then P in two halves
constexpr int kFactors = 4 * kC;       // e^G rk, e^G rq, e^(G_end - G) rk of its rows, then e^(G_end)

struct DeltaArgs {
    const bf16* qkv;                   // [tokens, channels]
    int channels;
    const float2* unit;                // (rq, rk) [tokens, kv_heads]
    const float2* steps;               // (log decay, beta) [tokens, heads]
    const int4* chunks;
    const int* longs;
    bf16* tri;                         // [chunks, heads, kTri]
    float* factors;                    // [chunks, heads, kFactors]
    float* state;
    long long slot_stride;
    const int* state_slots;
    float* o;                          // [tokens, heads, o_ld]
    int heads, kv_heads, dim, vdim, o_ld, write;
};

__global__ void __launch_bounds__(kThreads)
delta_tri_kernel(DeltaArgs a) {
    pdl_trigger();
    pdl_wait();
    extern __shared__ __align__(16) unsigned char sm_raw[];
    __shared__ float G[kC], rq[kC], rk[kC], beta[kC];
    const int D = a.dim, ld = D + 8, ald = kC + 1;
    bf16* sq = reinterpret_cast<bf16*>(sm_raw);
    bf16* sk = sq + kC * ld;
    float* A = reinterpret_cast<float*>(sk + kC * ld);     // [kC][kC + 1]
    float* X = A + kC * ald;                               // the inverse, the same shape
    float* Y = X + kC * ald;                               // [3][16][17]: a diagonal's sums
    const int4 ch = a.chunks[blockIdx.x];
    const int h = blockIdx.y, g = h / (a.heads / a.kv_heads), qk = a.kv_heads * D;
    load_rows(sq, ld, a.qkv, a.channels, ch.y, ch.z, g * D, D, D);
    load_rows(sk, ld, a.qkv, a.channels, ch.y, ch.z, qk + g * D, D, D);
    cp_async_commit();
    float* fac = a.factors + ((size_t)blockIdx.x * a.heads + h) * kFactors;
    if (threadIdx.x < 32) {
        const int lane = threadIdx.x;
        float s[2];
        float2 un[2];
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const int t = 2 * lane + e;
            const bool live = t < ch.z;
            const float2 st = live ? a.steps[(size_t)(ch.y + t) * a.heads + h] : make_float2(0.f, 0.f);
            un[e] = live ? a.unit[(size_t)(ch.y + t) * a.kv_heads + g] : make_float2(0.f, 0.f);
            s[e] = st.x;
            beta[t] = st.y; rq[t] = un[e].x; rk[t] = un[e].y;
        }
        scan64(s[0], s[1]);
        const float end = __shfl_sync(0xffffffffu, s[1], 31);          // tokens behind the chunk's end decay nothing
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const int t = 2 * lane + e;
            G[t] = s[e];
            fac[t] = expf(s[e]) * un[e].y;
            fac[kC + t] = expf(s[e]) * un[e].x;
            fac[2 * kC + t] = expf(end - s[e]) * un[e].y;
        }
        if (lane == 0) fac[3 * kC] = expf(end);
    }
    cp_async_wait<0>();
    __syncthreads();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, row = warp * 16;
    float kk[8][4] = {}, pq[8][4] = {};
    for (int k0 = 0; k0 < D; k0 += 16) {
        uint32_t q[4], k[4], b[4];
        ldsm4(q, at_a(sq, ld, row, k0));
        ldsm4(k, at_a(sk, ld, row, k0));
#pragma unroll
        for (int n = 0; n < 4; ++n) {
            if (n > warp) continue;
            ldsm4(b, at_b_nk(sk, ld, n * 16, k0));
            mma(kk[2 * n], k, b[0], b[1]);
            mma(kk[2 * n + 1], k, b[2], b[3]);
            mma(pq[2 * n], q, b[0], b[1]);
            mma(pq[2 * n + 1], q, b[2], b[3]);
        }
    }
    bf16* tri = a.tri + ((size_t)blockIdx.x * a.heads + h) * kTri;
#pragma unroll
    for (int n = 0; n < 8; ++n)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            const int t = row + (lane >> 2) + 8 * r, s = n * 8 + 2 * (lane & 3);
            float p[2];
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const float w = s + e <= t ? expf(G[t] - G[s + e]) * rk[s + e] : 0.f;
                A[t * ald + s + e] = s + e < t ? beta[t] * rk[t] * w * kk[n][2 * r + e] : 0.f;
                X[t * ald + s + e] = 0.f;
                p[e] = rq[t] * w * pq[n][2 * r + e];
            }
            uint32_t hi, lo;
            split2(p[0], p[1], hi, lo);
            *reinterpret_cast<uint32_t*>(tri + 2 * kC * kC + t * kC + s) = hi;
            *reinterpret_cast<uint32_t*>(tri + 3 * kC * kC + t * kC + s) = lo;
        }
    __syncthreads();
    // (I + A)^-1: a warp inverts a diagonal block, a lane a column of it
    if (lane < 16) {
        float x[16];
#pragma unroll
        for (int i = 0; i < 16; ++i) {
            float v = i == lane ? 1.f : 0.f;
#pragma unroll
            for (int j = 0; j < i; ++j) v = fmaf(-A[(row + i) * ald + row + j], x[j], v);
            x[i] = i < lane ? 0.f : v;
            X[(row + i) * ald + row + lane] = x[i];
        }
    }
    __syncthreads();
    // block (I, J) below the diagonal, d = I - J: -inverse_II * sum over K of A_IK inverse_KJ
    for (int d = 1; d < 4; ++d) {
        const int blocks = 4 - d;
        for (int x = threadIdx.x; x < blocks * 256; x += kThreads) {
            const int J = x >> 8, r = (x >> 4) & 15, c = x & 15, I = J + d;
            float acc = 0.f;
            for (int k = 16 * J; k < 16 * I; ++k) acc = fmaf(A[(16 * I + r) * ald + k], X[k * ald + 16 * J + c], acc);
            Y[(J * 16 + r) * 17 + c] = acc;
        }
        __syncthreads();
        for (int x = threadIdx.x; x < blocks * 256; x += kThreads) {
            const int J = x >> 8, r = (x >> 4) & 15, c = x & 15, I = J + d;
            float acc = 0.f;
#pragma unroll
            for (int k = 0; k < 16; ++k) acc = fmaf(X[(16 * I + r) * ald + 16 * I + k], Y[(J * 16 + k) * 17 + c], acc);
            X[(16 * I + r) * ald + 16 * J + c] = -acc;
        }
        __syncthreads();
    }
    for (int x = threadIdx.x; x < kC * kC / 2; x += kThreads) {
        const int t = x / (kC / 2), s = (x % (kC / 2)) * 2;
        uint32_t hi, lo;
        split2(X[t * ald + s] * beta[s], X[t * ald + s + 1] * beta[s + 1], hi, lo);
        *reinterpret_cast<uint32_t*>(tri + t * kC + s) = hi;
        *reinterpret_cast<uint32_t*>(tri + kC * kC + t * kC + s) = lo;
    }
}

constexpr int kCols = 32;              // columns of the state a block of the walk keeps
constexpr int kCld = kCols + 8, kTld = kC + 8;

template <int D> struct DeltaStage {
    bf16 k[kC][D + 8], q[kC][D + 8], v[kC][kCld], m[4][kC][kTld];
    float f[kFactors];
};
template <int D> struct DeltaShared {
    DeltaStage<D> stage[2];
    bf16 s[2][kCols][D + 8];           // the state at the chunk's start, [column][row], in two halves
    bf16 r[2][kC][kCld], u[2][kC][kCld], w[2][kC][kCld];
};

template <int D>
__global__ void __launch_bounds__(kThreads)
delta_walk_kernel(DeltaArgs a) {
    pdl_trigger();
    pdl_wait();
    extern __shared__ __align__(16) unsigned char sm_raw[];
    DeltaShared<D>& sh = *reinterpret_cast<DeltaShared<D>*>(sm_raw);
    constexpr int NT = D / 16;         // n-tiles of a warp's half of the state's rows
    const int b = a.longs[3 * blockIdx.z], first = a.longs[3 * blockIdx.z + 1], n_chunks = a.longs[3 * blockIdx.z + 2];
    const int h = blockIdx.y, c0 = blockIdx.x * kCols, g = h / (a.heads / a.kv_heads), qk = a.kv_heads * D;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, row = warp * 16, quad = lane >> 2, pair = 2 * (lane & 3);
    auto fetch = [&](int j) {
        DeltaStage<D>& st = sh.stage[j & 1];
        const int4 ch = a.chunks[first + j];
        load_rows(&st.k[0][0], D + 8, a.qkv, a.channels, ch.y, ch.z, qk + g * D, D, D);
        load_rows(&st.q[0][0], D + 8, a.qkv, a.channels, ch.y, ch.z, g * D, D, D);
        load_rows(&st.v[0][0], kCld, a.qkv, a.channels, ch.y, ch.z, 2 * qk + h * a.vdim + c0, kCols, a.vdim - c0);
        const size_t at = (size_t)(first + j) * a.heads + h;
        const bf16* tri = a.tri + at * kTri;
        for (int x = threadIdx.x; x < kTri / 8; x += kThreads) {
            const int r = x / (kC / 8), c = (x % (kC / 8)) * 8;
            cp_async16(&st.m[0][0][0] + (size_t)r * kTld + c, tri + (size_t)r * kC + c, true);
        }
        const float* f = a.factors + at * kFactors;
        for (int x = threadIdx.x; x < kFactors / 4; x += kThreads) cp_async16(st.f + 4 * x, f + 4 * x, true);
        cp_async_commit();
    };
    fetch(0);
    // the state's columns c (rows of these tiles) and rows i: warp w keeps columns 16 (w & 1) .. and the half w >> 1 of the rows
    const int cw = 16 * (warp & 1), iw = (warp >> 1) * (D / 2);
    float* S = a.state + (size_t)a.state_slots[b] * a.slot_stride + (size_t)h * a.vdim * D;
    float acc[NT][4];
    auto spill = [&]() {               // the state in two halves, for the products that read it
#pragma unroll
        for (int n = 0; n < NT; ++n)
#pragma unroll
            for (int r = 0; r < 2; ++r) {
                uint32_t hi, lo;
                split2(acc[n][2 * r], acc[n][2 * r + 1], hi, lo);
                *reinterpret_cast<uint32_t*>(&sh.s[0][cw + quad + 8 * r][iw + n * 8 + pair]) = hi;
                *reinterpret_cast<uint32_t*>(&sh.s[1][cw + quad + 8 * r][iw + n * 8 + pair]) = lo;
            }
    };
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            const int c = c0 + cw + quad + 8 * r;
            const float2 v = c < a.vdim ? *reinterpret_cast<const float2*>(S + (size_t)c * D + iw + n * 8 + pair) : make_float2(0.f, 0.f);
            acc[n][2 * r] = v.x;
            acc[n][2 * r + 1] = v.y;
        }
    spill();
    for (int j = 0; j < n_chunks; ++j) {
        const DeltaStage<D>& st = sh.stage[j & 1];
        if (j + 1 < n_chunks) {
            fetch(j + 1);              // (its stage was last read before the barrier that ended the chunk before)
            cp_async_wait<1>();
        } else {
            cp_async_wait<0>();
        }
        __syncthreads();
        const int4 ch = a.chunks[first + j];
        // K S and Q S for the warp's 16 tokens
        float ks[4][4] = {}, qs[4][4] = {};
#pragma unroll
        for (int k0 = 0; k0 < D; k0 += 16) {
            uint32_t fk[4], fq[4], bb[4];
            ldsm4(fk, at_a(&st.k[0][0], D + 8, row, k0));
            ldsm4(fq, at_a(&st.q[0][0], D + 8, row, k0));
#pragma unroll
            for (int half = 0; half < 2; ++half)
#pragma unroll
                for (int n = 0; n < 2; ++n) {
                    ldsm4(bb, at_b_nk(&sh.s[half][0][0], D + 8, n * 16, k0));
                    mma(ks[2 * n], fk, bb[0], bb[1]);
                    mma(ks[2 * n + 1], fk, bb[2], bb[3]);
                    mma(qs[2 * n], fq, bb[0], bb[1]);
                    mma(qs[2 * n + 1], fq, bb[2], bb[3]);
                }
        }
        // what every token has left to write before the earlier ones of its chunk are taken off: v - e^G rk (k S)
#pragma unroll
        for (int n = 0; n < 4; ++n)
#pragma unroll
            for (int r = 0; r < 2; ++r) {
                const int t = row + quad + 8 * r, c = n * 8 + pair;
                const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&st.v[t][c]));
                const float f = st.f[t];
                uint32_t hi, lo;
                split2(fmaf(-f, ks[n][2 * r], v.x), fmaf(-f, ks[n][2 * r + 1], v.y), hi, lo);
                *reinterpret_cast<uint32_t*>(&sh.r[0][t][c]) = hi;
                *reinterpret_cast<uint32_t*>(&sh.r[1][t][c]) = lo;
                qs[n][2 * r] *= st.f[kC + t];
                qs[n][2 * r + 1] *= st.f[kC + t];
            }
        __syncthreads();
        // U = the inverse times that (rows of later tokens weigh nothing: blocks above the diagonal are skipped)
        auto tri_product = [&](float (&d)[4][4], int which, const bf16 (&x)[2][kC][kCld]) {
#pragma unroll
            for (int k = 0; k < 4; ++k) {
                if (k > warp) continue;
                uint32_t hi[4], lo[4], bb[4];
                ldsm4(hi, at_a(&st.m[which][0][0], kTld, row, k * 16));
                ldsm4(lo, at_a(&st.m[which + 1][0][0], kTld, row, k * 16));
#pragma unroll
                for (int n = 0; n < 2; ++n) {
                    ldsm4t(bb, at_b_kn(&x[0][0][0], kCld, n * 16, k * 16));
                    mma(d[2 * n], hi, bb[0], bb[1]);
                    mma(d[2 * n + 1], hi, bb[2], bb[3]);
                    mma(d[2 * n], lo, bb[0], bb[1]);
                    mma(d[2 * n + 1], lo, bb[2], bb[3]);
                    ldsm4t(bb, at_b_kn(&x[1][0][0], kCld, n * 16, k * 16));
                    mma(d[2 * n], hi, bb[0], bb[1]);
                    mma(d[2 * n + 1], hi, bb[2], bb[3]);
                }
            }
        };
        float u[4][4] = {};
        tri_product(u, 0, sh.r);
#pragma unroll
        for (int n = 0; n < 4; ++n)
#pragma unroll
            for (int r = 0; r < 2; ++r) {
                const int t = row + quad + 8 * r, c = n * 8 + pair;
                const float w = st.f[2 * kC + t];
                uint32_t hi, lo;
                split2(u[n][2 * r], u[n][2 * r + 1], hi, lo);
                *reinterpret_cast<uint32_t*>(&sh.u[0][t][c]) = hi;
                *reinterpret_cast<uint32_t*>(&sh.u[1][t][c]) = lo;
                split2(w * u[n][2 * r], w * u[n][2 * r + 1], hi, lo);
                *reinterpret_cast<uint32_t*>(&sh.w[0][t][c]) = hi;
                *reinterpret_cast<uint32_t*>(&sh.w[1][t][c]) = lo;
            }
        __syncthreads();
        tri_product(qs, 2, sh.u);      // O = e^G rq (q S) + P U
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            const int t = row + quad + 8 * r;
            if (t >= ch.z) continue;
            float* at = a.o + ((size_t)(ch.y + t) * a.heads + h) * a.o_ld + c0;
#pragma unroll
            for (int n = 0; n < 4; ++n)
                if (c0 + n * 8 + pair < a.vdim) *reinterpret_cast<float2*>(at + n * 8 + pair) = make_float2(qs[n][2 * r], qs[n][2 * r + 1]);
        }
        // the state after the chunk
        const float keep = st.f[3 * kC];
#pragma unroll
        for (int n = 0; n < NT; ++n)
#pragma unroll
            for (int x = 0; x < 4; ++x) acc[n][x] *= keep;
#pragma unroll
        for (int k = 0; k < kC / 16; ++k) {
            uint32_t hi[4], lo[4], bb[4];
            ldsm4t(hi, at_a_t(&sh.w[0][0][0], kCld, cw, k * 16));
            ldsm4t(lo, at_a_t(&sh.w[1][0][0], kCld, cw, k * 16));
#pragma unroll
            for (int n = 0; n < NT / 2; ++n) {
                ldsm4t(bb, at_b_kn(&st.k[0][0], D + 8, iw + n * 16, k * 16));
                mma(acc[2 * n], hi, bb[0], bb[1]);
                mma(acc[2 * n + 1], hi, bb[2], bb[3]);
                mma(acc[2 * n], lo, bb[0], bb[1]);
                mma(acc[2 * n + 1], lo, bb[2], bb[3]);
            }
        }
        if (j + 1 < n_chunks) spill();         // (all reads of the halves ended two barriers ago)
        __syncthreads();
    }
    if (!a.write) return;
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            const int c = c0 + cw + quad + 8 * r;
            if (c < a.vdim) *reinterpret_cast<float2*>(S + (size_t)c * D + iw + n * 8 + pair) = make_float2(acc[n][2 * r], acc[n][2 * r + 1]);
        }
}

template <int D> int run_delta_walk(const DeltaArgs& a, int n_longs, cudaStream_t stream) {
    const size_t smem = sizeof(DeltaShared<D>);
    cudaError_t e = cudaFuncSetAttribute(delta_walk_kernel<D>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) LLM_FAIL(-2, "delta_chunk_walk: %s", cudaGetErrorString(e));
    llm_launch(delta_walk_kernel<D>, dim3((unsigned)((a.vdim + kCols - 1) / kCols), (unsigned)a.heads, (unsigned)n_longs), kThreads, smem,
               stream, a);
    LLM_CHECK_LAUNCH("delta_chunk_walk");
    return 0;
}

}  // namespace

LLM_API int llm_state_chunk_tokens() { return kC; }
// Which head sizes the chunked kernels take (rows of 16-byte pieces; what fits shared memory).
LLM_API int llm_memory_chunk_supported(int dim, int vdim) { return dim % 16 == 0 && dim > 0 && dim <= 256 && vdim % 8 == 0 && vdim > 0; }
LLM_API int llm_delta_chunk_supported(int dim, int vdim) { return dim % 32 == 0 && dim > 0 && dim <= 128 && vdim % 8 == 0 && vdim > 0; }
LLM_API int llm_delta_chunk_tri_numbers() { return kTri; }
LLM_API int llm_delta_chunk_factor_numbers() { return kFactors; }

// proj [tokens, ld] bfloat16: q, k, v ...; gates of llm_memory_gates; chunks [n_chunks, 4] and longs [n_longs, 3] int32.  own float32
// [n_chunks, heads, vdim + 1, dim], start_hi / start_lo bfloat16 of the same shape, decay float32 [n_chunks, heads].
LLM_API int llm_memory_chunks(const void* proj, int ld, const void* gates, const int* chunks, int n_chunks, const int* longs, int n_longs,
                              float* own, void* start_hi, void* start_lo, float* decay, float* state, long long slot_stride,
                              const int* state_slots, float* o, int o_ld, int heads, int dim, int vdim, float q_scale, int write,
                              cudaStream_t stream) {
    if (n_chunks == 0) return 0;
    if (!llm_memory_chunk_supported(dim, vdim) || ld % 8 || ((uintptr_t)proj & 15) || o_ld % 2)
        LLM_FAIL(-1, "memory_chunks: head sizes %d / %d or rows of %d numbers do not fit", dim, vdim, ld);
    MemoryArgs a{(const bf16*)proj, ld, (const float4*)gates, (const int4*)chunks, own, decay, (bf16*)start_hi, (bf16*)start_lo, o, heads, dim,
                 vdim, o_ld, q_scale};
    const dim3 grid((unsigned)n_chunks, (unsigned)heads, (unsigned)((vdim + 63) / 64));
    const size_t gather = sizeof(bf16) * kC * (72 + 2 * (size_t)(dim + 8)), outs = sizeof(bf16) * kC * (72 + 4 * (size_t)(dim + 8));
    cudaFuncSetAttribute(memory_gather_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)gather);
    cudaFuncSetAttribute(memory_out_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)outs);
    llm_launch(memory_gather_kernel, grid, kThreads, gather, stream, a);
    LLM_CHECK_LAUNCH("memory_chunk_gather");
    const long long quads = (long long)heads * (vdim + 1) * dim / 4;
    llm_launch(memory_scan_kernel, dim3((unsigned)((quads + 255) / 256), (unsigned)n_longs), 256, 0, stream, (const float*)own,
               (const float*)decay, (bf16*)start_hi, (bf16*)start_lo, longs, state, slot_stride, state_slots, heads, (vdim + 1) * dim, write);
    LLM_CHECK_LAUNCH("memory_chunk_scan");
    llm_launch(memory_out_kernel, grid, kThreads, outs, stream, a);
    LLM_CHECK_LAUNCH("memory_chunk_out");
    return 0;
}

// qkv [tokens, channels] bfloat16 as llm_delta_prepare leaves it.  tri bfloat16 [n_chunks, heads, llm_delta_chunk_tri_numbers()],
// factors float32 [n_chunks, heads, llm_delta_chunk_factor_numbers()].
LLM_API int llm_delta_chunks(const void* qkv, int channels, const void* unit, const void* steps, const int* chunks, int n_chunks,
                             const int* longs, int n_longs, void* tri, float* factors, float* state, long long slot_stride,
                             const int* state_slots, float* o, int o_ld, int heads, int kv_heads, int dim, int vdim, int write,
                             cudaStream_t stream) {
    if (n_chunks == 0) return 0;
    if (!llm_delta_chunk_supported(dim, vdim) || channels % 8 || ((uintptr_t)qkv & 15) || o_ld % 2)
        LLM_FAIL(-1, "delta_chunks: head sizes %d / %d or rows of %d numbers do not fit", dim, vdim, channels);
    DeltaArgs a{(const bf16*)qkv, channels, (const float2*)unit, (const float2*)steps, (const int4*)chunks, longs, (bf16*)tri, factors, state,
                slot_stride, state_slots, o, heads, kv_heads, dim, vdim, o_ld, write};
    const size_t smem = sizeof(bf16) * 2 * kC * (size_t)(dim + 8) + sizeof(float) * (2 * kC * (kC + 1) + 3 * 16 * 17);
    cudaFuncSetAttribute(delta_tri_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    llm_launch(delta_tri_kernel, dim3((unsigned)n_chunks, (unsigned)heads), kThreads, smem, stream, a);
    LLM_CHECK_LAUNCH("delta_chunk_tri");
    switch (dim) {
        case 32: return run_delta_walk<32>(a, n_longs, stream);
        case 64: return run_delta_walk<64>(a, n_longs, stream);
        case 96: return run_delta_walk<96>(a, n_longs, stream);
        default: return run_delta_walk<128>(a, n_longs, stream);
    }
}

LLM_TRACE_EXPORT(matrix_state_mma)
