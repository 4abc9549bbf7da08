// Recurrent mixers with a matrix state per head (see matrix_state.cuh): a matrix memory with exponential gates and a normaliser, and a
// gated delta rule behind short convolutions.  All state arithmetic is float32.
//
// llm_matrix_memory_step / llm_gated_delta_step:  steps of single tokens, everything between the projections and the output product in
//                   one launch: gates, (delta: convolution, silu, unit norms,) the state's update and read-out, head norm, gain, gate.
//                   A block owns a head of a request, or a cluster of up to eight blocks shares it by columns and exchanges the head
//                   norm's sums of squares.  A block asks for its first columns before it waits for the kernel ahead of it: a
//                   state slot is written by this layer's kernels alone, in an earlier step.
// llm_memory_gates: the gates of every token and the running maximum m along each request, a block per request and head: m_t =
//                   max(f_t + m_(t-1), i_t) is scanned with the pairs (sum of f, maximum), 256 tokens at a time.
// llm_delta_prepare: convolution, silu, unit lengths, decays and step sizes of every token; the convolution's rows it leaves behind
//                   (llm_delta_rows) are written by a launch of their own, since other blocks of this one still read them.
// llm_state_walk:   portions of prompts token by token: a block owns some columns of a head of a request in registers, a column's rows
//                   shared out over `ds` lanes, and walks the tokens in order; sixteen tokens' rows are staged in shared memory at a
//                   time.  Works for all sizes and types; long portions in bfloat16 take the chunked kernels of matrix_state_mma.cu.
// llm_state_finish: head norm, gain and gate of what walk or chunks left, a warp per token and head.
#include "matrix_state.cuh"

namespace {

typedef __nv_bfloat16 bf16;
constexpr int kStage = 16;             // tokens whose rows the walk stages at a time

struct StepArgs {
    const void* proj;                  // [requests' tokens, ld]: q, k, v and the output gate's input z
    int ld;
    const float* gates;                // [tokens, 2 * heads]: memory: i, f;  delta: b, a
    const float* p0;                   // memory: gate bias [2 * heads];  delta: convolution [channels, taps]
    const float* p1;                   // delta: exp(A_log) [heads]
    const float* p2;                   // delta: dt_bias [heads]
    const float* gain;                 // memory: [heads * vdim];  delta: [vdim]
    float* state;
    long long slot_stride;
    const int* state_slots;
    const int* positions;              // delta
    const int* cu_seqlens;
    void* out;                         // [tokens, heads * vdim]
    int heads, kv_heads, dim, vdim, taps, write, slices, ds;
    float cap, eps, tiny, q_scale;
};

__device__ __forceinline__ float4 fma4(float a, float4 x, float4 y) {
    return make_float4(fmaf(a, x.x, y.x), fmaf(a, x.y, y.y), fmaf(a, x.z, y.z), fmaf(a, x.w, y.w));
}
__device__ __forceinline__ float4 mul4(float a, float4 x) { return make_float4(a * x.x, a * x.y, a * x.z, a * x.w); }
__device__ __forceinline__ float dot4(float4 a, float4 b, float acc) {
    return fmaf(a.w, b.w, fmaf(a.z, b.z, fmaf(a.y, b.y, fmaf(a.x, b.x, acc))));
}
__device__ __forceinline__ float lanes_sum(float v, int ds) {
    for (int o = ds >> 1; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}

// Sums of three numbers over a block (a multiple of 32 threads), in an order that depends on blockDim alone.
__device__ __forceinline__ float3 block_sum3(float a, float b, float c, float* scratch /* >= 96 floats */) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarp = blockDim.x >> 5;
    a = warp_sum(a); b = warp_sum(b); c = warp_sum(c);
    __syncthreads();
    if (lane == 0) { scratch[warp] = a; scratch[32 + warp] = b; scratch[64 + warp] = c; }
    __syncthreads();
    return make_float3(warp_sum(lane < nwarp ? scratch[lane] : 0.f), warp_sum(lane < nwarp ? scratch[32 + lane] : 0.f),
                       warp_sum(lane < nwarp ? scratch[64 + lane] : 0.f));
}

template <typename T, int KIND, int PIECES, int COLS>
__global__ void __launch_bounds__(512)
state_step_kernel(StepArgs a) {
    pdl_trigger();
    extern __shared__ __align__(16) float sm[];
    __shared__ float red[96];
    __shared__ float all_ss[8];
    const int dp = state_dp(a.dim), dpad = a.ds * 4 * PIECES;          // a column's lanes cover dpad >= dp rows
    const int rank = a.slices > 1 ? (int)llm_cluster_rank() : 0;
    const int b = blockIdx.x / a.slices, h = blockIdx.y;
    const int per = (a.vdim + a.slices - 1) / a.slices;
    const int c_lo = min(a.vdim, rank * per), c_hi = min(a.vdim, c_lo + per), mine = c_hi - c_lo;
    float* sq = sm;                    // [dpad]
    float* sk = sq + dpad;             // [dpad]
    float* sv = sk + dpad;             // [per]
    float* so = sv + per;              // [per]
    const int columns = KIND == kMemory ? a.vdim + 1 : a.vdim;
    const int groups = blockDim.x / a.ds, s = threadIdx.x % a.ds, cg = threadIdx.x / a.ds;
    const int t = a.cu_seqlens[b];     // (index arrays were in place before the step's first kernel)
    float* rec = a.state + (size_t)a.state_slots[b] * a.slot_stride;
    float* S = rec + (size_t)h * columns * dp;
    float4 reg[COLS][PIECES];
    auto fetch = [&](int cb) {
#pragma unroll
        for (int j = 0; j < COLS; ++j) {
            const int c = c_lo + cb + j * groups + cg;
#pragma unroll
            for (int r = 0; r < PIECES; ++r) {
                const int i = 4 * (s + a.ds * r);
                reg[j][r] = c < c_hi && i < dp ? *reinterpret_cast<const float4*>(S + (size_t)c * dp + i) : make_float4(0.f, 0.f, 0.f, 0.f);
            }
        }
    };
    fetch(0);
    float keep, den = 1.f, beta = 0.f, kq = 0.f, n_new = 0.f, m_new = 0.f;
    float* n_col = S + (size_t)a.vdim * dp;                            // memory: the normaliser, a number a thread and step
    float* m_at = rec + (size_t)a.heads * columns * dp + h;
    const bool one_n = a.dim <= (int)blockDim.x;
    float n_old = 0.f, m_old = 0.f;
    if (KIND == kMemory) {
        if (one_n && (int)threadIdx.x < a.dim) n_old = n_col[threadIdx.x];
        m_old = *m_at;
    }
    pdl_wait();
    const T* row = static_cast<const T*>(a.proj) + (size_t)t * a.ld;
    const float* gates = a.gates + (size_t)t * 2 * a.heads;
    for (int i = threadIdx.x; i < dpad; i += blockDim.x)
        if (i >= a.dim) { sq[i] = 0.f; sk[i] = 0.f; }
    int z_col;
    if (KIND == kMemory) {
        const int qk = a.heads * a.dim;
        z_col = 2 * qk + a.heads * a.vdim + h * a.vdim;
        const float2 g = memory_gates(gates, a.p0, a.heads, h, a.cap);
        m_new = fmaxf(g.x + m_old, g.y);
        keep = expf(g.x + m_old - m_new);
        const float add = expf(g.y - m_new);
        for (int i = threadIdx.x; i < a.dim; i += blockDim.x) {
            sq[i] = to_f32(row[h * a.dim + i]) * a.q_scale;
            sk[i] = to_f32(row[qk + h * a.dim + i]) * add;
        }
        for (int c = threadIdx.x; c < mine; c += blockDim.x) sv[c] = to_f32(row[2 * qk + h * a.vdim + c_lo + c]);
        __syncthreads();
        float nq = 0.f;
        if (one_n) {
            if ((int)threadIdx.x < a.dim) { n_new = fmaf(keep, n_old, sk[threadIdx.x]); nq = n_new * sq[threadIdx.x]; }
        } else {
            for (int i = threadIdx.x; i < a.dim; i += blockDim.x) nq = fmaf(fmaf(keep, n_col[i], sk[i]), sq[i], nq);
        }
        nq = block_sum(nq, red);
        den = 1.0f / (fmaxf(fabsf(nq), expf(-m_new)) + a.tiny);
    } else {
        const int per_head = a.heads / a.kv_heads, g = h / per_head, qk = a.kv_heads * a.dim, channels = 2 * qk + a.heads * a.vdim;
        z_col = channels + h * a.vdim;
        float* ring = rec + (size_t)a.heads * columns * dp;
        const int p = a.positions[t], now = p % a.taps;
        const bool writes_qk = a.write && h == g * per_head && rank == 0;
        float ssq = 0.f, ssk = 0.f;
        for (int x = threadIdx.x; x < 2 * a.dim + mine; x += blockDim.x) {
            const int which = x < a.dim ? 0 : x < 2 * a.dim ? 1 : 2;
            const int c = which == 2 ? 2 * qk + h * a.vdim + c_lo + x - 2 * a.dim : which * qk + g * a.dim + x - which * a.dim;
            const float u = to_f32(row[c]);
            const float* w = a.p0 + (size_t)c * a.taps;
            float acc = 0.f;
            for (int j = 0; j < a.taps - 1; ++j) acc = fmaf(w[j], ring[(size_t)((p + 1 + j) % a.taps) * channels + c], acc);
            acc = fmaf(w[a.taps - 1], u, acc);
            if (which == 2 ? a.write : writes_qk) ring[(size_t)now * channels + c] = u;      // a row that this step reads nowhere
            const float y = acc * sigmoid_f(acc);
            if (which == 0) { sq[x] = y; ssq = fmaf(y, y, ssq); }
            else if (which == 1) { sk[x - a.dim] = y; ssk = fmaf(y, y, ssk); }
            else sv[x - 2 * a.dim] = y;
        }
        __syncthreads();
        float qk_dot = 0.f;
        for (int i = threadIdx.x; i < a.dim; i += blockDim.x) qk_dot = fmaf(sq[i], sk[i], qk_dot);
        const float3 sums = block_sum3(ssq, ssk, qk_dot, red);
        const float rq = a.q_scale / sqrtf(sums.x + a.tiny), rk = 1.0f / sqrtf(sums.y + a.tiny);
        kq = sums.z * rq * rk;
        for (int i = threadIdx.x; i < a.dim; i += blockDim.x) { sq[i] *= rq; sk[i] *= rk; }
        beta = sigmoid_f(gates[h]);
        keep = expf(-a.p1[h] * soft_plus(gates[a.heads + h] + a.p2[h]));
        __syncthreads();
    }
    float4 q4[PIECES], k4[PIECES];
#pragma unroll
    for (int r = 0; r < PIECES; ++r) {
        const int i = 4 * (s + a.ds * r);
        q4[r] = *reinterpret_cast<const float4*>(sq + i);
        k4[r] = *reinterpret_cast<const float4*>(sk + i);
    }
    for (int cb = 0; cb < mine; cb += groups * COLS) {
        if (cb) fetch(cb);
#pragma unroll
        for (int j = 0; j < COLS; ++j) {
            const int at = cb + j * groups + cg;
            const float v = at < mine ? sv[at] : 0.f;
            float o = 0.f, u = v;
            if (KIND == kDelta) {
                float pk = 0.f;
#pragma unroll
                for (int r = 0; r < PIECES; ++r) { pk = dot4(reg[j][r], k4[r], pk); o = dot4(reg[j][r], q4[r], o); }
                pk = lanes_sum(pk, a.ds);
                o = lanes_sum(o, a.ds);
                u = beta * (v - keep * pk);
                o = fmaf(keep, o, kq * u);
#pragma unroll
                for (int r = 0; r < PIECES; ++r) reg[j][r] = fma4(u, k4[r], mul4(keep, reg[j][r]));
            } else {
#pragma unroll
                for (int r = 0; r < PIECES; ++r) {
                    reg[j][r] = fma4(v, k4[r], mul4(keep, reg[j][r]));
                    o = dot4(reg[j][r], q4[r], o);
                }
                o = lanes_sum(o, a.ds) * den;
            }
            if (at < mine) {
                if (s == 0) so[at] = o;
                if (a.write) {
#pragma unroll
                    for (int r = 0; r < PIECES; ++r) {
                        const int i = 4 * (s + a.ds * r);
                        if (i < dp) *reinterpret_cast<float4*>(S + (size_t)(c_lo + at) * dp + i) = reg[j][r];
                    }
                }
            }
        }
    }
    __syncthreads();
    float ss = 0.f;
    for (int c = threadIdx.x; c < mine; c += blockDim.x) ss = fmaf(so[c], so[c], ss);
    ss = block_sum(ss, red);
    if (a.slices > 1) {
        if ((int)threadIdx.x < a.slices) llm_cluster_write(&all_ss[rank], (uint32_t)threadIdx.x, ss);
        llm_cluster_sync();            // all sums are everywhere; every block has read n and m
        ss = 0.f;
#pragma unroll
        for (int k = 0; k < 8; ++k)
            if (k < a.slices) ss += all_ss[k];
    }
    if (KIND == kMemory && a.write && rank == 0) {
        if (one_n) {
            if ((int)threadIdx.x < a.dim) n_col[threadIdx.x] = n_new;
        } else {
            for (int i = threadIdx.x; i < a.dim; i += blockDim.x) n_col[i] = fmaf(keep, n_col[i], sk[i]);
        }
        if (threadIdx.x == 0) *m_at = m_new;
    }
    const float inv = 1.0f / sqrtf(ss / (float)a.vdim + a.eps);
    T* out = static_cast<T*>(a.out) + (size_t)t * a.heads * a.vdim + (size_t)h * a.vdim;
    for (int c = threadIdx.x; c < mine; c += blockDim.x) {
        const float z = to_f32(row[z_col + c_lo + c]), sg = sigmoid_f(z);
        out[c_lo + c] = from_f32<T>(so[c] * inv * a.gain[(KIND == kMemory ? h * a.vdim : 0) + c_lo + c] * (KIND == kMemory ? sg : z * sg));
    }
}

// gates of the step's tokens [tokens, heads] as (f, i, m, m of the token before); a block per request and head
constexpr int kGateThreads = 256;
__global__ void __launch_bounds__(kGateThreads)
memory_gates_kernel(const float* __restrict__ gates, const float* __restrict__ bias, float cap, float* __restrict__ state,
                    long long slot_stride, long long m_offset, const int* __restrict__ state_slots, const int* __restrict__ cu_seqlens,
                    float4* __restrict__ out, int heads, int write) {
    pdl_trigger();
    pdl_wait();
    __shared__ float2 part[2][kGateThreads / 32];          // two buffers in turn: one barrier a round
    const int b = blockIdx.x, h = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int lo = cu_seqlens[b], hi = cu_seqlens[b + 1];
    if (hi <= lo) return;
    float* m_at = state + (size_t)state_slots[b] * slot_stride + m_offset + h;
    float m0 = *m_at;
    auto load = [&](int t) {
        return t < hi ? memory_gates(gates + (size_t)t * 2 * heads, bias, heads, h, cap) : make_float2(0.f, -INFINITY);
    };
    float2 next = load(lo + threadIdx.x);
    int turn = 0;
    for (int t0 = lo; t0 < hi; t0 += kGateThreads, turn ^= 1) {
        const float2 g = next;
        if (t0 + kGateThreads < hi) next = load(t0 + kGateThreads + threadIdx.x);
        // (F, A): the warp's tokens up to this one turn m into max(F + m, A)
        float F = g.x, A = g.y;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float Fb = __shfl_up_sync(0xffffffffu, F, o), Ab = __shfl_up_sync(0xffffffffu, A, o);
            if (lane >= o) { A = fmaxf(Ab + F, A); F += Fb; }
        }
        if (lane == 31) part[turn][warp] = make_float2(F, A);
        __syncthreads();
        float start = m0;
#pragma unroll
        for (int w = 0; w < kGateThreads / 32; ++w) {
            if (w == warp) start = m0;
            m0 = fmaxf(part[turn][w].x + m0, part[turn][w].y);       // behind the last token nothing changes m
        }
        const float m = fmaxf(F + start, A);
        float before = __shfl_up_sync(0xffffffffu, m, 1);
        if (lane == 0) before = start;
        const int t = t0 + threadIdx.x;
        // the token's own m beside the m before it: the pair every consumer takes its weights from
        if (t < hi) out[(size_t)t * heads + h] = make_float4(g.x, g.y, m, before);
    }
    if (write && threadIdx.x == 0) *m_at = m0;
}

// c [tokens, channels] = silu(convolution) as the engine's type; unit [tokens, kv_heads] = factors that make q (times q_scale) and k unit
// vectors; steps [tokens, heads] = (log decay, beta).  One block a token.
template <typename T>
__global__ void __launch_bounds__(256)
delta_prepare_kernel(const T* __restrict__ proj, int ld, const float* __restrict__ gates, const float* __restrict__ conv,
                     const float* __restrict__ rate, const float* __restrict__ dt_bias, const float* __restrict__ state,
                     long long slot_stride, long long ring_offset, const int* __restrict__ state_slots, const int* __restrict__ positions,
                     const int* __restrict__ token_request, const int* __restrict__ cu_seqlens, T* __restrict__ c_out,
                     float2* __restrict__ unit, float2* __restrict__ steps, int heads, int kv_heads, int dim, int vdim, int taps, float tiny,
                     float q_scale) {
    pdl_trigger();
    pdl_wait();
    extern __shared__ float y[];           // q and k channels
    const int t = blockIdx.x, b = token_request[t], local = t - cu_seqlens[b], p = positions[t];
    const int qk = kv_heads * dim, channels = 2 * qk + heads * vdim;
    const float* ring = state + (size_t)state_slots[b] * slot_stride + ring_offset;
    for (int c = threadIdx.x; c < channels; c += blockDim.x) {
        const float* w = conv + (size_t)c * taps;
        float acc = 0.f;
        for (int j = 0; j < taps; ++j) {
            const int back = taps - 1 - j;
            const float u = back <= local ? to_f32(proj[(size_t)(t - back) * ld + c]) : ring[(size_t)((p + 1 + j) % taps) * channels + c];
            acc = fmaf(w[j], u, acc);
        }
        const T r = from_f32<T>(acc * sigmoid_f(acc));
        c_out[(size_t)t * channels + c] = r;
        if (c < 2 * qk) y[c] = to_f32(r);
    }
    for (int h = threadIdx.x; h < heads; h += blockDim.x) {
        const float* g = gates + (size_t)t * 2 * heads;
        steps[(size_t)t * heads + h] = make_float2(-rate[h] * soft_plus(g[heads + h] + dt_bias[h]), sigmoid_f(g[h]));
    }
    __syncthreads();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nwarp = blockDim.x >> 5;
    for (int g = warp; g < kv_heads; g += nwarp) {
        float ssq = 0.f, ssk = 0.f;
        for (int i = lane; i < dim; i += 32) {
            const float q = y[g * dim + i], k = y[qk + g * dim + i];
            ssq = fmaf(q, q, ssq);
            ssk = fmaf(k, k, ssk);
        }
        ssq = warp_sum(ssq);
        ssk = warp_sum(ssk);
        if (lane == 0) unit[(size_t)t * kv_heads + g] = make_float2(q_scale / sqrtf(ssq + tiny), 1.0f / sqrtf(ssk + tiny));
    }
}

// The same for two channels a lane and taps known when compiling: a warp takes a run of tokens and one head of q, of k or of v (or, last,
// the decays and step sizes of all heads), and the rows a run's convolutions share are read once.
constexpr int kRun = 8;
template <typename T> __device__ __forceinline__ float2 pair_of(const T* p);
template <> __device__ __forceinline__ float2 pair_of<float>(const float* p) { return *reinterpret_cast<const float2*>(p); }
template <> __device__ __forceinline__ float2 pair_of<bf16>(const bf16* p) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p)); }
__device__ __forceinline__ float2 round_pair(float* p, float a, float b) {
    *reinterpret_cast<float2*>(p) = make_float2(a, b);
    return make_float2(a, b);
}
__device__ __forceinline__ float2 round_pair(bf16* p, float a, float b) {
    const __nv_bfloat162 v = __floats2bfloat162_rn(a, b);
    *reinterpret_cast<__nv_bfloat162*>(p) = v;
    return __bfloat1622float2(v);
}

template <typename T, int TAPS>
__global__ void __launch_bounds__(128, 8)
delta_prepare_run_kernel(const T* __restrict__ proj, int ld, const float* __restrict__ gates, const float* __restrict__ conv,
                         const float* __restrict__ rate, const float* __restrict__ dt_bias, const float* __restrict__ state,
                         long long slot_stride, long long ring_offset, const int* __restrict__ state_slots, const int* __restrict__ positions,
                         const int* __restrict__ token_request, const int* __restrict__ cu_seqlens, T* __restrict__ c_out,
                         float2* __restrict__ unit, float2* __restrict__ steps, int tokens, int heads, int kv_heads, int dim, int vdim,
                         float tiny, float q_scale) {
    pdl_trigger();
    pdl_wait();
    const int t0 = blockIdx.x * kRun, n = min(kRun, tokens - t0), lane = threadIdx.x & 31;
    const int u = blockIdx.y * 4 + (threadIdx.x >> 5);
    const int qk = kv_heads * dim, channels = 2 * qk + heads * vdim;
    if (u > 2 * kv_heads + heads) return;
    if (u == 2 * kv_heads + heads) {
        for (int x = lane; x < n * heads; x += 32) {
            const int h = x % heads;
            const float* g = gates + (size_t)(t0 + x / heads) * 2 * heads;
            steps[(size_t)t0 * heads + x] = make_float2(-rate[h] * soft_plus(g[heads + h] + dt_bias[h]), sigmoid_f(g[h]));
        }
        return;
    }
    const bool is_v = u >= 2 * kv_heads;
    const int c0 = is_v ? 2 * qk + (u - 2 * kv_heads) * vdim : u * dim, width = is_v ? vdim : dim;
    float ss[kRun];
#pragma unroll
    for (int r = 0; r < kRun; ++r) ss[r] = 0.f;
    for (int i = 2 * lane; i < width; i += 64) {
        const int c = c0 + i;
        float w[2 * TAPS];             // both channels' taps lie side by side
#pragma unroll
        for (int j = 0; j < TAPS; ++j) {
            const float2 v = *reinterpret_cast<const float2*>(conv + (size_t)c * TAPS + 2 * j);
            w[2 * j] = v.x;
            w[2 * j + 1] = v.y;
        }
        float2 x[kRun];
#pragma unroll
        for (int r = 0; r < kRun; ++r)
            if (r < n) x[r] = pair_of(proj + (size_t)(t0 + r) * ld + c);
        float2 win[TAPS];              // the inputs of the current token's convolution, the oldest first
        int b = -1;
#pragma unroll
        for (int r = 0; r < kRun; ++r) {
            if (r >= n) continue;
            const int t = t0 + r;
            if (r == 0 || token_request[t] != b) {         // the run's start, or a request's first token of the step
                b = token_request[t];
                const int local = t - cu_seqlens[b], p = positions[t];
                const float* ring = state + (size_t)state_slots[b] * slot_stride + ring_offset;
#pragma unroll
                for (int j = 0; j < TAPS - 1; ++j) {
                    const int back = TAPS - 1 - j;
                    win[j + 1] = back <= local ? pair_of(proj + (size_t)(t - back) * ld + c)
                                               : make_float2(ring[(size_t)((p + 1 + j) % TAPS) * channels + c], ring[(size_t)((p + 1 + j) % TAPS) * channels + c + 1]);
                }
            }
#pragma unroll
            for (int j = 0; j < TAPS - 1; ++j) win[j] = win[j + 1];
            win[TAPS - 1] = x[r];
            float a0 = 0.f, a1 = 0.f;
#pragma unroll
            for (int j = 0; j < TAPS; ++j) { a0 = fmaf(w[j], win[j].x, a0); a1 = fmaf(w[TAPS + j], win[j].y, a1); }
            const float2 y = round_pair(c_out + (size_t)t * channels + c, a0 * sigmoid_f(a0), a1 * sigmoid_f(a1));
            ss[r] = fmaf(y.x, y.x, fmaf(y.y, y.y, ss[r]));
        }
    }
    if (is_v) return;
#pragma unroll
    for (int r = 0; r < kRun; ++r) {
        const float sum = warp_sum(ss[r]);
        if (lane != 0 || r >= n) continue;
        float* at = reinterpret_cast<float*>(unit + (size_t)(t0 + r) * kv_heads + u % kv_heads);
        at[u / kv_heads] = (u < kv_heads ? q_scale : 1.0f) / sqrtf(sum + tiny);
    }
}

// the last `taps` projected rows of every request into its record (row p % taps for position p)
template <typename T>
__global__ void __launch_bounds__(256)
delta_rows_kernel(const T* __restrict__ proj, int ld, float* __restrict__ state, long long slot_stride, long long ring_offset,
                  const int* __restrict__ state_slots, const int* __restrict__ positions, const int* __restrict__ cu_seqlens, int channels,
                  int taps) {
    pdl_trigger();
    pdl_wait();
    const int b = blockIdx.x, hi = cu_seqlens[b + 1], lo = max(cu_seqlens[b], hi - taps);
    float* ring = state + (size_t)state_slots[b] * slot_stride + ring_offset;
    for (int t = lo; t < hi; ++t) {
        const int r = positions[t] % taps;
        for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < channels; c += gridDim.y * blockDim.x)
            ring[(size_t)r * channels + c] = to_f32(proj[(size_t)t * ld + c]);
    }
}

struct WalkArgs {
    const void* qkv;                   // rows of q, k, v (memory: the projection; delta: what the convolution left)
    int ld;
    const float4* gates;               // memory: (f, i, m, m before) [tokens, heads]
    const float2* unit;                // delta: [tokens, kv_heads]
    const float2* steps;               // delta: (log decay, beta) [tokens, heads]
    float* state;
    long long slot_stride;
    const int* state_slots;
    const int* cu_seqlens;
    const int* walks;                  // requests to walk (null: all)
    float* o;                          // [tokens, heads, o_ld]
    int heads, kv_heads, dim, vdim, o_ld, write, ds;
    float q_scale;
};

template <typename T, int KIND, int PIECES, int COLS>
__global__ void __launch_bounds__(128)
state_walk_kernel(WalkArgs a) {
    pdl_trigger();
    pdl_wait();
    extern __shared__ __align__(16) float sm[];
    const int dp = state_dp(a.dim), dpad = a.ds * 4 * PIECES;
    const int b = a.walks ? a.walks[blockIdx.z] : blockIdx.z, h = blockIdx.y;
    const int lo = a.cu_seqlens[b], hi = a.cu_seqlens[b + 1];
    if (hi <= lo) return;
    const int columns = KIND == kMemory ? a.vdim + 1 : a.vdim;
    const int groups = 128 / a.ds, s = threadIdx.x % a.ds, cg = threadIdx.x / a.ds;
    const int cpb = groups * COLS, c0 = blockIdx.x * cpb;
    float* sq = sm;                            // [kStage][dpad]
    float* sk = sq + kStage * dpad;            // [kStage][dpad]
    float* sv = sk + kStage * dpad;            // [kStage][cpb]
    float* s_keep = sv + kStage * cpb;         // [kStage] x 3
    float* s_beta = s_keep + kStage;
    float* s_kq = s_beta + kStage;
    float* S = a.state + (size_t)a.state_slots[b] * a.slot_stride + (size_t)h * columns * dp;
    const int g = KIND == kDelta ? h / (a.heads / a.kv_heads) : h;
    const int qk = a.kv_heads * a.dim;
    float4 reg[COLS][PIECES];
#pragma unroll
    for (int j = 0; j < COLS; ++j) {
        const int c = c0 + j * groups + cg;
#pragma unroll
        for (int r = 0; r < PIECES; ++r) {
            const int i = 4 * (s + a.ds * r);
            reg[j][r] = c < columns && i < dp ? *reinterpret_cast<const float4*>(S + (size_t)c * dp + i) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
    }
    const T* rows = static_cast<const T*>(a.qkv);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    for (int t0 = lo; t0 < hi; t0 += kStage) {
        const int nb = min(kStage, hi - t0);
        __syncthreads();
        for (int tt = warp; tt < nb; tt += 4) {            // a warp brings a token's rows
            const T* row = rows + (size_t)(t0 + tt) * a.ld;
            float fq = a.q_scale, fk, keep, kq = 0.f;
            if (KIND == kMemory) {
                const float4 gt = a.gates[(size_t)(t0 + tt) * a.heads + h];
                keep = expf(gt.x + gt.w - gt.z);
                fk = expf(gt.y - gt.z);
            } else {
                const float2 st = a.steps[(size_t)(t0 + tt) * a.heads + h], un = a.unit[(size_t)(t0 + tt) * a.kv_heads + g];
                keep = expf(st.x);
                fq = un.x;
                fk = un.y;
                if (lane == 0) s_beta[tt] = st.y;
            }
            for (int i = lane; i < dpad; i += 32) {
                const float q = i < a.dim ? to_f32(row[g * a.dim + i]) * fq : 0.f, k = i < a.dim ? to_f32(row[qk + g * a.dim + i]) * fk : 0.f;
                sq[tt * dpad + i] = q;
                sk[tt * dpad + i] = k;
                kq = fmaf(q, k, kq);
            }
            if (KIND == kDelta) kq = warp_sum(kq);
            if (lane == 0) { s_keep[tt] = keep; s_kq[tt] = kq; }
            for (int c = lane; c < cpb; c += 32)
                sv[tt * cpb + c] = c0 + c < a.vdim ? to_f32(row[2 * qk + h * a.vdim + c0 + c]) : 1.0f;
        }
        __syncthreads();
        for (int tt = 0; tt < nb; ++tt) {
            const float keep = s_keep[tt];
            float4 q4[PIECES], k4[PIECES];
#pragma unroll
            for (int r = 0; r < PIECES; ++r) {
                const int i = tt * dpad + 4 * (s + a.ds * r);
                q4[r] = *reinterpret_cast<const float4*>(sq + i);
                k4[r] = *reinterpret_cast<const float4*>(sk + i);
            }
            float o[COLS], pk[COLS];
#pragma unroll
            for (int j = 0; j < COLS; ++j) {
                const float v = sv[tt * cpb + j * groups + cg];
                o[j] = pk[j] = 0.f;
#pragma unroll
                for (int r = 0; r < PIECES; ++r) {
                    if (KIND == kMemory) reg[j][r] = fma4(v, k4[r], mul4(keep, reg[j][r]));
                    else pk[j] = dot4(reg[j][r], k4[r], pk[j]);
                    o[j] = dot4(reg[j][r], q4[r], o[j]);
                }
            }
            for (int x = a.ds >> 1; x > 0; x >>= 1)
#pragma unroll
                for (int j = 0; j < COLS; ++j) {
                    o[j] += __shfl_xor_sync(0xffffffffu, o[j], x);
                    if (KIND == kDelta) pk[j] += __shfl_xor_sync(0xffffffffu, pk[j], x);
                }
            float* o_at = a.o + ((size_t)(t0 + tt) * a.heads + h) * a.o_ld + c0;
#pragma unroll
            for (int j = 0; j < COLS; ++j) {
                if (KIND == kDelta) {
                    const float u = s_beta[tt] * (sv[tt * cpb + j * groups + cg] - keep * pk[j]);
                    o[j] = fmaf(keep, o[j], s_kq[tt] * u);
#pragma unroll
                    for (int r = 0; r < PIECES; ++r) reg[j][r] = fma4(u, k4[r], mul4(keep, reg[j][r]));
                }
                if (s == 0 && c0 + j * groups + cg < columns) o_at[j * groups + cg] = o[j];
            }
        }
    }
    if (!a.write) return;
#pragma unroll
    for (int j = 0; j < COLS; ++j) {
        const int c = c0 + j * groups + cg;
#pragma unroll
        for (int r = 0; r < PIECES; ++r) {
            const int i = 4 * (s + a.ds * r);
            if (c < columns && i < dp) *reinterpret_cast<float4*>(S + (size_t)c * dp + i) = reg[j][r];
        }
    }
}

// out = (head of o / root mean square) * gain * gate; memory: o is divided by its normaliser first.  A warp per (token, head).
template <typename T, int KIND>
__global__ void __launch_bounds__(256)
state_finish_kernel(const float* __restrict__ o, int o_ld, const float4* __restrict__ gates, const T* __restrict__ proj, int ld, int z_col,
                    const float* __restrict__ gain, T* __restrict__ out, int heads, int vdim, float eps, float tiny, unsigned rows) {
    pdl_trigger();
    pdl_wait();
    const unsigned index = blockIdx.x * 8 + (threadIdx.x >> 5), token = index / (unsigned)heads;      // (the launcher keeps them in 32 bits)
    if (index >= rows) return;
    const int lane = threadIdx.x & 31, h = (int)(index - token * (unsigned)heads);
    const size_t row = index, t = token;
    const float* x = o + row * o_ld;
    float den = 1.f;
    if (KIND == kMemory) den = 1.0f / (fmaxf(fabsf(x[vdim]), expf(-gates[row].z)) + tiny);
    float ss = 0.f;
    for (int c = lane; c < vdim; c += 32) { const float v = x[c] * den; ss = fmaf(v, v, ss); }
    const float inv = den / sqrtf(warp_sum(ss) / (float)vdim + eps);
    const T* z_row = proj + (size_t)t * ld + z_col + h * vdim;
    for (int c = lane; c < vdim; c += 32) {
        const float z = to_f32(z_row[c]), sg = sigmoid_f(z);
        out[(size_t)row * vdim + c] = from_f32<T>(x[c] * inv * gain[KIND == kMemory ? h * vdim + c : c] * (KIND == kMemory ? sg : z * sg));
    }
}

template <typename T> __device__ __forceinline__ float4 four_of(const T* p);
template <> __device__ __forceinline__ float4 four_of<float>(const float* p) { return *reinterpret_cast<const float4*>(p); }
template <> __device__ __forceinline__ float4 four_of<bf16>(const bf16* p) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x)), b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
    return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void put_four(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void put_four(bf16* p, float4 v) {
    __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<uint32_t*>(&a), *reinterpret_cast<uint32_t*>(&b));
}

// The same, four columns a lane and up to 128 * PER columns: everything a lane needs is asked for at once.
template <typename T, int KIND, int PER>
__global__ void __launch_bounds__(256)
state_finish_vec_kernel(const float* __restrict__ o, int o_ld, const float4* __restrict__ gates, const T* __restrict__ proj, int ld, int z_col,
                        const float* __restrict__ gain, T* __restrict__ out, int heads, int vdim, float eps, float tiny, unsigned rows) {
    pdl_trigger();
    pdl_wait();
    const unsigned index = blockIdx.x * 8 + (threadIdx.x >> 5), token = index / (unsigned)heads;      // (the launcher keeps them in 32 bits)
    if (index >= rows) return;
    const int lane = threadIdx.x & 31, h = (int)(index - token * (unsigned)heads);
    const size_t row = index, t = token;
    const float* x = o + row * o_ld;
    const T* z_row = proj + (size_t)t * ld + z_col + h * vdim;
    float4 v[PER], z[PER], g[PER];
    float nq = 0.f, m = 0.f;
    if (KIND == kMemory) { nq = x[vdim]; m = gates[row].z; }
#pragma unroll
    for (int j = 0; j < PER; ++j) {
        const int c = 4 * lane + 128 * j;
        v[j] = z[j] = g[j] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (c < vdim) {
            v[j] = four_of(x + c);
            z[j] = four_of(z_row + c);
            g[j] = four_of(gain + (KIND == kMemory ? h * vdim : 0) + c);
        }
    }
    const float den = KIND == kMemory ? 1.0f / (fmaxf(fabsf(nq), expf(-m)) + tiny) : 1.0f;
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < PER; ++j) {
        v[j] = make_float4(v[j].x * den, v[j].y * den, v[j].z * den, v[j].w * den);
        ss += v[j].x * v[j].x + v[j].y * v[j].y + v[j].z * v[j].z + v[j].w * v[j].w;
    }
    const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)vdim + eps);
    auto gate = [](float y) { const float sg = sigmoid_f(y); return KIND == kMemory ? sg : y * sg; };
#pragma unroll
    for (int j = 0; j < PER; ++j) {
        const int c = 4 * lane + 128 * j;
        if (c < vdim)
            put_four(out + (size_t)row * vdim + c, make_float4(v[j].x * inv * g[j].x * gate(z[j].x), v[j].y * inv * g[j].y * gate(z[j].y),
                                                               v[j].z * inv * g[j].z * gate(z[j].z), v[j].w * inv * g[j].w * gate(z[j].w)));
    }
}

// how a column's rows are shared out: lanes a column, four-number pieces a lane
struct Split { int ds, pieces; };
Split split_rows(int dim) {
    Split x{dim <= 16 ? 4 : 8, 1};
    while (x.pieces < 4 && x.ds * 4 * x.pieces < dim) x.pieces *= 2;
    while (x.ds < 32 && x.ds * 4 * x.pieces < dim) x.ds *= 2;
    if (x.ds * 4 * x.pieces < dim) x.pieces = 8;
    return x;
}

template <int KIND>
int run_step(StepArgs& a, int dtype, int requests, cudaStream_t stream) {
    if (requests == 0) return 0;
    if (a.dim > 1024 || a.dim <= 0 || a.vdim <= 0) LLM_FAIL(-1, "state_step: head sizes %d / %d (1 to 1024 rows)", a.dim, a.vdim);
    const Split sp = split_rows(a.dim);
    a.ds = sp.ds;
    // a head's columns over a cluster while the grid leaves SMs idle
    a.slices = 1;
    while (a.slices < 8 && (long long)requests * a.heads * a.slices * 2 <= 2 * 148 && a.vdim / (a.slices * 2) >= 16) a.slices *= 2;
    const int per = (a.vdim + a.slices - 1) / a.slices;
    return llm_dispatch_dtype(dtype, [&](auto tag) {
        using T = decltype(tag);
        auto go = [&](auto kern, int cols) {
            int threads = (a.ds * ((per + cols - 1) / cols) + 31) / 32 * 32;
            threads = threads < 128 ? 128 : threads > 512 ? 512 : threads;
            const size_t smem = sizeof(float) * (2 * (size_t)a.ds * 4 * sp.pieces + 2 * (size_t)per);
            if (smem > 48 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
            if (a.slices > 1)
                llm_launch_cluster(kern, dim3((unsigned)(requests * a.slices), (unsigned)a.heads), threads, smem, stream, (unsigned)a.slices, a);
            else
                llm_launch(kern, dim3((unsigned)requests, (unsigned)a.heads), threads, smem, stream, a);
        };
        if (sp.pieces == 1) go(state_step_kernel<T, KIND, 1, 4>, 4);
        else if (sp.pieces == 2) go(state_step_kernel<T, KIND, 2, 4>, 4);
        else if (sp.pieces == 4) go(state_step_kernel<T, KIND, 4, 4>, 4);
        else go(state_step_kernel<T, KIND, 8, 2>, 2);
        LLM_CHECK_LAUNCH(KIND == kMemory ? "matrix_memory_step" : "gated_delta_step");
        return 0;
    });
}

template <int KIND>
int run_walk(WalkArgs& a, int dtype, int n_walks, cudaStream_t stream) {
    const Split sp = split_rows(a.dim);
    a.ds = sp.ds;
    const int columns = KIND == kMemory ? a.vdim + 1 : a.vdim;
    return llm_dispatch_dtype(dtype, [&](auto tag) {
        using T = decltype(tag);
        auto go = [&](auto kern, int cols) {
            const int cpb = 128 / a.ds * cols;
            const size_t smem = sizeof(float) * kStage * (2 * (size_t)a.ds * 4 * sp.pieces + cpb + 3);
            if (smem > 48 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
            llm_launch(kern, dim3((unsigned)((columns + cpb - 1) / cpb), (unsigned)a.heads, (unsigned)n_walks), 128, smem, stream, a);
        };
        if (sp.pieces == 1) go(state_walk_kernel<T, KIND, 1, 2>, 2);
        else if (sp.pieces == 2) go(state_walk_kernel<T, KIND, 2, 2>, 2);
        else if (sp.pieces == 4) go(state_walk_kernel<T, KIND, 4, 2>, 2);
        else go(state_walk_kernel<T, KIND, 8, 1>, 1);
        LLM_CHECK_LAUNCH("state_walk");
        return 0;
    });
}

}  // namespace

// proj [requests, ld] (one token a request, q, k, v, z), gates float32 [requests, 2 * heads] (i then f), state float32 records
// `slot_stride` numbers apart.
LLM_API int llm_matrix_memory_step(const void* proj, int ld, const float* gates, const float* gate_bias, float cap, const float* gain,
                                   float eps, float tiny, float* state, long long slot_stride, const int* state_slots,
                                   const int* cu_seqlens, void* out, int dtype, int requests, int heads, int dim, int vdim, float q_scale,
                                   int write, cudaStream_t stream) {
    StepArgs a{proj, ld, gates, gate_bias, nullptr, nullptr, gain, state, slot_stride, state_slots, nullptr, cu_seqlens, out,
               heads, heads, dim, vdim, 1, write, 1, 8, cap, eps, tiny, q_scale};
    return run_step<kMemory>(a, dtype, requests, stream);
}

// gates: b then a; conv float32 [channels, taps]; rate = exp(A_log).
LLM_API int llm_gated_delta_step(const void* proj, int ld, const float* gates, const float* conv, int taps, const float* rate,
                                 const float* dt_bias, const float* gain, float eps, float tiny, float* state, long long slot_stride,
                                 const int* state_slots, const int* positions, const int* cu_seqlens, void* out, int dtype, int requests,
                                 int heads, int kv_heads, int dim, int vdim, float q_scale, int write, cudaStream_t stream) {
    if (taps < 1 || kv_heads < 1 || heads % kv_heads) LLM_FAIL(-1, "gated_delta_step: %d taps, %d heads over %d", taps, heads, kv_heads);
    StepArgs a{proj, ld, gates, conv, rate, dt_bias, gain, state, slot_stride, state_slots, positions, cu_seqlens, out,
               heads, kv_heads, dim, vdim, taps, write, 1, 8, 1.f, eps, tiny, q_scale};
    return run_step<kDelta>(a, dtype, requests, stream);
}

LLM_API int llm_memory_gates(const float* gates, const float* bias, float cap, float* state, long long slot_stride, long long m_offset,
                             const int* state_slots, const int* cu_seqlens, void* out, int requests, int heads, int write, cudaStream_t stream) {
    if (requests == 0) return 0;
    llm_launch(memory_gates_kernel, dim3((unsigned)requests, (unsigned)heads), kGateThreads, 0, stream, gates, bias, cap, state, slot_stride,
               m_offset, state_slots, cu_seqlens, (float4*)out, heads, write);
    LLM_CHECK_LAUNCH("memory_gates");
    return 0;
}

LLM_API int llm_delta_prepare(const void* proj, int ld, const float* gates, const float* conv, int taps, const float* rate,
                              const float* dt_bias, float* state, long long slot_stride, const int* state_slots, const int* positions,
                              const int* token_request, const int* cu_seqlens, void* c_out, void* unit, void* steps, int dtype, int tokens,
                              int requests, int heads, int kv_heads, int dim, int vdim, float tiny, float q_scale, int write,
                              cudaStream_t stream) {
    if (tokens == 0) return 0;
    if (taps < 1 || kv_heads < 1 || heads % kv_heads) LLM_FAIL(-1, "delta_prepare: %d taps, %d heads over %d", taps, heads, kv_heads);
    const size_t smem = (size_t)2 * kv_heads * dim * sizeof(float);
    if (smem > 200 * 1024) LLM_FAIL(-1, "delta_prepare: %d query and key channels do not fit shared memory", 2 * kv_heads * dim);
    const long long ring = (long long)heads * vdim * state_dp(dim);
    const int channels = 2 * kv_heads * dim + heads * vdim;
    return llm_dispatch_dtype(dtype, [&](auto tag) {
        using T = decltype(tag);
        const int units = 2 * kv_heads + heads + 1;
        auto run = [&](auto kern) {
            llm_launch(kern, dim3((unsigned)((tokens + kRun - 1) / kRun), (unsigned)((units + 3) / 4)), 128, 0, stream, (const T*)proj, ld, gates, conv,
                       rate, dt_bias, (const float*)state, slot_stride, ring, state_slots, positions, token_request, cu_seqlens, (T*)c_out,
                       (float2*)unit, (float2*)steps, tokens, heads, kv_heads, dim, vdim, tiny, q_scale);
        };
        auto kern = delta_prepare_kernel<T>;
        const bool pairs = dim % 2 == 0 && vdim % 2 == 0 && ld % 2 == 0 && !((uintptr_t)conv & 7);
        if (pairs && taps == 2) run(delta_prepare_run_kernel<T, 2>);
        else if (pairs && taps == 3) run(delta_prepare_run_kernel<T, 3>);
        else if (pairs && taps == 4) run(delta_prepare_run_kernel<T, 4>);
        else {
        if (smem > 48 * 1024) cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        llm_launch(kern, (unsigned)tokens, 256, smem, stream, (const T*)proj, ld, gates, conv, rate, dt_bias, (const float*)state, slot_stride,
                   ring, state_slots, positions, token_request, cu_seqlens, (T*)c_out, (float2*)unit, (float2*)steps, heads, kv_heads, dim,
                   vdim, taps, tiny, q_scale);
        }
        LLM_CHECK_LAUNCH("delta_prepare");
        if (write) {
            const int by = (channels + 255) / 256 < 16 ? (channels + 255) / 256 : 16;
            llm_launch(delta_rows_kernel<T>, dim3((unsigned)requests, (unsigned)by), 256, 0, stream, (const T*)proj, ld, state, slot_stride, ring,
                       state_slots, positions, cu_seqlens, channels, taps);
            LLM_CHECK_LAUNCH("delta_rows");
        }
        return 0;
    });
}

// kind 0: matrix memory (gates), kind 1: gated delta rule (unit, steps).  walks: null (all of `n_walks` requests) or their indices.
LLM_API int llm_state_walk(int kind, const void* qkv, int ld, const void* gates, const void* unit, const void* steps, float* state,
                           long long slot_stride, const int* state_slots, const int* cu_seqlens, const int* walks, int n_walks, float* o,
                           int o_ld, int dtype, int heads, int kv_heads, int dim, int vdim, float q_scale, int write, cudaStream_t stream) {
    if (n_walks == 0) return 0;
    if (dim > 1024 || dim <= 0 || vdim <= 0) LLM_FAIL(-1, "state_walk: head sizes %d / %d (1 to 1024 rows)", dim, vdim);
    WalkArgs a{qkv, ld, (const float4*)gates, (const float2*)unit, (const float2*)steps, state, slot_stride, state_slots, cu_seqlens, walks, o,
               heads, kv_heads, dim, vdim, o_ld, write, 8, q_scale};
    return kind == kMemory ? run_walk<kMemory>(a, dtype, n_walks, stream) : run_walk<kDelta>(a, dtype, n_walks, stream);
}

LLM_API int llm_state_finish(int kind, const float* o, int o_ld, const void* gates, const void* proj, int ld, int z_col, const float* gain, void* out,
                             int dtype, int tokens, int heads, int vdim, float eps, float tiny, cudaStream_t stream) {
    if (tokens == 0) return 0;
    const long long rows = (long long)tokens * heads;
    if (rows > 0x7ffffff0LL) LLM_FAIL(-1, "state_finish: %d tokens of %d heads are too many for a launch", tokens, heads);
    return llm_dispatch_dtype(dtype, [&](auto tag) {
        using T = decltype(tag);
        auto go = [&](auto kern) {
            llm_launch(kern, (unsigned)((rows + 7) / 8), 256, 0, stream, o, o_ld, (const float4*)gates, (const T*)proj, ld, z_col, gain, (T*)out, heads,
                       vdim, eps, tiny, (unsigned)rows);
        };
        const bool fours = vdim % 4 == 0 && ld % 4 == 0 && z_col % 4 == 0 && o_ld % 4 == 0 && !((uintptr_t)proj & 15) && !((uintptr_t)out & 15) &&
                           !((uintptr_t)gain & 15) && vdim <= 512;
        if (fours && kind == kMemory) go(vdim <= 128 ? state_finish_vec_kernel<T, kMemory, 1> : state_finish_vec_kernel<T, kMemory, 4>);
        else if (fours) go(vdim <= 128 ? state_finish_vec_kernel<T, kDelta, 1> : state_finish_vec_kernel<T, kDelta, 4>);
        else if (kind == kMemory) go(state_finish_kernel<T, kMemory>);
        else go(state_finish_kernel<T, kDelta>);
        LLM_CHECK_LAUNCH("state_finish");
        return 0;
    });
}

LLM_TRACE_EXPORT(matrix_state)
