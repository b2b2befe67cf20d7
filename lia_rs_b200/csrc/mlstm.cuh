// What the kernels of the matrix memory with exponential gates (mLSTM) share, on the 32-bit pipes and on the tensor cores:
// their arguments, the gates and exponents of a chunk's tokens, and the carry of the memory from chunk to chunk.
//
// The recurrence per request and head, with log gates i_t and f_t <= 0 and a running maximum m:
//     m_t = max(f_t + m_(t-1), i_t)
//     S_t = exp(f_t + m_(t-1) - m_t) S_(t-1) + exp(i_t - m_t) k_t v_t^T,   n_t likewise with k_t alone
//     o_t = S_t^T q_t / (max(|n_t . q_t|, exp(-m_t)) + 1e-6)
// Inside a chunk that begins behind (S_0, n_0, m_0), with F_t = f_1 + ... + f_t, a_j = i_j - F_j and
// M_t = max(m_0, a_1, ..., a_t):
//     m_t = F_t + M_t,   S_t = exp(m_0 - M_t) S_0 + sum_(j<=t) exp(a_j - M_t) k_j v_j^T
// so every exponent is <= 0.  F, a and M are sums of many terms that cancel in those exponents: they are formed in 64-bit
// (a few numbers a token), and an exponent is the difference of two pairs of 32-bit numbers.
#pragma once
#include "common.cuh"

namespace {
constexpr int MLSTM_THREADS = 256;
constexpr int MLSTM_MAX = 512;                // largest head size of keys and of values

struct MlstmArgs {
    const void* qkv; long long ld; int qkv_bf16;           // [n, ld] [q: heads d | k: heads d | v: heads dv]
    const float* gates; long long ld_g;                    // [n, ld_g] [output gate: heads dv | i: heads | f: heads]
    const float* i_bias; const float* f_bias; float cap;   // log gates: cap * tanh(. / cap), the forget gate's through log sigmoid
    float* state; long long slot_stride;                   // slot s: S [heads, d, dv], n [heads, d], m [heads]
    const int* segments; int n_segments; const int* single_rows; const int* slots;
    const float* norm_weight; float eps;                   // [heads dv]
    void* out;                                             // [n, heads dv] in the compute element type
    float* y;                                              // [n, heads dv] 32-bit: o ahead of its norm (where a head is cut)
    float* sums; float* totals; float* tops; float* starts;// [chunks, heads, d dv + d], and [chunks, heads] each: F of the chunk,
                                                           // its largest exponent counted from its end, m ahead of it
    int heads, d, dv, vec;
    float q_scale;
};

__device__ __forceinline__ float mlstm_sigmoid(float v) { return 1.0f / (1.0f + expf(-v)); }

// log gates of token t and head h
__device__ __forceinline__ void mlstm_log_gates(const MlstmArgs& p, int t, int h, float& i, float& f) {
    const float* g = p.gates + (size_t)t * p.ld_g + (size_t)p.heads * p.dv;
    i = p.cap * tanhf((g[h] + p.i_bias[h]) / p.cap);
    const float z = p.cap * tanhf((g[p.heads + h] + p.f_bias[h]) / p.cap);
    f = -(fmaxf(-z, 0.f) + log1pf(expf(-fabsf(z))));
}

// Two 32-bit numbers whose sum is x to about 48 bits (an infinite x: itself and zero).
__device__ __forceinline__ float2 mlstm_pair(double x) {
    const float hi = (float)x;
    return make_float2(hi, isinf(hi) ? 0.f : (float)(x - (double)hi));
}
__device__ __forceinline__ float mlstm_difference(float2 a, float2 b) { return (a.x - b.x) + (a.y - b.y); }

// The numbers of a chunk's token that thread t < TOKENS gets back; every thread of the CTA calls it (it holds barriers).
struct MlstmToken {
    double total;      // F_t (behind the chunk's end: F of the chunk)
    double a;          // a_t; minus infinity behind the chunk's end
    double top;        // max(a_1 .. a_t)
};
template <int TOKENS>
__device__ __forceinline__ MlstmToken mlstm_tokens(const MlstmArgs& p, int first, int len, int h, double* scratch) {
    constexpr int WARPS = TOKENS / 32;                     // scratch: [2 * WARPS]
    const int t = threadIdx.x, lane = t & 31, warp = t >> 5;
    MlstmToken r = {0.0, -INFINITY, -INFINITY};
    float i = -INFINITY, f = 0.f;
    if (t < TOKENS) {
        if (t < len) mlstm_log_gates(p, first + t, h, i, f);
        r.total = (double)f;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const double before = __shfl_up_sync(0xffffffffu, r.total, o);
            if (lane >= o) r.total += before;
        }
        if (WARPS > 1 && lane == 31) scratch[warp] = r.total;
    }
    if (WARPS > 1) __syncthreads();
    if (t < TOKENS) {
        for (int w = 0; w < warp; ++w) r.total += scratch[w];
        r.a = t < len ? (double)i - r.total : -INFINITY;
        r.top = r.a;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const double before = __shfl_up_sync(0xffffffffu, r.top, o);
            if (lane >= o) r.top = fmax(r.top, before);
        }
        if (WARPS > 1 && lane == 31) scratch[WARPS + warp] = r.top;
    }
    if (WARPS > 1) __syncthreads();
    if (t < TOKENS)
        for (int w = 0; w < warp; ++w) r.top = fmax(r.top, scratch[WARPS + w]);
    return r;
}

// which portion and which of its chunks the CTA `index` serves: false when there is none; `last`: the portion ends here
template <int TOKENS>
__device__ __forceinline__ bool mlstm_find_chunk(const MlstmArgs& p, int index, int* first, int* len, bool* last) {
    for (int s = 0; s < p.n_segments; ++s) {
        const int count = p.segments[3 * s + 2], chunks = (count + TOKENS - 1) / TOKENS;
        if (index < chunks) {
            *first = p.segments[3 * s] + index * TOKENS;
            *len = min(TOKENS, count - index * TOKENS);
            *last = index == chunks - 1;
            return true;
        }
        index -= chunks;
    }
    return false;
}

// Along each portion: scratch[c] <- what chunk c starts from; (S, n) <- exp(m + F_c - m') (S, n) + exp(top_c - m') U_c,
// m' = max(m + F_c, top_c); the last (S, n) goes back to the request's state (its m is written by the last chunk's output
// CTA, which runs behind every reader of the old one).
template <int VEC>
__global__ void __launch_bounds__(MLSTM_THREADS)
mlstm_carry_kernel(MlstmArgs p, int chunk_length) {
    pdl_launch_dependents();
    pdl_wait();
    const int s = blockIdx.x, h = blockIdx.y;
    if (s >= p.n_segments) return;
    const int first = p.segments[3 * s], count = p.segments[3 * s + 2];
    const int slot = p.slots[first];
    if (slot < 0) return;
    int before = 0;
    for (int q = 0; q < s; ++q) before += (p.segments[3 * q + 2] + chunk_length - 1) / chunk_length;
    const int chunks = (count + chunk_length - 1) / chunk_length;
    const int size = p.d * p.dv, unit = size + p.d;
    float* base = p.state + (size_t)slot * p.slot_stride;
    const float m_start = base[(size_t)p.heads * unit + h];
    const size_t at = (size_t)before * p.heads + h;
    const bool keeper = blockIdx.z == 0 && threadIdx.x == 0;
    for (int e = (blockIdx.z * blockDim.x + threadIdx.x) * VEC; e < unit; e += gridDim.z * blockDim.x * VEC) {
        float* home = e < size ? base + (size_t)h * size + e : base + (size_t)p.heads * size + (size_t)h * p.d + (e - size);
        float value[VEC];
#pragma unroll
        for (int v = 0; v < VEC; ++v) value[v] = home[v];
        float m = m_start;
        float* U = p.sums + at * unit + e;
        constexpr int AHEAD = 8;                          // (the loads of eight chunks are in flight together)
        for (int c0 = 0; c0 < chunks; c0 += AHEAD) {
            float u[AHEAD][VEC], total[AHEAD], top[AHEAD];
#pragma unroll
            for (int k = 0; k < AHEAD; ++k) {
                const bool there = c0 + k < chunks;
                const size_t chunk = (size_t)(c0 + k) * p.heads;
                if constexpr (VEC == 4) {
                    const float4 x = there ? *reinterpret_cast<const float4*>(U + chunk * unit) : make_float4(0.f, 0.f, 0.f, 0.f);
                    u[k][0] = x.x, u[k][1] = x.y, u[k][2] = x.z, u[k][3] = x.w;
                } else {
                    u[k][0] = there ? U[chunk * unit] : 0.f;
                }
                total[k] = there ? p.totals[at + chunk] : 0.f;
                top[k] = there ? p.tops[at + chunk] : 0.f;
            }
#pragma unroll
            for (int k = 0; k < AHEAD; ++k)
                if (c0 + k < chunks) {
                    const size_t chunk = (size_t)(c0 + k) * p.heads;
                    if constexpr (VEC == 4)
                        *reinterpret_cast<float4*>(U + chunk * unit) = make_float4(value[0], value[1], value[2], value[3]);
                    else
                        U[chunk * unit] = value[0];
                    if (keeper) p.starts[at + chunk] = m;
                    const float kept = m + total[k], next = fmaxf(kept, top[k]);
                    const float keep = expf(kept - next), put = expf(top[k] - next);
#pragma unroll
                    for (int v = 0; v < VEC; ++v) value[v] = fmaf(keep, value[v], put * u[k][v]);
                    m = next;
                }
        }
#pragma unroll
        for (int v = 0; v < VEC; ++v) home[v] = value[v];
    }
}

inline int mlstm_launch_carry(const MlstmArgs& p, int chunk_length, bool four, cudaStream_t stream) {
    const int unit = p.d * p.dv + p.d, per = MLSTM_THREADS * (four ? 4 : 1);
    const dim3 grid(p.n_segments, p.heads, (unit + per - 1) / per);
    if (four) return lia_launch(mlstm_carry_kernel<4>, grid, dim3(MLSTM_THREADS), 0, stream, p, chunk_length);
    return lia_launch(mlstm_carry_kernel<1>, grid, dim3(MLSTM_THREADS), 0, stream, p, chunk_length);
}

// Words of scratch and where its parts lie.
inline long long mlstm_scratch_words(int chunks, int heads, int d, int dv) { return (long long)chunks * heads * ((long long)d * dv + d + 3); }
inline void mlstm_place_scratch(MlstmArgs& p, float* scratch, int chunks) {
    const size_t n = (size_t)chunks * p.heads;
    p.sums = scratch;
    p.totals = scratch + n * ((size_t)p.d * p.dv + p.d);
    p.tops = p.totals + n;
    p.starts = p.tops + n;
}
}  // namespace
