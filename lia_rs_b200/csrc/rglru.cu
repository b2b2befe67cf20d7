// The real-gated linear recurrent unit on a step's rows.  Per channel of `width` channels in `blocks` equal parts
//     r = sigmoid(Wr_b u_b + br),  i = sigmoid(Wi_b u_b + bi)       (a square matrix per part)
//     a = exp(-rate r),  S_t = a S_(t-1) + sqrt(1 - a^2) i u,  out_t = S_t * gelu(y_t)
// u the convolution's output, y the other branch of the product, rate = 8 softplus(lambda) per channel, S 32-bit, zero
// before a request's first token.
//  * `rglru_gates`: the parts' products on the 32-bit pipes and what follows from them, a and the inflow
//    sqrt(1 - a^2) i u (1 - a^2 taken as -expm1(2 log a): no cancellation where a is close to one), 32-bit.
//  * `rglru_scan`: the recurrence along the step's runs.  Single tokens: a thread a channel.  Prompt portions: a CTA owns a few
//    channels of one portion; groups of threads take TOKENS_AHEAD consecutive tokens each, all at once: every group walks its
//    tokens from zero, the groups' end states and products of decays meet by shuffles and in shared memory, every group takes
//    its true start state from those before it and walks again, writing the outputs, while the rows of the next span of
//    tokens are on their way.  Two passes over registers, one over memory.  It also leaves the convolution's last inputs in
//    the slot's ring.
// A row whose slot is negative belongs to nobody and is skipped.
#include "conv_ring.cuh"

namespace {
constexpr int GATE_TOKENS = 8, GATE_COLUMNS = 64, GATE_THREADS = 256;

template <typename TU, typename TW>
__global__ void __launch_bounds__(GATE_THREADS)
rglru_gates_kernel(const TU* __restrict__ u, const TW* __restrict__ weight, const float* __restrict__ bias,
                   const float* __restrict__ rate, const int* __restrict__ slots, float* __restrict__ a_out,
                   float* __restrict__ inflow, int n_tokens, int width, int size) {
    extern __shared__ float gates_u[];                    // [GATE_TOKENS][size]
    pdl_launch_dependents();
    pdl_wait();
    const int first = blockIdx.x * GATE_TOKENS, block = blockIdx.y;
    for (int e = threadIdx.x; e < GATE_TOKENS * size; e += GATE_THREADS) {
        const int t = e / size, k = e - t * size;
        gates_u[e] = first + t < n_tokens ? to_float(u[(size_t)(first + t) * width + block * size + k]) : 0.f;
    }
    __syncthreads();
    const int o = blockIdx.z * GATE_COLUMNS + threadIdx.x % GATE_COLUMNS;
    if (o >= size) return;
    constexpr int PER = GATE_TOKENS / (GATE_THREADS / GATE_COLUMNS);
    const int t0 = (threadIdx.x / GATE_COLUMNS) * PER, c = block * size + o;
    float r[PER], i[PER];
#pragma unroll
    for (int p = 0; p < PER; ++p) r[p] = bias[c], i[p] = bias[width + c];
    const TW* w = weight + (size_t)block * size * 2 * size + o;         // [in][r: size | i: size]
    for (int k = 0; k < size; ++k) {
        const float wr = to_float(w[(size_t)k * 2 * size]), wi = to_float(w[(size_t)k * 2 * size + size]);
#pragma unroll
        for (int p = 0; p < PER; ++p) {
            const float v = gates_u[(t0 + p) * size + k];
            r[p] = fmaf(wr, v, r[p]);
            i[p] = fmaf(wi, v, i[p]);
        }
    }
#pragma unroll
    for (int p = 0; p < PER; ++p) {
        const int t = first + t0 + p;
        if (t >= n_tokens || slots[t] < 0) continue;
        const float log_a = -rate[c] * ring_sigmoid(r[p]);
        a_out[(size_t)t * width + c] = expf(log_a);
        inflow[(size_t)t * width + c] = sqrtf(-expm1f(2.0f * log_a)) * ring_sigmoid(i[p]) * gates_u[(t0 + p) * size + o];
    }
}

// LANES channels side by side, SCAN_THREADS / LANES groups of TOKENS_AHEAD tokens at once
constexpr int SCAN_THREADS = 256, SCAN_WARPS = SCAN_THREADS / 32, TOKENS_AHEAD = 8;

struct ScanArgs {
    const float* a; const float* inflow;                  // [n, width]
    const float* y; long long ld; const float* y_bias;    // the gate branch: rows of `ld` columns
    const float* x; const float* x_bias;                  // the convolution's inputs: rows of `ld` columns
    float* ring; float* state; long long slot_stride;     // slot s: [taps, width] and [width]
    const int* segments; int n_segments; const int* single_rows; int n_single; const int* positions; const int* slots;
    void* out; int width, taps;
};

template <typename TO>
__device__ __forceinline__ float gate_of(float z) {
    if (sizeof(TO) == 4) return ring_gelu_tanh(z);
    const float u = 0.7978845608028654f * (z + 0.044715f * z * z * z);       // (rounded to 16 bits with S: the hardware's exponential)
    return __fdividef(z, 1.0f + __expf(fminf(-2.0f * u, 80.f)));
}

template <typename TO, int LANES>
__global__ void __launch_bounds__(SCAN_THREADS)
rglru_scan_kernel(ScanArgs p) {
    constexpr int SPAN = SCAN_THREADS / LANES * TOKENS_AHEAD;
    __shared__ float2 ends[SCAN_WARPS][LANES];              // per warp: (product of the decays, end state from zero)
    __shared__ float carry[LANES];
    pdl_launch_dependents();
    pdl_wait();
    const int first = p.segments[3 * blockIdx.x], count = p.segments[3 * blockIdx.x + 2];
    if (first < 0 || count <= 0) return;
    const int slot = p.slots[first];
    if (slot < 0) return;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & (LANES - 1), group = threadIdx.x / LANES;
    const int c = blockIdx.y * LANES + lane;
    const bool live = c < p.width;
    const int cc = live ? c : 0;
    float* state = p.state + (size_t)slot * p.slot_stride + cc;
    const float y_bias = p.y_bias ? p.y_bias[cc] : 0.f;
    if (group == 0) carry[lane] = live ? *state : 0.f;
    __syncthreads();
    const size_t step_w = p.width, step_y = p.ld;
    const float* a_at = p.a + (size_t)first * step_w + cc;
    const float* b_at = p.inflow + (size_t)first * step_w + cc;
    const float* g_at = p.y + (size_t)first * step_y + cc;
    TO* out = reinterpret_cast<TO*>(p.out) + (size_t)first * step_w + cc;
    float a[TOKENS_AHEAD], b[TOKENS_AHEAD], g[TOKENS_AHEAD], na[TOKENS_AHEAD], nb[TOKENS_AHEAD], ng[TOKENS_AHEAD];
    auto fetch = [&](int r0) {
#pragma unroll
        for (int k = 0; k < TOKENS_AHEAD; ++k) {
            const bool there = r0 + k < count;
            na[k] = there ? a_at[(size_t)(r0 + k) * step_w] : 1.f;
            nb[k] = there ? b_at[(size_t)(r0 + k) * step_w] : 0.f;
            ng[k] = there ? g_at[(size_t)(r0 + k) * step_y] : 0.f;
        }
    };
    fetch(group * TOKENS_AHEAD);
    for (int base = 0; base < count; base += SPAN) {
        const int r0 = base + group * TOKENS_AHEAD;
#pragma unroll
        for (int k = 0; k < TOKENS_AHEAD; ++k) a[k] = na[k], b[k] = nb[k], g[k] = ng[k];
        if (base + SPAN < count) fetch(r0 + SPAN);          // the next span's rows travel while this one is walked
        float end = 0.f, decay = 1.f;
#pragma unroll
        for (int k = 0; k < TOKENS_AHEAD; ++k) {
            end = fmaf(a[k], end, b[k]);
            decay *= a[k];
        }
        // the groups of a warp, then the warps
        const int in_warp = threadIdx.x & 31;
#pragma unroll
        for (int o = LANES; o < 32; o *= 2) {
            const float other_end = __shfl_up_sync(0xffffffffu, end, o), other_decay = __shfl_up_sync(0xffffffffu, decay, o);
            if (in_warp >= o) {
                end = fmaf(decay, other_end, end);
                decay *= other_decay;
            }
        }
        float before_end = 0.f, before_decay = 1.f;         // of this warp's groups ahead of this one
        if (LANES < 32) {
            const float e = __shfl_up_sync(0xffffffffu, end, LANES % 32), d = __shfl_up_sync(0xffffffffu, decay, LANES % 32);
            if (in_warp >= LANES) before_end = e, before_decay = d;
        }
        if (in_warp >= 32 - LANES) ends[warp][lane] = make_float2(decay, end);
        __syncthreads();
        float S = carry[lane];
#pragma unroll
        for (int w = 0; w < SCAN_WARPS - 1; ++w) {
            const float2 e = ends[w][lane];
            if (w < warp) S = fmaf(e.x, S, e.y);
        }
        S = fmaf(before_decay, S, before_end);
#pragma unroll
        for (int k = 0; k < TOKENS_AHEAD; ++k) {
            S = fmaf(a[k], S, b[k]);
            if (live && r0 + k < count) out[(size_t)(r0 + k) * step_w] = from_float<TO>(S * gate_of<TO>(g[k] + y_bias));
        }
        __syncthreads();
        if (group == SCAN_THREADS / LANES - 1) carry[lane] = S;      // (tokens that are not there leave S as it is)
        __syncthreads();
    }
    if (group == 0 && live) *state = carry[lane];
    // the convolution's last inputs, each in its position's row of the ring
    if (p.taps > 1 && live) {
        const int kept = min(count, p.taps);
        const float x_bias = p.x_bias ? p.x_bias[c] : 0.f;
        const int pos0 = p.positions[first];
        for (int k = group; k < kept; k += SCAN_THREADS / LANES) {
            const int r = count - kept + k;
            p.ring[(size_t)slot * p.slot_stride + (size_t)((pos0 + r) % p.taps) * p.width + c] =
                p.x[((size_t)first + r) * p.ld + c] + x_bias;
        }
    }
}

// single tokens: a thread a channel
template <typename TO>
__global__ void rglru_step_kernel(ScanArgs p) {
    pdl_launch_dependents();
    pdl_wait();
    const int t = p.single_rows[blockIdx.x];
    if (t < 0) return;
    const int slot = p.slots[t];
    const int c = blockIdx.y * blockDim.x + threadIdx.x;
    if (slot < 0 || c >= p.width) return;
    float* state = p.state + (size_t)slot * p.slot_stride + c;
    const float S = fmaf(p.a[(size_t)t * p.width + c], *state, p.inflow[(size_t)t * p.width + c]);
    const float gate = p.y[(size_t)t * p.ld + c] + (p.y_bias ? p.y_bias[c] : 0.f);
    *state = S;
    reinterpret_cast<TO*>(p.out)[(size_t)t * p.width + c] = from_float<TO>(S * ring_gelu_tanh(gate));
    if (p.taps > 1)
        p.ring[(size_t)slot * p.slot_stride + (size_t)(p.positions[t] % p.taps) * p.width + c] =
            p.x[(size_t)t * p.ld + c] + (p.x_bias ? p.x_bias[c] : 0.f);
}
}  // namespace

// u [n, width] of u_dtype; weight [blocks, size, 2 size] of w_dtype: part b's [in][r's outputs | i's outputs]; bias
// [2, width] (r then i), rate [width]; a_out, inflow [n, width]: all 32-bit.
LIA_EXPORT int lia_rglru_gates(const void* u, int u_dtype, const void* weight, int w_dtype, const float* bias, const float* rate,
                               const int* slots, float* a_out, float* inflow, int n_tokens, int width, int blocks,
                               cudaStream_t stream) {
    if (n_tokens <= 0) return LIA_OK;
    if (width <= 0 || blocks <= 0 || width % blocks || blocks > 65535) return LIA_ERR_SIZE;
    const int size = width / blocks;
    const size_t bytes = (size_t)GATE_TOKENS * size * sizeof(float);
    if (bytes > 200 * 1024) return LIA_ERR_SIZE;
    const dim3 grid((n_tokens + GATE_TOKENS - 1) / GATE_TOKENS, blocks, (size + GATE_COLUMNS - 1) / GATE_COLUMNS);
    static bool raised = false;
    if (!raised) {
        cudaFuncSetAttribute(rglru_gates_kernel<float, float>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
        cudaFuncSetAttribute(rglru_gates_kernel<__nv_bfloat16, __nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
        raised = true;
    }
    if (u_dtype == LIA_F32 && w_dtype == LIA_F32)
        return lia_launch(rglru_gates_kernel<float, float>, grid, dim3(GATE_THREADS), bytes, stream, (const float*)u,
                          (const float*)weight, bias, rate, slots, a_out, inflow, n_tokens, width, size);
    if (u_dtype == LIA_BF16 && w_dtype == LIA_BF16)
        return lia_launch(rglru_gates_kernel<__nv_bfloat16, __nv_bfloat16>, grid, dim3(GATE_THREADS), bytes, stream,
                          (const __nv_bfloat16*)u, (const __nv_bfloat16*)weight, bias, rate, slots, a_out, inflow, n_tokens,
                          width, size);
    return LIA_ERR_DTYPE;
}

// a, inflow [n, width]; y, x [n, ld] (the product's two branches, y_bias and x_bias [width] or null to be added); ring and
// state: slot s at + s slot_stride, [taps, width] and [width]: all 32-bit.  `segments` [n_segments, 3] (first row, first
// position, count) and `single_rows` [n_single] name the step's runs.  out [n, width] of out_dtype.
LIA_EXPORT int lia_rglru_scan(const float* a, const float* inflow, const float* y, const float* x, long long ld,
                              const float* y_bias, const float* x_bias, float* ring, float* state, long long slot_stride,
                              const int* segments, int n_segments, const int* single_rows, int n_single,
                              const int* positions, const int* slots, void* out, int out_dtype, int width, int taps,
                              cudaStream_t stream) {
    if (n_segments + n_single <= 0) return LIA_OK;
    if (width <= 0 || taps < 1 || taps > RING_MAX_TAPS || ld < width || n_segments < 0 || n_single < 0 || (taps > 1 && !ring))
        return LIA_ERR_SIZE;
    if (out_dtype != LIA_F32 && out_dtype != LIA_BF16) return LIA_ERR_DTYPE;
    ScanArgs p = {a, inflow, y, ld, y_bias, x, x_bias, ring, state, slot_stride, segments, n_segments, single_rows, n_single,
                  positions, slots, out, width, taps};
    if (n_segments > 0) {
        // as many channels a CTA as still give about two CTAs an SM (32 channels: whole 128-byte rows)
        const int lanes = (long long)n_segments * width / 32 >= 256 ? 32 : (long long)n_segments * width / 16 >= 256 ? 16 : 8;
        const dim3 grid(n_segments, (width + lanes - 1) / lanes);
        int rc;
#define LIA_SCAN(TO)                                                                                                          \
    rc = lanes == 32   ? lia_launch(rglru_scan_kernel<TO, 32>, grid, dim3(SCAN_THREADS), 0, stream, p)                         \
         : lanes == 16 ? lia_launch(rglru_scan_kernel<TO, 16>, grid, dim3(SCAN_THREADS), 0, stream, p)                         \
                       : lia_launch(rglru_scan_kernel<TO, 8>, grid, dim3(SCAN_THREADS), 0, stream, p)
        if (out_dtype == LIA_F32) LIA_SCAN(float);
        else LIA_SCAN(__nv_bfloat16);
#undef LIA_SCAN
        if (rc != LIA_OK || n_single <= 0) return rc;
    }
    const dim3 grid(n_single, (width + 127) / 128);
    if (out_dtype == LIA_F32) return lia_launch(rglru_step_kernel<float>, grid, dim3(128), 0, stream, p);
    return lia_launch(rglru_step_kernel<__nv_bfloat16>, grid, dim3(128), 0, stream, p);
}
