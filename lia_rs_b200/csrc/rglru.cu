// The real-gated linear recurrent unit on a step's rows.  Per channel of `width` channels in `blocks` equal parts
//     r = sigmoid(Wr_b u_b + br),  i = sigmoid(Wi_b u_b + bi)       (a square matrix per part)
//     a = exp(-rate r),  S_t = a S_(t-1) + sqrt(1 - a^2) i u,  out_t = S_t * gelu(y_t)
// u the convolution's output, y the other branch of the product, rate = 8 softplus(lambda) per channel, S 32-bit, zero
// before a request's first token.
//  * `rglru_gates`: the parts' products on the 32-bit pipes and what follows from them, a and the inflow
//    sqrt(1 - a^2) i u (1 - a^2 taken as -expm1(2 log a): no cancellation where a is close to one), 32-bit.
//  * `rglru_scan`: the recurrence along the step's runs (single tokens: a thread a channel; prompt portions:).  A CTA owns 32 channels of one
//    run; its warps take WARP_TOKENS consecutive tokens each, all at once: every warp walks its tokens from zero, the
//    warps' end states and products of decays meet in shared memory, every warp takes its true start state from those
//    before it and walks again, writing the outputs.  Two passes over registers, one over memory.  It also leaves the
//    convolution's last inputs in the slot's ring.
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

constexpr int SCAN_WARPS = 16, WARP_TOKENS = 16, SCAN_SPAN = SCAN_WARPS * WARP_TOKENS;

struct ScanArgs {
    const float* a; const float* inflow;                  // [n, width]
    const float* y; long long ld; const float* y_bias;    // the gate branch: rows of `ld` columns
    const float* x; const float* x_bias;                  // the convolution's inputs: rows of `ld` columns
    float* ring; float* state; long long slot_stride;     // slot s: [taps, width] and [width]
    const int* segments; int n_segments; const int* single_rows; int n_single; const int* positions; const int* slots;
    void* out; int width, taps;
};

template <typename TO>
__global__ void __launch_bounds__(SCAN_WARPS * 32)
rglru_scan_kernel(ScanArgs p) {
    __shared__ float ends[SCAN_WARPS][32], decays[SCAN_WARPS][32], carry[32];
    pdl_launch_dependents();
    pdl_wait();
    const int first = p.segments[3 * blockIdx.x], count = p.segments[3 * blockIdx.x + 2];
    if (first < 0 || count <= 0) return;
    const int slot = p.slots[first];
    if (slot < 0) return;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int c = blockIdx.y * 32 + lane;
    const bool live = c < p.width;
    const int cc = live ? c : 0;
    float* state = p.state + (size_t)slot * p.slot_stride + cc;
    const float y_bias = p.y_bias ? p.y_bias[cc] : 0.f;
    if (warp == 0) carry[lane] = live ? *state : 0.f;
    __syncthreads();
    TO* out = reinterpret_cast<TO*>(p.out);
    float a[WARP_TOKENS], b[WARP_TOKENS], g[WARP_TOKENS], na[WARP_TOKENS], nb[WARP_TOKENS], ng[WARP_TOKENS];
    auto fetch = [&](int r0) {
#pragma unroll
        for (int k = 0; k < WARP_TOKENS; ++k) {
            const bool there = r0 + k < count;
            const size_t t = (size_t)first + (there ? r0 + k : 0);
            na[k] = there ? p.a[t * p.width + cc] : 1.f;
            nb[k] = there ? p.inflow[t * p.width + cc] : 0.f;
            ng[k] = there ? p.y[t * p.ld + cc] : 0.f;
        }
    };
    fetch(warp * WARP_TOKENS);
    for (int base = 0; base < count; base += SCAN_SPAN) {
        const int r0 = base + warp * WARP_TOKENS;
#pragma unroll
        for (int k = 0; k < WARP_TOKENS; ++k) a[k] = na[k], b[k] = nb[k], g[k] = ng[k];
        if (base + SCAN_SPAN < count) fetch(r0 + SCAN_SPAN);      // the next span's rows travel while this one is walked
        float end = 0.f, decay = 1.f;
#pragma unroll
        for (int k = 0; k < WARP_TOKENS; ++k) {
            end = fmaf(a[k], end, b[k]);
            decay *= a[k];
        }
        ends[warp][lane] = end;
        decays[warp][lane] = decay;
        __syncthreads();
        float S = carry[lane];
        for (int w = 0; w < warp; ++w) S = fmaf(decays[w][lane], S, ends[w][lane]);
#pragma unroll
        for (int k = 0; k < WARP_TOKENS; ++k) {
            S = fmaf(a[k], S, b[k]);
            if (live && r0 + k < count)
                out[((size_t)first + r0 + k) * p.width + c] = from_float<TO>(S * ring_gelu_tanh(g[k] + y_bias));
        }
        __syncthreads();
        if (warp == SCAN_WARPS - 1) carry[lane] = S;       // (tokens that are not there leave S as it is)
        __syncthreads();
    }
    if (warp == 0 && live) *state = carry[lane];
    // the convolution's last inputs, each in its position's row of the ring
    if (p.taps > 1 && live) {
        const int kept = min(count, p.taps);
        const float x_bias = p.x_bias ? p.x_bias[c] : 0.f;
        const int pos0 = p.positions[first];
        for (int k = warp; k < kept; k += SCAN_WARPS) {
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
        const dim3 grid(n_segments, (width + 31) / 32);
        const int rc = out_dtype == LIA_F32 ? lia_launch(rglru_scan_kernel<float>, grid, dim3(SCAN_WARPS * 32), 0, stream, p)
                                            : lia_launch(rglru_scan_kernel<__nv_bfloat16>, grid, dim3(SCAN_WARPS * 32), 0, stream, p);
        if (rc != LIA_OK || n_single <= 0) return rc;
    }
    const dim3 grid(n_single, (width + 127) / 128);
    if (out_dtype == LIA_F32) return lia_launch(rglru_step_kernel<float>, grid, dim3(128), 0, stream, p);
    return lia_launch(rglru_step_kernel<__nv_bfloat16>, grid, dim3(128), 0, stream, p);
}
