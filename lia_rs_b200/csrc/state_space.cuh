// What the kernels of the state-space recurrence share (on the 32-bit pipes and on the tensor cores): their arguments and
// the carry of the state from chunk to chunk along a portion.
#pragma once
#include "conv_ring.cuh"

namespace {
constexpr int SSD_THREADS = 256;
constexpr int SSD_MAX = 256;                  // largest state size N and largest head size P
constexpr float LOG2_E = 1.4426950408889634f;

struct SsdArgs {
    const float* xbc; long long ld;           // [n, ld] [x | B | C]
    const float* dt; long long ld_dt;         // [n, ld_dt] raw step sizes, one a head
    const float* dt_bias; const float* rate;  // [heads]; rate = exp(A_log)
    const float* skip;                        // D [heads]
    float* state; long long slot_stride;      // slot s: [heads, N, P]
    const int* segments; int n_segments; const int* single_rows; const int* slots;
    float* y;                                 // [n, heads P]
    float* sums; float* totals;               // [chunks, heads, N, P], [chunks, heads]
    int heads, groups, N, P, vec;
};

// along each portion: scratch[c] <- the state chunk c starts from; S <- 2^C_len S + U_c; state <- the last S
__global__ void __launch_bounds__(SSD_THREADS)
ssd_carry_kernel(SsdArgs p, int chunk_length) {
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
    const int size = p.N * p.P;
    float* S = p.state + (size_t)slot * p.slot_stride + (size_t)h * size;
    const size_t chunk_stride = (size_t)p.heads * size;
    const float* total = p.totals + (size_t)before * p.heads + h;
    for (int e = blockIdx.z * blockDim.x + threadIdx.x; e < size; e += gridDim.z * blockDim.x) {
        float value = S[e];
        float* U = p.sums + ((size_t)before * p.heads + h) * size + e;
        constexpr int AHEAD = 8;                          // (the loads of eight chunks are in flight together)
        for (int c0 = 0; c0 < chunks; c0 += AHEAD) {
            float u[AHEAD], a[AHEAD];
#pragma unroll
            for (int k = 0; k < AHEAD; ++k) {
                u[k] = c0 + k < chunks ? U[(size_t)(c0 + k) * chunk_stride] : 0.f;
                a[k] = c0 + k < chunks ? total[(size_t)(c0 + k) * p.heads] : 0.f;
            }
#pragma unroll
            for (int k = 0; k < AHEAD; ++k)
                if (c0 + k < chunks) {
                    U[(size_t)(c0 + k) * chunk_stride] = value;
                    value = fmaf(exp2f(a[k]), value, u[k]);
                }
        }
        S[e] = value;
    }
}
}  // namespace
