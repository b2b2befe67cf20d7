// What the mixers with a short causal convolution over a ring share.  Per request slot the convolution's last inputs lie
// in a ring of `taps` rows of 32-bit channels: the input of position p is row p % taps.  A token at position p reads the
// rows of p - 1 .. p - taps + 1 and writes row p % taps, which none of those is, so in a step of single tokens any number
// of CTAs may read a token's earlier inputs while one of them stores its own.  A prompt portion reads the ring only
// for its first tokens; its last tokens' inputs are stored by a kernel behind the convolution.
#pragma once
#include "common.cuh"

namespace {
constexpr int RING_MAX_TAPS = 8;

// how many of the rows just before row t continue the same run (at most `most`)
__device__ __forceinline__ int ring_run_before(const int* __restrict__ positions, const int* __restrict__ slots, int t,
                                               int slot, int pos, int most) {
    int m = 0;
    while (m < most && t - m - 1 >= 0 && slots[t - m - 1] == slot && positions[t - m - 1] == pos - m - 1) ++m;
    return m;
}

// input of channel c at distance k (>= 1) before the token at row t and position pos, whose run has m rows before t:
// zero before the sequence's start, `bias_c` added to rows of the step (the ring holds inputs with it)
__device__ __forceinline__ float ring_input(const float* __restrict__ x, long long ld, float bias_c, const float* ring,
                                            int channels, int taps, int t, int pos, int m, int k, int c) {
    if (pos - k < 0) return 0.f;
    if (k <= m) return x[(size_t)(t - k) * ld + c] + bias_c;
    return ring[(size_t)((pos - k) % taps) * channels + c];
}

__device__ __forceinline__ float ring_silu(float v) { return v / (1.0f + expf(-v)); }
// z/2 (1 + tanh(sqrt(2/pi) (z + 0.044715 z^3))) as z / (1 + exp(-2u)): the same function, one exponential
__device__ __forceinline__ float ring_gelu_tanh(float z) {
    const float u = 0.7978845608028654f * (z + 0.044715f * z * z * z);
    return z / (1.0f + expf(-2.0f * u));
}
__device__ __forceinline__ float ring_sigmoid(float v) { return 1.0f / (1.0f + expf(-v)); }
__device__ __forceinline__ float ring_softplus(float v) { return fmaxf(v, 0.f) + log1pf(expf(-fabsf(v))); }
}  // namespace
