// A short causal convolution on each channel of a step's rows,
//     y_t[c] = act(bias[c] + sum_j w[j, c] x_(t - taps + 1 + j)[c]),   act: none or SiLU,
// x the product's 32-bit rows plus `in_bias`, zero before the sequence's start; inputs before the step come from the
// slot's ring (conv_ring.cuh), which this kernel reads and does not change.  Every sum is 32-bit, in the order of j.
#include "conv_ring.cuh"

namespace {
template <typename TO> __device__ __forceinline__ void put_four(TO* dst, const float (&v)[4]);
template <> __device__ __forceinline__ void put_four<float>(float* dst, const float (&v)[4]) {
    *reinterpret_cast<float4*>(dst) = make_float4(v[0], v[1], v[2], v[3]);
}
template <> __device__ __forceinline__ void put_four<__nv_bfloat16>(__nv_bfloat16* dst, const float (&v)[4]) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(v[0], v[1]), hi = __floats2bfloat162_rn(v[2], v[3]);
    *reinterpret_cast<uint2*>(dst) = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
}

template <typename TO, int VEC>                   // VEC: channels a thread takes (4: every row 16-byte aligned)
__global__ void ring_conv_kernel(const float* __restrict__ x, long long ld, const float* __restrict__ in_bias,
                                 const float* __restrict__ weight, const float* __restrict__ bias, const float* ring,
                                 long long ring_stride, const int* __restrict__ positions, const int* __restrict__ slots,
                                 TO* __restrict__ out, int n_tokens, int channels, int taps, int act) {
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x;
    if (t >= n_tokens) return;
    const int slot = slots[t];
    if (slot < 0) return;
    const int pos = positions[t];
    const int m = ring_run_before(positions, slots, t, slot, pos, taps - 1);
    const float* own = ring ? ring + (size_t)slot * ring_stride : nullptr;
    for (int c = (blockIdx.y * blockDim.x + threadIdx.x) * VEC; c < channels; c += gridDim.y * blockDim.x * VEC) {
        float y[VEC];
        if (VEC == 4) {
            const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
            const float4 ib = in_bias ? *reinterpret_cast<const float4*>(in_bias + c) : zero;
            const float4 b = bias ? *reinterpret_cast<const float4*>(bias + c) : zero;
            y[0] = b.x, y[1] = b.y, y[2] = b.z, y[3] = b.w;
            for (int j = 0; j < taps; ++j) {
                const int k = taps - 1 - j;
                float4 v = zero;
                if (k <= m) {
                    v = *reinterpret_cast<const float4*>(x + (size_t)(t - k) * ld + c);
                    v.x += ib.x, v.y += ib.y, v.z += ib.z, v.w += ib.w;
                } else if (pos - k >= 0) {
                    v = *reinterpret_cast<const float4*>(own + (size_t)((pos - k) % taps) * channels + c);
                }
                const float4 w = *reinterpret_cast<const float4*>(weight + (size_t)j * channels + c);
                y[0] = fmaf(w.x, v.x, y[0]);
                y[1] = fmaf(w.y, v.y, y[1]);
                y[2] = fmaf(w.z, v.z, y[2]);
                y[3] = fmaf(w.w, v.w, y[3]);
            }
        } else {
            const float ib = in_bias ? in_bias[c] : 0.f;
            y[0] = bias ? bias[c] : 0.f;
            for (int j = 0; j < taps - 1; ++j)
                y[0] = fmaf(weight[(size_t)j * channels + c], ring_input(x, ld, ib, own, channels, taps, t, pos, m, taps - 1 - j, c), y[0]);
            y[0] = fmaf(weight[(size_t)(taps - 1) * channels + c], x[(size_t)t * ld + c] + ib, y[0]);
        }
        if (act == 1) {
#pragma unroll
            for (int i = 0; i < VEC; ++i) y[i] = ring_silu(y[i]);
        }
        if constexpr (VEC == 4) {
            put_four<TO>(out + (size_t)t * channels + c, y);
        } else {
            out[(size_t)t * channels + c] = from_float<TO>(y[0]);
        }
    }
}
// The same for many tokens and four taps: a thread takes four channels of RUN consecutive rows, whose inputs it has in flight
// at once, and shifts its window along; where a row does not continue the run of the row before it, the window is read anew.
constexpr int RUN = 8;
template <typename TO>
__global__ void ring_conv_run_kernel(const float* __restrict__ x, long long ld, const float* __restrict__ in_bias,
                                     const float* __restrict__ weight, const float* __restrict__ bias, const float* ring,
                                     long long ring_stride, const int* __restrict__ positions, const int* __restrict__ slots,
                                     TO* __restrict__ out, int n_tokens, int channels, int act) {
    constexpr int TAPS = 4;
    pdl_launch_dependents();
    pdl_wait();
    const int t0 = blockIdx.x * RUN, c = (blockIdx.y * blockDim.x + threadIdx.x) * 4;
    if (c >= channels) return;
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    const float4 ib = in_bias ? *reinterpret_cast<const float4*>(in_bias + c) : zero;
    auto input = [&](int t) {
        float4 v = *reinterpret_cast<const float4*>(x + (size_t)t * ld + c);
        v.x += ib.x, v.y += ib.y, v.z += ib.z, v.w += ib.w;
        return v;
    };
    float4 own[RUN];
    int row_slot[RUN], row_pos[RUN];
#pragma unroll
    for (int r = 0; r < RUN; ++r) {
        row_slot[r] = t0 + r < n_tokens ? slots[t0 + r] : -1;
        row_pos[r] = t0 + r < n_tokens ? positions[t0 + r] : 0;
    }
#pragma unroll
    for (int r = 0; r < RUN; ++r) own[r] = t0 + r < n_tokens ? input(t0 + r) : zero;
    const float4 b = bias ? *reinterpret_cast<const float4*>(bias + c) : zero;
    float4 w[TAPS], window[TAPS - 1];                    // window[k - 1]: the input k tokens back
#pragma unroll
    for (int j = 0; j < TAPS; ++j) w[j] = *reinterpret_cast<const float4*>(weight + (size_t)j * channels + c);
    int last_slot = -1, last_pos = 0;
#pragma unroll
    for (int r = 0; r < RUN; ++r) {
        const int t = t0 + r;
        if (t >= n_tokens) break;
        const int slot = row_slot[r], pos = row_pos[r];
        if (slot >= 0) {
            if (slot != last_slot || pos != last_pos + 1) {
                const int m = ring_run_before(positions, slots, t, slot, pos, TAPS - 1);
#pragma unroll
                for (int k = 1; k < TAPS; ++k) {
                    window[k - 1] = zero;
                    if (k <= m) window[k - 1] = input(t - k);
                    else if (pos - k >= 0)
                        window[k - 1] = *reinterpret_cast<const float4*>(ring + (size_t)slot * ring_stride + (size_t)((pos - k) % TAPS) * channels + c);
                }
            }
            float y[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
            for (int j = 0; j < TAPS; ++j) {
                const float4 v = j == TAPS - 1 ? own[r] : window[TAPS - 2 - j];
                y[0] = fmaf(w[j].x, v.x, y[0]);
                y[1] = fmaf(w[j].y, v.y, y[1]);
                y[2] = fmaf(w[j].z, v.z, y[2]);
                y[3] = fmaf(w[j].w, v.w, y[3]);
            }
            if (act == 1) {
#pragma unroll
                for (int i = 0; i < 4; ++i) y[i] = ring_silu(y[i]);
            }
            put_four<TO>(out + (size_t)t * channels + c, y);
#pragma unroll
            for (int k = TAPS - 2; k > 0; --k) window[k] = window[k - 1];
            window[0] = own[r];
        }
        last_slot = slot;
        last_pos = pos;
    }
}
}  // namespace

// x [n, ld] 32-bit (the first `channels` columns), in_bias [channels] or null, weight [taps, channels] (row j: the tap of
// distance taps - 1 - j), bias [channels] or null, ring (slot s at ring + s ring_stride: [taps, channels]; null for one
// tap), all 32-bit.  out [n, channels] of `out_dtype`.
LIA_EXPORT int lia_ring_conv(const float* x, long long ld, const float* in_bias, const float* weight, const float* bias,
                             const float* ring, long long ring_stride, const int* positions, const int* slots, void* out,
                             int out_dtype, int n_tokens, int channels, int taps, int act, cudaStream_t stream) {
    if (n_tokens <= 0) return LIA_OK;
    if (channels <= 0 || taps < 1 || taps > RING_MAX_TAPS || ld < channels || (taps > 1 && !ring) || act < 0 || act > 1)
        return LIA_ERR_SIZE;
    if (out_dtype != LIA_F32 && out_dtype != LIA_BF16) return LIA_ERR_DTYPE;
    const uintptr_t bits = (uintptr_t)x | (uintptr_t)in_bias | (uintptr_t)weight | (uintptr_t)bias | (uintptr_t)ring | (uintptr_t)out;
    const bool four = channels % 4 == 0 && ld % 4 == 0 && ring_stride % 4 == 0 && (bits & 15u) == 0;
    const int threads = 128, per_block = threads * (four ? 4 : 1);
    const dim3 grid(n_tokens, (channels + per_block - 1) / per_block);
    if (four && taps == 4 && n_tokens >= 128) {
        const dim3 runs((n_tokens + RUN - 1) / RUN, grid.y);
        if (out_dtype == LIA_F32)
            return lia_launch(ring_conv_run_kernel<float>, runs, dim3(threads), 0, stream, x, ld, in_bias, weight, bias, ring,
                              ring_stride, positions, slots, (float*)out, n_tokens, channels, act);
        return lia_launch(ring_conv_run_kernel<__nv_bfloat16>, runs, dim3(threads), 0, stream, x, ld, in_bias, weight, bias, ring,
                          ring_stride, positions, slots, (__nv_bfloat16*)out, n_tokens, channels, act);
    }
#define LIA_CONV(TO, VEC)                                                                                              \
    return lia_launch(ring_conv_kernel<TO, VEC>, grid, dim3(threads), 0, stream, x, ld, in_bias, weight, bias, ring,  \
                      ring_stride, positions, slots, (TO*)out, n_tokens, channels, taps, act)
    if (out_dtype == LIA_F32) {
        if (four) LIA_CONV(float, 4);
        LIA_CONV(float, 1);
    }
    if (four) LIA_CONV(__nv_bfloat16, 4);
    LIA_CONV(__nv_bfloat16, 1);
#undef LIA_CONV
}
