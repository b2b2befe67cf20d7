// What a layer with a norm on both sides of each sublayer needs on the 32-bit residual stream:
//  * residual[r] += rms(y[r] + bias) * w        (the sublayer's output y, normed, joins the stream), and in the same
//    pass, optionally, next[r] = rms(residual[r]) * w2 in the compute element type (the input of the sublayer that
//    follows), so that the stream is read once between two sublayers;
//  * out[r, :] = act(in[r, :]) for 32-bit rows with any row stride: the activation between the two products of a dense
//    feed-forward (tanh form of GELU), SiLU, or a plain change of element type of some columns.
// Sums of squares, means and reciprocal roots are 32-bit; the order of a row's additions depends on the width alone.
#include "common.cuh"

namespace {
template <typename TO>
__global__ void norm_residual_kernel(const float* __restrict__ y, const float* __restrict__ bias,
                                     const float* __restrict__ weight, float* __restrict__ residual,
                                     const float* __restrict__ next_weight, TO* __restrict__ next, int rows, int hidden,
                                     float eps, float next_eps) {
    __shared__ float scratch[32];
    pdl_launch_dependents();
    pdl_wait();
    const int r = blockIdx.x;
    if (r >= rows) return;
    const float* yr = y + (size_t)r * hidden;
    float* xr = residual + (size_t)r * hidden;
    float sum = 0.f;
    for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
        const float v = yr[i] + (bias ? bias[i] : 0.f);
        sum = fmaf(v, v, sum);
    }
    sum = block_sum(sum, scratch);
    const float inv = 1.0f / sqrtf(sum / (float)hidden + eps);
    float sum2 = 0.f;
    for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
        const float v = yr[i] + (bias ? bias[i] : 0.f);
        const float x = xr[i] + v * inv * weight[i];
        xr[i] = x;
        sum2 = fmaf(x, x, sum2);
    }
    if (!next) return;
    sum2 = block_sum(sum2, scratch);
    const float inv2 = 1.0f / sqrtf(sum2 / (float)hidden + next_eps);
    TO* nr = next + (size_t)r * hidden;
    for (int i = threadIdx.x; i < hidden; i += blockDim.x)          // (each thread reads back what it wrote itself)
        nr[i] = from_float<TO>(xr[i] * inv2 * next_weight[i]);
}

template <typename TO> __device__ __forceinline__ void store_four(TO* dst, float a, float b, float c, float d);
template <> __device__ __forceinline__ void store_four<float>(float* dst, float a, float b, float c, float d) {
    *reinterpret_cast<float4*>(dst) = make_float4(a, b, c, d);
}
template <> __device__ __forceinline__ void store_four<__nv_bfloat16>(__nv_bfloat16* dst, float a, float b, float c, float d) {
    __nv_bfloat162 lo = __floats2bfloat162_rn(a, b), hi = __floats2bfloat162_rn(c, d);
    uint2 v;
    v.x = *reinterpret_cast<uint32_t*>(&lo);
    v.y = *reinterpret_cast<uint32_t*>(&hi);
    *reinterpret_cast<uint2*>(dst) = v;
}

// The same with a row in registers: PER quads a thread (width a multiple of 4, rows 16-byte aligned), the row read once and
// the weights, which no kernel writes, on their way before the kernel ahead is awaited.
template <typename TO, int PER>
__global__ void norm_residual_quads_kernel(const float* __restrict__ y, const float* __restrict__ bias,
                                           const float* __restrict__ weight, float* __restrict__ residual,
                                           const float* __restrict__ next_weight, TO* __restrict__ next, int hidden, float eps,
                                           float next_eps) {
    __shared__ float scratch[32];
    pdl_launch_dependents();
    const int r = blockIdx.x, quads = hidden / 4;
    float4 w[PER], w2[PER], b[PER];
#pragma unroll
    for (int i = 0; i < PER; ++i) {
        const int q = threadIdx.x + i * blockDim.x;
        const bool in = q < quads;
        w[i] = in ? reinterpret_cast<const float4*>(weight)[q] : make_float4(0.f, 0.f, 0.f, 0.f);
        w2[i] = in && next ? reinterpret_cast<const float4*>(next_weight)[q] : make_float4(0.f, 0.f, 0.f, 0.f);
        b[i] = in && bias ? reinterpret_cast<const float4*>(bias)[q] : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    pdl_wait();
    float4 v[PER], x[PER];
#pragma unroll
    for (int i = 0; i < PER; ++i) {
        const int q = threadIdx.x + i * blockDim.x;
        v[i] = q < quads ? reinterpret_cast<const float4*>(y + (size_t)r * hidden)[q] : make_float4(0.f, 0.f, 0.f, 0.f);
        x[i] = q < quads ? reinterpret_cast<const float4*>(residual + (size_t)r * hidden)[q] : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    float sum = 0.f;
#pragma unroll
    for (int i = 0; i < PER; ++i) {
        v[i].x += b[i].x, v[i].y += b[i].y, v[i].z += b[i].z, v[i].w += b[i].w;
        sum = fmaf(v[i].x, v[i].x, sum), sum = fmaf(v[i].y, v[i].y, sum);
        sum = fmaf(v[i].z, v[i].z, sum), sum = fmaf(v[i].w, v[i].w, sum);
    }
    const float inv = 1.0f / sqrtf(block_sum(sum, scratch) / (float)hidden + eps);
    float sum2 = 0.f;
#pragma unroll
    for (int i = 0; i < PER; ++i) {
        const int q = threadIdx.x + i * blockDim.x;
        x[i].x += v[i].x * inv * w[i].x, x[i].y += v[i].y * inv * w[i].y;
        x[i].z += v[i].z * inv * w[i].z, x[i].w += v[i].w * inv * w[i].w;
        if (q < quads) reinterpret_cast<float4*>(residual + (size_t)r * hidden)[q] = x[i];
        sum2 = fmaf(x[i].x, x[i].x, sum2), sum2 = fmaf(x[i].y, x[i].y, sum2);
        sum2 = fmaf(x[i].z, x[i].z, sum2), sum2 = fmaf(x[i].w, x[i].w, sum2);
    }
    if (!next) return;
    const float inv2 = 1.0f / sqrtf(block_sum(sum2, scratch) / (float)hidden + next_eps);
#pragma unroll
    for (int i = 0; i < PER; ++i) {
        const int q = threadIdx.x + i * blockDim.x;
        if (q < quads)
            store_four<TO>(next + (size_t)r * hidden + 4 * q, x[i].x * inv2 * w2[i].x, x[i].y * inv2 * w2[i].y, x[i].z * inv2 * w2[i].z,
                           x[i].w * inv2 * w2[i].w);
    }
}

// residual[r] += rms(v) * weight with v = sum_i scale_i * (w_i ? rms_i(y_i + b_i) * w_i : y_i + b_i) over one or two terms, and
// `next` (optional) the new stream in the compute element type: what follows a sublayer whose output is normed and whose
// successor reads the stream itself, in one pass.  A thread keeps PER quads of the row in registers (width a multiple of
// 4, rows 16-byte aligned); PER 0: any width, the row read again for every pass.
struct NormTerm { const float* y; const float* bias; const float* weight; float scale, eps; };

template <typename TO, int TERMS, int PER>
__global__ void norm_terms_residual_kernel(NormTerm t0, NormTerm t1, const float* __restrict__ weight,
                                           float* __restrict__ residual, TO* __restrict__ next, int hidden, float eps) {
    __shared__ float scratch[32];
    pdl_launch_dependents();
    const int r = blockIdx.x;
    if constexpr (PER > 0) {
        const int quads = hidden / 4;
        pdl_wait();
        float4 v[PER], x[PER];
#pragma unroll
        for (int i = 0; i < PER; ++i) {
            const int q = threadIdx.x + i * blockDim.x;
            x[i] = q < quads ? reinterpret_cast<const float4*>(residual + (size_t)r * hidden)[q] : make_float4(0.f, 0.f, 0.f, 0.f);
            v[i] = make_float4(0.f, 0.f, 0.f, 0.f);
        }
        float4 y[TERMS][PER];
#pragma unroll
        for (int n = 0; n < TERMS; ++n) {
            const NormTerm& term = n ? t1 : t0;
#pragma unroll
            for (int i = 0; i < PER; ++i) {
                const int q = threadIdx.x + i * blockDim.x;
                y[n][i] = q < quads ? reinterpret_cast<const float4*>(term.y + (size_t)r * hidden)[q] : make_float4(0.f, 0.f, 0.f, 0.f);
                if (term.bias && q < quads) {
                    const float4 b = reinterpret_cast<const float4*>(term.bias)[q];
                    y[n][i].x += b.x, y[n][i].y += b.y, y[n][i].z += b.z, y[n][i].w += b.w;
                }
            }
        }
        float sum = 0.f;
#pragma unroll
        for (int n = 0; n < TERMS; ++n) {
            const NormTerm& term = n ? t1 : t0;
            float factor = term.scale;
            if (term.weight) {
                sum = 0.f;
#pragma unroll
                for (int i = 0; i < PER; ++i) {
                    sum = fmaf(y[n][i].x, y[n][i].x, sum), sum = fmaf(y[n][i].y, y[n][i].y, sum);
                    sum = fmaf(y[n][i].z, y[n][i].z, sum), sum = fmaf(y[n][i].w, y[n][i].w, sum);
                }
                factor *= 1.0f / sqrtf(block_sum(sum, scratch) / (float)hidden + term.eps);
            }
#pragma unroll
            for (int i = 0; i < PER; ++i) {
                const int q = threadIdx.x + i * blockDim.x;
                float4 w = make_float4(1.f, 1.f, 1.f, 1.f);
                if (term.weight && q < quads) w = reinterpret_cast<const float4*>(term.weight)[q];
                v[i].x = fmaf(y[n][i].x * factor, w.x, v[i].x), v[i].y = fmaf(y[n][i].y * factor, w.y, v[i].y);
                v[i].z = fmaf(y[n][i].z * factor, w.z, v[i].z), v[i].w = fmaf(y[n][i].w * factor, w.w, v[i].w);
            }
        }
        sum = 0.f;
#pragma unroll
        for (int i = 0; i < PER; ++i) {
            sum = fmaf(v[i].x, v[i].x, sum), sum = fmaf(v[i].y, v[i].y, sum);
            sum = fmaf(v[i].z, v[i].z, sum), sum = fmaf(v[i].w, v[i].w, sum);
        }
        const float inv = 1.0f / sqrtf(block_sum(sum, scratch) / (float)hidden + eps);
#pragma unroll
        for (int i = 0; i < PER; ++i) {
            const int q = threadIdx.x + i * blockDim.x;
            if (q < quads) {
                const float4 w = reinterpret_cast<const float4*>(weight)[q];
                x[i].x += v[i].x * inv * w.x, x[i].y += v[i].y * inv * w.y;
                x[i].z += v[i].z * inv * w.z, x[i].w += v[i].w * inv * w.w;
                reinterpret_cast<float4*>(residual + (size_t)r * hidden)[q] = x[i];
                if (next) store_four<TO>(next + (size_t)r * hidden + 4 * q, x[i].x, x[i].y, x[i].z, x[i].w);
            }
        }
    } else {
        pdl_wait();
        float factor[TERMS];
#pragma unroll
        for (int n = 0; n < TERMS; ++n) {
            const NormTerm& term = n ? t1 : t0;
            factor[n] = term.scale;
            if (!term.weight) continue;
            float sum = 0.f;
            for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
                const float y = term.y[(size_t)r * hidden + i] + (term.bias ? term.bias[i] : 0.f);
                sum = fmaf(y, y, sum);
            }
            factor[n] *= 1.0f / sqrtf(block_sum(sum, scratch) / (float)hidden + term.eps);
        }
        auto value = [&](int i) {
            float v = 0.f;
#pragma unroll
            for (int n = 0; n < TERMS; ++n) {
                const NormTerm& term = n ? t1 : t0;
                const float y = term.y[(size_t)r * hidden + i] + (term.bias ? term.bias[i] : 0.f);
                v = fmaf(y * factor[n], term.weight ? term.weight[i] : 1.f, v);
            }
            return v;
        };
        float sum = 0.f;
        for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
            const float v = value(i);
            sum = fmaf(v, v, sum);
        }
        const float inv = 1.0f / sqrtf(block_sum(sum, scratch) / (float)hidden + eps);
        for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
            const float x = residual[(size_t)r * hidden + i] + value(i) * inv * weight[i];
            residual[(size_t)r * hidden + i] = x;
            if (next) next[(size_t)r * hidden + i] = from_float<TO>(x);
        }
    }
}

// 0.5 z (1 + tanh(u)), u = sqrt(2/pi) (z + 0.044715 z^3), written as z / (1 + exp(-2u)): the same function, one exponential
__device__ __forceinline__ float gelu_tanh(float z) {
    const float u = 0.7978845608028654f * (z + 0.044715f * z * z * z);
    return z / (1.0f + expf(-2.0f * u));
}

// act: 0 identity, 1 GELU (tanh form), 2 SiLU, 3 the square of ReLU, 4 ReLU, 5 xIELU with the constants p0, p1
__device__ __forceinline__ float activate(int act, float z, float p0 = 0.f, float p1 = 0.f) {
    if (act == 5) return lia_xielu(z, p0, p1);
    if (act == 1) return gelu_tanh(z);
    if (act == 2) return z / (1.0f + expf(-z));
    if (act == 3) { const float r = fmaxf(z, 0.f); return r * r; }
    if (act == 4) return fmaxf(z, 0.f);
    return z;
}

// four elements a thread: rows whose width and strides are multiples of 4 from 16-byte aligned bases.  `gated`: the
// row holds `width` gate elements and then `width` more, out = act(gate) * the other.
template <typename TO>
__global__ void activation_rows4_kernel(const float* __restrict__ in, long long ld_in, TO* __restrict__ out,
                                        long long ld_out, int rows, int quads, int act, int gated, float p0, float p1) {
    pdl_launch_dependents();
    pdl_wait();
    const long long total = (long long)rows * quads;
    for (long long e = (long long)blockIdx.x * blockDim.x + threadIdx.x; e < total; e += (long long)gridDim.x * blockDim.x) {
        const long long r = e / quads;
        const int i = (int)(e - r * quads) * 4;
        const float4 z = *reinterpret_cast<const float4*>(in + r * ld_in + i);
        float4 u = make_float4(1.f, 1.f, 1.f, 1.f);
        if (gated) u = *reinterpret_cast<const float4*>(in + r * ld_in + 4 * quads + i);
        store_four<TO>(out + r * ld_out + i, activate(act, z.x, p0, p1) * u.x, activate(act, z.y, p0, p1) * u.y, activate(act, z.z, p0, p1) * u.z,
                       activate(act, z.w, p0, p1) * u.w);
    }
}

template <typename TO>
__global__ void activation_rows_kernel(const float* __restrict__ in, long long ld_in, TO* __restrict__ out,
                                       long long ld_out, int rows, int width, int act, int gated, float p0, float p1) {
    pdl_launch_dependents();
    pdl_wait();
    const long long total = (long long)rows * width;
    for (long long e = (long long)blockIdx.x * blockDim.x + threadIdx.x; e < total; e += (long long)gridDim.x * blockDim.x) {
        const long long r = e / width;
        const int i = (int)(e - r * width);
        const float u = gated ? in[r * ld_in + width + i] : 1.f;
        out[r * ld_out + i] = from_float<TO>(activate(act, in[r * ld_in + i], p0, p1) * u);
    }
}
}  // namespace

// residual [rows, hidden] += rms(y [rows, hidden] + bias [hidden] or nothing) * weight [hidden]; with `next`
// (next_dtype) also next = rms(residual) * next_weight.  Everything but `next` is 32-bit.
LIA_EXPORT int lia_norm_residual(const float* y, const float* bias, const float* weight, float* residual,
                                 const float* next_weight, void* next, int next_dtype, int rows, int hidden, float eps,
                                 float next_eps, cudaStream_t stream) {
    if (rows <= 0) return LIA_OK;
    if (hidden <= 0 || (next && !next_weight)) return LIA_ERR_SIZE;
    int threads = hidden >= 2048 ? 512 : hidden >= 512 ? 256 : 128;
    if (next && next_dtype != LIA_F32 && next_dtype != LIA_BF16) return LIA_ERR_DTYPE;
    const uintptr_t bits = (uintptr_t)y | (uintptr_t)bias | (uintptr_t)weight | (uintptr_t)residual | (uintptr_t)next_weight | (uintptr_t)next;
    if (hidden % 4 == 0 && (bits & 15u) == 0 && hidden <= 8192) {
        const int quads = hidden / 4;
        threads = quads <= 64 ? 64 : quads <= 128 ? 128 : quads <= 256 ? 256 : 512;
        const int per = (quads + threads - 1) / threads;
#define LIA_QUADS(TO, PER)                                                                                                  \
    return lia_launch(norm_residual_quads_kernel<TO, PER>, dim3(rows), dim3(threads), 0, stream, y, bias, weight, residual, \
                      next_weight, (TO*)next, hidden, eps, next_eps)
        if (next && next_dtype == LIA_BF16) {
            if (per == 1) LIA_QUADS(__nv_bfloat16, 1);
            if (per == 2) LIA_QUADS(__nv_bfloat16, 2);
            LIA_QUADS(__nv_bfloat16, 4);
        }
        if (per == 1) LIA_QUADS(float, 1);
        if (per == 2) LIA_QUADS(float, 2);
        LIA_QUADS(float, 4);
#undef LIA_QUADS
    }
    if (!next || next_dtype == LIA_F32)
        return lia_launch(norm_residual_kernel<float>, dim3(rows), dim3(threads), 0, stream, y, bias, weight, residual,
                          next_weight, (float*)next, rows, hidden, eps, next_eps);
    return lia_launch(norm_residual_kernel<__nv_bfloat16>, dim3(rows), dim3(threads), 0, stream, y, bias, weight, residual,
                      next_weight, (__nv_bfloat16*)next, rows, hidden, eps, next_eps);
}

// One or two terms (y1 null: one) of rows [rows, hidden], each with an optional bias [hidden] and an optional norm (weight
// [hidden], eps); residual [rows, hidden] += rms(sum of the terms) * weight; next [rows, hidden] of next_dtype or null.
LIA_EXPORT int lia_norm_terms_residual(const float* y0, const float* bias0, const float* weight0, float scale0, float eps0,
                                       const float* y1, const float* bias1, const float* weight1, float scale1, float eps1,
                                       const float* weight, float* residual, void* next, int next_dtype, int rows,
                                       int hidden, float eps, cudaStream_t stream) {
    if (rows <= 0) return LIA_OK;
    if (hidden <= 0 || !y0 || !weight) return LIA_ERR_SIZE;
    if (next && next_dtype != LIA_F32 && next_dtype != LIA_BF16) return LIA_ERR_DTYPE;
    const NormTerm a = {y0, bias0, weight0, scale0, eps0}, b = {y1, bias1, weight1, scale1, eps1};
    const uintptr_t bits = (uintptr_t)y0 | (uintptr_t)bias0 | (uintptr_t)weight0 | (uintptr_t)y1 | (uintptr_t)bias1 |
                           (uintptr_t)weight1 | (uintptr_t)weight | (uintptr_t)residual | (uintptr_t)next;
    int per = 0, threads = hidden >= 2048 ? 512 : hidden >= 512 ? 256 : 128;
    if (hidden % 4 == 0 && (bits & 15u) == 0 && hidden <= 8192) {
        const int quads = hidden / 4;
        threads = quads <= 64 ? 64 : quads <= 128 ? 128 : quads <= 256 ? 256 : 512;
        per = (quads + threads - 1) / threads;
        per = per > 2 ? 4 : per;
    }
#define LIA_TERMS(TO, TERMS, PER)                                                                                     \
    return lia_launch(norm_terms_residual_kernel<TO, TERMS, PER>, dim3(rows), dim3(threads), 0, stream, a, b, weight, \
                      residual, (TO*)next, hidden, eps)
#define LIA_TERMS_PER(TO, TERMS)                   \
    {                                              \
        if (per == 1) LIA_TERMS(TO, TERMS, 1);     \
        if (per == 2) LIA_TERMS(TO, TERMS, 2);     \
        if (per == 4) LIA_TERMS(TO, TERMS, 4);     \
        LIA_TERMS(TO, TERMS, 0);                   \
    }
    if (next && next_dtype == LIA_BF16) {
        if (y1) LIA_TERMS_PER(__nv_bfloat16, 2)
        LIA_TERMS_PER(__nv_bfloat16, 1)
    }
    if (y1) LIA_TERMS_PER(float, 2)
    LIA_TERMS_PER(float, 1)
#undef LIA_TERMS_PER
#undef LIA_TERMS
}

// out[r, i] = act(in[r, i]), i < width, or with `gated` act(in[r, i]) * in[r, width + i]; act: 0 identity, 1 GELU
// (tanh form), 2 SiLU, 3 the square of ReLU, 4 ReLU, 5 xIELU with the constants p0, p1.  Row strides in elements.
LIA_EXPORT int lia_activation_rows(const float* in, long long ld_in, void* out, int out_dtype, long long ld_out,
                                   int rows, int width, int act, int gated, float p0, float p1,
                                   cudaStream_t stream) {
    if (rows <= 0 || width <= 0) return LIA_OK;
    if (ld_in < (gated ? 2 : 1) * (long long)width || ld_out < width || act < 0 || act > 5) return LIA_ERR_SIZE;
    const bool four = width % 4 == 0 && ld_in % 4 == 0 && ld_out % 4 == 0 && ((uintptr_t)in & 15u) == 0 && ((uintptr_t)out & 15u) == 0;
    const long long total = four ? (long long)rows * (width / 4) : (long long)rows * width;
    const int blocks = (int)((total + 255) / 256 < 8192 ? (total + 255) / 256 : 8192);
#define LIA_ACT(TO)                                                                                                      \
    {                                                                                                                    \
        if (four)                                                                                                        \
            return lia_launch(activation_rows4_kernel<TO>, dim3(blocks), dim3(256), 0, stream, in, ld_in, (TO*)out,     \
                              ld_out, rows, width / 4, act, gated, p0, p1);                                                      \
        return lia_launch(activation_rows_kernel<TO>, dim3(blocks), dim3(256), 0, stream, in, ld_in, (TO*)out,          \
                          ld_out, rows, width, act, gated, p0, p1);                                                              \
    }
    if (out_dtype == LIA_F32) LIA_ACT(float)
    if (out_dtype == LIA_BF16) LIA_ACT(__nv_bfloat16)
#undef LIA_ACT
    return LIA_ERR_DTYPE;
}
