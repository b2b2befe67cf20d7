// The matrix memory's prompt portions on the tensor cores (bfloat16 q, k and v; see mlstm.cuh for the recurrence inside a
// chunk and mlstm.cu for the three launches).  Chunks of 128 tokens; per (chunk, head, up to 128 value columns)
//     sums    U[i, j] = sum_t k_t[i] v'_t[j],  v'_t = exp(a_t - max a) v_t;   and sum_t exp(a_t - max a) k_t[i]
//     output  p_tj = (q_t . k_j) d^(-1/2) exp(a_j - M_t) for j <= t,   w_t = d^(-1/2) exp(m_0 - M_t)
//             o_t = (w_t S_in^T q_t + sum_j p_tj v_j) / (max(|w_t n_in . q_t + sum_j p_tj|, exp(-m_t)) + 1e-6)
// q, k and v are bfloat16 as the input product left them, so products of two of them are exact in the 32-bit accumulators.
// What is 32-bit, v', the weights p and the incoming memory, enters a product as the sum of two bfloat16 numbers (the nearest
// one and the nearest one to what it misses; the rest is below 2^-17 of it), two products in place of one.  Gates, exponents
// (pairs of 32-bit numbers), all sums and the memory itself are 32-bit.  Where a head's values are one piece its norm, the
// weight and the output gate are taken from the accumulators; where they are cut, o goes out in 32-bit rows and
// `mlstm_norm_kernel` follows.
//
// `mma.sync` (16 x 8 x 16) and not tcgen05: the weights p are made of accumulators and used as operands at once, in the
// registers they lie in, and a head's matrices are 64 to 128 wide; eight warps own 16 rows each (tokens in the output,
// key channels in the sums) and meet nowhere after the loads.
#include "mlstm.cuh"

namespace {
constexpr int TOKENS = 128;
constexpr double LOG2_E = 1.4426950408889634;

__device__ __forceinline__ uint32_t shared_address(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void ldsm4(uint32_t at, uint32_t (&r)[4]) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(at));
}
__device__ __forceinline__ void ldsm4_trans(uint32_t at, uint32_t (&r)[4]) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(at));
}
__device__ __forceinline__ void mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ float pow2(float x) {             // x <= 0; relative error about 2^-22, one factor of one term
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
// the logistic function by the hardware's exponential and division (relative error about 2^-21; the result is rounded to 16 bits)
__device__ __forceinline__ float fast_sigmoid(float v) { return __fdividef(1.0f, 1.0f + __expf(-v)); }
// two numbers as bfloat16 pairs: the nearest, and the nearest to what that misses
__device__ __forceinline__ void split_pair(float x, float y, uint32_t& hi, uint32_t& lo) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
    const __nv_bfloat162 l = __floats2bfloat162_rn(x - __low2float(h), y - __high2float(h));
    hi = *reinterpret_cast<const uint32_t*>(&h);
    lo = *reinterpret_cast<const uint32_t*>(&l);
}

// [TOKENS][width] of bfloat16 rows into shared memory (row stride width + 8: 16-byte aligned, an odd number of 16-byte
// pieces, so eight rows of a matrix lie in different banks), zeros behind `len` rows; asynchronous
__device__ __forceinline__ void bring_rows(__nv_bfloat16* dst, const __nv_bfloat16* src, long long ld, int len, int width) {
    const int pieces = width / 8;
    for (int e = threadIdx.x; e < TOKENS * pieces; e += MLSTM_THREADS) {
        const int t = e / pieces, i = (e - t * pieces) * 8;
        const int bytes = t < len ? 16 : 0;
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(shared_address(dst + t * (width + 8) + i)),
                     "l"(src + (size_t)(t < len ? t : 0) * ld + i), "r"(bytes) : "memory");
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
}
__device__ __forceinline__ void rows_there() { asm volatile("cp.async.wait_group 0;" ::: "memory"); }

// TILES: most 16-wide tiles of a piece of the values; FULL: every piece has that many (nothing then depends on the width)
template <int TILES, bool FULL>
__global__ void __launch_bounds__(MLSTM_THREADS)
mlstm_sums_tc_kernel(MlstmArgs p, int piece) {
    extern __shared__ __align__(16) uint8_t sums_raw[];  // k [TOKENS][d + 8], v [TOKENS][w + 8] (then v' near), v' rest [TOKENS][w + 8]
    __shared__ float weight[TOKENS], partial[2 * MLSTM_THREADS];
    __shared__ double scratch[2 * TOKENS / 32], highest, total;
    pdl_launch_dependents();
    pdl_wait();
    int first, len;
    bool last;
    if (!mlstm_find_chunk<TOKENS>(p, blockIdx.x, &first, &len, &last)) return;
    const int h = blockIdx.y, d = p.d, dv = p.dv, c0 = blockIdx.z * piece, w = FULL ? TILES * 16 : min(piece, dv - c0), ks = d + 8, vs = w + 8;
    __nv_bfloat16* k_s = reinterpret_cast<__nv_bfloat16*>(sums_raw);
    __nv_bfloat16* hi = k_s + TOKENS * ks;
    __nv_bfloat16* lo = hi + TOKENS * vs;
    const __nv_bfloat16* rows = reinterpret_cast<const __nv_bfloat16*>(p.qkv) + (size_t)first * p.ld;
    bring_rows(k_s, rows + (size_t)(p.heads + h) * d, p.ld, len, d);
    bring_rows(hi, rows + (size_t)2 * p.heads * d + (size_t)h * dv + c0, p.ld, len, w);
    const MlstmToken token = mlstm_tokens<TOKENS>(p, first, len, h, scratch);
    if (threadIdx.x == TOKENS - 1) {
        highest = token.top;
        total = token.total;
        if (blockIdx.z == 0) {
            p.totals[(size_t)blockIdx.x * p.heads + h] = (float)token.total;
            p.tops[(size_t)blockIdx.x * p.heads + h] = (float)(token.top + token.total);
        }
    }
    __syncthreads();
    if (threadIdx.x < TOKENS) weight[threadIdx.x] = (int)threadIdx.x < len ? expf((float)(token.a - highest)) : 0.f;
    rows_there();
    __syncthreads();
    for (int e = threadIdx.x; e < TOKENS * (w / 2); e += MLSTM_THREADS) {
        const int t = e / (w / 2), i = (e - t * (w / 2)) * 2;
        const __nv_bfloat162 x = *reinterpret_cast<const __nv_bfloat162*>(hi + t * vs + i);
        uint32_t near, rest;
        split_pair(__low2float(x) * weight[t], __high2float(x) * weight[t], near, rest);
        *reinterpret_cast<uint32_t*>(hi + t * vs + i) = near;
        *reinterpret_cast<uint32_t*>(lo + t * vs + i) = rest;
    }
    float* U = p.sums + ((size_t)blockIdx.x * p.heads + h) * ((size_t)d * dv + d);
    if (blockIdx.z == 0) {
        // the weighted keys' sum: two channels and a share of the tokens a thread
        const int pairs = d / 2, shares = MLSTM_THREADS / pairs, share = threadIdx.x / pairs, i = (threadIdx.x % pairs) * 2;
        float x = 0.f, y = 0.f;
        if (share < shares) {
            for (int t = share; t < len; t += shares) {
                const __nv_bfloat162 k = *reinterpret_cast<const __nv_bfloat162*>(k_s + t * ks + i);
                x = fmaf(weight[t], __low2float(k), x);
                y = fmaf(weight[t], __high2float(k), y);
            }
            partial[share * d + i] = x;
            partial[share * d + i + 1] = y;
        }
        __syncthreads();
        for (int c = threadIdx.x; c < d; c += MLSTM_THREADS) {
            float sum = partial[c];
            for (int r = 1; r < shares; ++r) sum += partial[r * d + c];
            U[(size_t)d * dv + c] = sum;
        }
    }
    __syncthreads();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gr = lane >> 2, tq = lane & 3;
    const int steps_k = (len + 15) / 16;
    // a warp takes 16 key channels and (where those are fewer than the warps) a share of the columns
    const int row_tiles = d / 16, col_tiles = w / 16;
    const int shares = row_tiles >= MLSTM_THREADS / 32 ? 1 : (MLSTM_THREADS / 32) / row_tiles;
    const int per_share = (col_tiles + shares - 1) / shares;
    for (int unit = warp; unit < row_tiles * shares; unit += MLSTM_THREADS / 32) {
        const int n0 = (unit % row_tiles) * 16, c_begin = (unit / row_tiles) * per_share, c_end = min(col_tiles, c_begin + per_share);
        if (c_begin >= c_end) continue;
        float acc[2 * TILES][4];
#pragma unroll
        for (int j = 0; j < 2 * TILES; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
        for (int k = 0; k < steps_k; ++k) {
            uint32_t a[4];
            ldsm4_trans(shared_address(k_s + (k * 16 + (lane & 7) + (lane >> 4) * 8) * ks + n0 + ((lane >> 3) & 1) * 8), a);
#pragma unroll
            for (int c = 0; c < TILES; ++c) {
                if (c_begin + c >= c_end) break;
                uint32_t b[4], r[4];
                const int at = (k * 16 + (lane & 15)) * vs + (c_begin + c) * 16 + (lane >> 4) * 8;
                ldsm4_trans(shared_address(hi + at), b);
                ldsm4_trans(shared_address(lo + at), r);
                mma(acc[2 * c], a, b[0], b[1]);
                mma(acc[2 * c + 1], a, b[2], b[3]);
                mma(acc[2 * c], a, r[0], r[1]);
                mma(acc[2 * c + 1], a, r[2], r[3]);
            }
        }
#pragma unroll
        for (int c = 0; c < TILES; ++c) {
            if (c_begin + c >= c_end) break;
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int col = c0 + (c_begin + c) * 16 + e * 8 + tq * 2;
                *reinterpret_cast<float2*>(U + (size_t)(n0 + gr) * dv + col) = make_float2(acc[2 * c + e][0], acc[2 * c + e][1]);
                *reinterpret_cast<float2*>(U + (size_t)(n0 + gr + 8) * dv + col) = make_float2(acc[2 * c + e][2], acc[2 * c + e][3]);
            }
        }
    }
}

template <int TILES, bool FULL>
__global__ void __launch_bounds__(MLSTM_THREADS, 2)
mlstm_output_tc_kernel(MlstmArgs p, int piece) {
    // q [TOKENS][d + 8], v [TOKENS][w + 8], then k [TOKENS][d + 8] and, in the same room once the chunk's own tokens are done
    // with, the incoming memory near and rest [d][w + 8] each
    extern __shared__ __align__(16) uint8_t out_raw[];
    __shared__ float2 a_s[TOKENS], top_s[TOKENS];
    __shared__ float start_s[TOKENS], floor_s[TOKENS], n_in[256], qn[TOKENS];
    __shared__ double scratch[2 * TOKENS / 32];
    pdl_launch_dependents();
    pdl_wait();
    int first, len;
    bool last;
    if (!mlstm_find_chunk<TOKENS>(p, blockIdx.x, &first, &len, &last)) return;
    const int slot = p.slots[first];
    if (slot < 0) return;
    const int h = blockIdx.y, d = p.d, dv = p.dv, c0 = blockIdx.z * piece, w = FULL ? TILES * 16 : min(piece, dv - c0), ds = d + 8, ws = w + 8;
    __nv_bfloat16* q_s = reinterpret_cast<__nv_bfloat16*>(out_raw);
    __nv_bfloat16* v_s = q_s + TOKENS * ds;
    __nv_bfloat16* k_s = v_s + TOKENS * ws;
    __nv_bfloat16* sh = k_s;
    __nv_bfloat16* sl = sh + d * ws;
    const __nv_bfloat16* rows = reinterpret_cast<const __nv_bfloat16*>(p.qkv) + (size_t)first * p.ld;
    bring_rows(q_s, rows + (size_t)h * d, p.ld, len, d);
    bring_rows(k_s, rows + (size_t)(p.heads + h) * d, p.ld, len, d);
    bring_rows(v_s, rows + (size_t)2 * p.heads * d + (size_t)h * dv + c0, p.ld, len, w);
    const size_t at = (size_t)blockIdx.x * p.heads + h;
    const float* S = p.sums + at * ((size_t)d * dv + d);
    const float m0 = p.starts[at];
    for (int i = threadIdx.x; i < d; i += MLSTM_THREADS) n_in[i] = S[(size_t)d * dv + i];
    const MlstmToken token = mlstm_tokens<TOKENS>(p, first, len, h, scratch);
    if (threadIdx.x < TOKENS) {
        const int t = threadIdx.x;
        const double top = fmax((double)m0, token.top);
        a_s[t] = mlstm_pair(token.a * LOG2_E);
        top_s[t] = mlstm_pair(top * LOG2_E);
        start_s[t] = expf((float)((double)m0 - top)) * p.q_scale;
        floor_s[t] = expf(-(float)(token.total + top));
        if (last && t == len - 1 && blockIdx.z == 0)
            p.state[(size_t)slot * p.slot_stride + (size_t)p.heads * ((size_t)d * dv + d) + h] = fmaxf(m0 + p.totals[at], p.tops[at]);
    }
    rows_there();
    __syncthreads();
    {   // n_in . q_t: two threads a token
        const int t = threadIdx.x >> 1, half = threadIdx.x & 1;
        float sum = 0.f;
        for (int i = half * 2; i < d; i += 4) {
            const __nv_bfloat162 q = *reinterpret_cast<const __nv_bfloat162*>(q_s + t * ds + i);
            sum = fmaf(__low2float(q), n_in[i], fmaf(__high2float(q), n_in[i + 1], sum));
        }
        sum += __shfl_xor_sync(0xffffffffu, sum, 1);
        if (half == 0) qn[t] = sum;
    }
    __syncthreads();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gr = lane >> 2, tq = lane & 3;
    const int r0 = warp * 16;
    const bool active = r0 < len;
    const int col_tiles = w / 16, k_tiles = d / 16;
    float acc[2 * TILES][4];
#pragma unroll
    for (int j = 0; j < 2 * TILES; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
    const uint32_t q_at = shared_address(q_s + (r0 + (lane & 15)) * ds + (lane >> 4) * 8);
    const int t_low = r0 + gr, t_high = t_low + 8;
    const float2 top_low = top_s[t_low], top_high = top_s[t_high];
    float dot_low = 0.f, dot_high = 0.f;                 // this lane's part of sum_j p_tj
    // the chunk's own tokens up to this warp's, 32 at a time
    for (int j0 = 0; active && j0 < r0 + 16; j0 += 32) {
        float s[4][4];
#pragma unroll
        for (int q = 0; q < 4; ++q) s[q][0] = s[q][1] = s[q][2] = s[q][3] = 0.f;
        for (int k = 0; k < k_tiles; ++k) {
            uint32_t a[4], b[4], c[4];
            ldsm4(q_at + k * 32, a);
            const int k_at = (j0 + (lane & 7) + (lane >> 4) * 8) * ds + k * 16 + ((lane >> 3) & 1) * 8;
            ldsm4(shared_address(k_s + k_at), b);
            ldsm4(shared_address(k_s + k_at + 16 * ds), c);
            mma(s[0], a, b[0], b[1]);
            mma(s[1], a, b[2], b[3]);
            mma(s[2], a, c[0], c[1]);
            mma(s[3], a, c[2], c[3]);
        }
#pragma unroll
        for (int q = 0; q < 4; ++q)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int j = j0 + q * 8 + tq * 2 + e;
                const float2 a_j = a_s[j];
                s[q][e] = j > t_low ? 0.f : s[q][e] * p.q_scale * pow2(mlstm_difference(a_j, top_low));
                s[q][2 + e] = j > t_high ? 0.f : s[q][2 + e] * p.q_scale * pow2(mlstm_difference(a_j, top_high));
                dot_low += s[q][e];
                dot_high += s[q][2 + e];
            }
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            uint32_t near[4], rest[4];
#pragma unroll
            for (int q = 0; q < 2; ++q) {
                split_pair(s[2 * half + q][0], s[2 * half + q][1], near[2 * q], rest[2 * q]);
                split_pair(s[2 * half + q][2], s[2 * half + q][3], near[2 * q + 1], rest[2 * q + 1]);
            }
#pragma unroll
            for (int c = 0; c < TILES; ++c) {
                if (!FULL && c >= col_tiles) break;
                uint32_t b[4];
                ldsm4_trans(shared_address(v_s + (j0 + half * 16 + (lane & 15)) * ws + c * 16 + (lane >> 4) * 8), b);
                mma(acc[2 * c], near, b[0], b[1]);
                mma(acc[2 * c + 1], near, b[2], b[3]);
                mma(acc[2 * c], rest, b[0], b[1]);
                mma(acc[2 * c + 1], rest, b[2], b[3]);
            }
        }
    }
    // what comes in from the chunk's start: S_in^T q_t
    __syncthreads();
#pragma unroll 8
    for (int e = threadIdx.x; e < d * (w / 4); e += MLSTM_THREADS) {
        const int n = e / (w / 4), i = (e - n * (w / 4)) * 4;
        const float4 v = *reinterpret_cast<const float4*>(S + (size_t)n * dv + c0 + i);
        uint2 near, rest;
        split_pair(v.x, v.y, near.x, rest.x);
        split_pair(v.z, v.w, near.y, rest.y);
        *reinterpret_cast<uint2*>(sh + n * ws + i) = near;
        *reinterpret_cast<uint2*>(sl + n * ws + i) = rest;
    }
    __syncthreads();
    if (!active) return;
    const float w_low = start_s[t_low], w_high = start_s[t_high];
#pragma unroll
    for (int c = 0; c < TILES; ++c) {
        if (!FULL && c >= col_tiles) break;
        float in[2][4] = {};
        for (int k = 0; k < k_tiles; ++k) {
            uint32_t a[4], b[4], r[4];
            ldsm4(q_at + k * 32, a);
            const int s_at = (k * 16 + (lane & 15)) * ws + c * 16 + (lane >> 4) * 8;
            ldsm4_trans(shared_address(sh + s_at), b);
            ldsm4_trans(shared_address(sl + s_at), r);
            mma(in[0], a, b[0], b[1]);
            mma(in[1], a, b[2], b[3]);
            mma(in[0], a, r[0], r[1]);
            mma(in[1], a, r[2], r[3]);
        }
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            acc[2 * c + e][0] = fmaf(w_low, in[e][0], acc[2 * c + e][0]);
            acc[2 * c + e][1] = fmaf(w_low, in[e][1], acc[2 * c + e][1]);
            acc[2 * c + e][2] = fmaf(w_high, in[e][2], acc[2 * c + e][2]);
            acc[2 * c + e][3] = fmaf(w_high, in[e][3], acc[2 * c + e][3]);
        }
    }
    dot_low += __shfl_xor_sync(0xffffffffu, dot_low, 1);
    dot_high += __shfl_xor_sync(0xffffffffu, dot_high, 1);
    dot_low += __shfl_xor_sync(0xffffffffu, dot_low, 2);
    dot_high += __shfl_xor_sync(0xffffffffu, dot_high, 2);
    const float inv_low = 1.0f / (fmaxf(fabsf(fmaf(w_low, qn[t_low], dot_low)), floor_s[t_low]) + 1e-6f);
    const float inv_high = 1.0f / (fmaxf(fabsf(fmaf(w_high, qn[t_high], dot_high)), floor_s[t_high]) + 1e-6f);
    float sq_low = 0.f, sq_high = 0.f;
#pragma unroll
    for (int j = 0; j < 2 * TILES; ++j) {
        if (!FULL && j >= 2 * col_tiles) break;
        acc[j][0] *= inv_low, acc[j][1] *= inv_low, acc[j][2] *= inv_high, acc[j][3] *= inv_high;
        sq_low = fmaf(acc[j][0], acc[j][0], fmaf(acc[j][1], acc[j][1], sq_low));
        sq_high = fmaf(acc[j][2], acc[j][2], fmaf(acc[j][3], acc[j][3], sq_high));
    }
    if (gridDim.z > 1) {                                 // the head is cut: its norm follows
        float* y = p.y + ((size_t)(first + r0) * p.heads + h) * dv + c0;
        const size_t down = (size_t)p.heads * dv;
#pragma unroll
        for (int j = 0; j < 2 * TILES; ++j) {
            if (!FULL && j >= 2 * col_tiles) break;
            const int col = j * 8 + tq * 2;
            if (t_low < len) *reinterpret_cast<float2*>(y + gr * down + col) = make_float2(acc[j][0], acc[j][1]);
            if (t_high < len) *reinterpret_cast<float2*>(y + (gr + 8) * down + col) = make_float2(acc[j][2], acc[j][3]);
        }
        return;
    }
    sq_low += __shfl_xor_sync(0xffffffffu, sq_low, 1);
    sq_high += __shfl_xor_sync(0xffffffffu, sq_high, 1);
    sq_low += __shfl_xor_sync(0xffffffffu, sq_low, 2);
    sq_high += __shfl_xor_sync(0xffffffffu, sq_high, 2);
    const float norm_low = 1.0f / sqrtf(sq_low / (float)dv + p.eps), norm_high = 1.0f / sqrtf(sq_high / (float)dv + p.eps);
    const float* weights = p.norm_weight + (size_t)h * dv + tq * 2;
    // (rows behind the chunk's end read the gate of the chunk's first token and write nothing)
    const float* g_low = p.gates + (size_t)(first + (t_low < len ? t_low : 0)) * p.ld_g + (size_t)h * dv + tq * 2;
    const float* g_high = p.gates + (size_t)(first + (t_high < len ? t_high : 0)) * p.ld_g + (size_t)h * dv + tq * 2;
    __nv_bfloat16* out_low = reinterpret_cast<__nv_bfloat16*>(p.out) + ((size_t)(first + t_low) * p.heads + h) * dv + tq * 2;
    __nv_bfloat16* out_high = out_low + (size_t)8 * p.heads * dv;
    constexpr int BATCH = 4;                             // (the loads of four columns' tiles are in flight together)
#pragma unroll
    for (int j0 = 0; j0 < 2 * TILES; j0 += BATCH) {
        if (!FULL && j0 >= 2 * col_tiles) break;
        float2 f[BATCH], low[BATCH], high[BATCH];
#pragma unroll
        for (int k = 0; k < BATCH; ++k) {
            if (!FULL && j0 + k >= 2 * col_tiles) break;
            f[k] = *reinterpret_cast<const float2*>(weights + (j0 + k) * 8);
            low[k] = *reinterpret_cast<const float2*>(g_low + (j0 + k) * 8);
            high[k] = *reinterpret_cast<const float2*>(g_high + (j0 + k) * 8);
        }
#pragma unroll
        for (int k = 0; k < BATCH; ++k) {
            const int j = j0 + k;
            if (!FULL && j >= 2 * col_tiles) break;
            if (t_low < len)
                *reinterpret_cast<__nv_bfloat162*>(out_low + j * 8) = __floats2bfloat162_rn(
                    acc[j][0] * norm_low * f[k].x * fast_sigmoid(low[k].x), acc[j][1] * norm_low * f[k].y * fast_sigmoid(low[k].y));
            if (t_high < len)
                *reinterpret_cast<__nv_bfloat162*>(out_high + j * 8) = __floats2bfloat162_rn(
                    acc[j][2] * norm_high * f[k].x * fast_sigmoid(high[k].x), acc[j][3] * norm_high * f[k].y * fast_sigmoid(high[k].y));
        }
    }
}

// a cut head's norm, weight and gate for the portions' tokens: a warp a (token, head)
__global__ void __launch_bounds__(MLSTM_THREADS)
mlstm_norm_kernel(MlstmArgs p) {
    pdl_launch_dependents();
    pdl_wait();
    int first, len;
    bool last;
    if (!mlstm_find_chunk<TOKENS>(p, blockIdx.x, &first, &len, &last)) return;
    if (p.slots[first] < 0) return;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, h = blockIdx.y, dv = p.dv;
    const int t = blockIdx.z * (MLSTM_THREADS / 32) + warp;
    if (t >= len) return;
    const size_t row = ((size_t)(first + t) * p.heads + h) * dv;
    float sum = 0.f;
    for (int j = lane; j < dv; j += 32) sum = fmaf(p.y[row + j], p.y[row + j], sum);
    const float inv = 1.0f / sqrtf(warp_sum(sum) / (float)dv + p.eps);
    const float* g = p.gates + (size_t)(first + t) * p.ld_g + (size_t)h * dv;
    __nv_bfloat16* dst = reinterpret_cast<__nv_bfloat16*>(p.out) + row;
    for (int j = lane; j < dv; j += 32)
        dst[j] = from_float<__nv_bfloat16>(p.y[row + j] * inv * p.norm_weight[(size_t)h * dv + j] * mlstm_sigmoid(g[j]));
}

size_t sums_bytes(int d, int w) { return (size_t)TOKENS * ((d + 8) + 2 * (w + 8)) * 2; }
size_t output_bytes(int d, int w) {
    const size_t k = (size_t)TOKENS * (d + 8), memory = (size_t)2 * d * (w + 8);
    return ((size_t)TOKENS * (d + 8 + w + 8) + (k > memory ? k : memory)) * 2;
}
constexpr size_t MOST_BYTES = 218 * 1024;                // beside the kernels' own shared arrays

// Value columns of a head that one CTA takes: all of them up to 128, pieces of 128, 64, 32 or 16 (what shared memory holds) else.
int piece_of(int d, int dv) {
    if (dv <= 128 && output_bytes(d, dv) <= MOST_BYTES && sums_bytes(d, dv) <= MOST_BYTES) return dv;
    for (int w = 128; w >= 16; w /= 2)
        if (w < dv && output_bytes(d, w) <= MOST_BYTES && sums_bytes(d, w) <= MOST_BYTES) return w;
    return 0;
}

template <int TILES, bool FULL>
int launch_portions(const MlstmArgs& p, int piece, int max_chunks, bool four, cudaStream_t stream) {
    static bool raised = false;
    if (!raised) {
        if (cudaFuncSetAttribute(mlstm_sums_tc_kernel<TILES, FULL>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)MOST_BYTES) != cudaSuccess ||
            cudaFuncSetAttribute(mlstm_output_tc_kernel<TILES, FULL>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)MOST_BYTES) != cudaSuccess)
            return LIA_ERR_LAUNCH;
        raised = true;
    }
    const dim3 grid(max_chunks, p.heads, (p.dv + piece - 1) / piece);
    int code = lia_launch(mlstm_sums_tc_kernel<TILES, FULL>, grid, dim3(MLSTM_THREADS), sums_bytes(p.d, piece), stream, p, piece);
    if (code != LIA_OK) return code;
    code = mlstm_launch_carry(p, TOKENS, four, stream);
    if (code != LIA_OK) return code;
    code = lia_launch(mlstm_output_tc_kernel<TILES, FULL>, grid, dim3(MLSTM_THREADS), output_bytes(p.d, piece), stream, p, piece);
    if (code != LIA_OK || grid.z == 1) return code;
    return lia_launch(mlstm_norm_kernel, dim3(max_chunks, p.heads, TOKENS / (MLSTM_THREADS / 32)), dim3(MLSTM_THREADS), 0, stream, p);
}
}  // namespace

// Most chunks that the portions of a step with `portion_tokens` tokens in `n_segments` portions are cut into.
LIA_EXPORT int lia_mlstm_tc_chunks(int portion_tokens, int n_segments) {
    return n_segments > 0 ? portion_tokens / TOKENS + n_segments : 0;
}

// How many pieces a head's values are cut into; 0: the kernels do not take the sizes (both must be multiples of 16, keys up
// to 256, values up to 512).
LIA_EXPORT int lia_mlstm_tc_pieces(int d, int dv) {
    if (d <= 0 || dv <= 0 || d % 16 || dv % 16 || d > 256 || dv > MLSTM_MAX) return 0;
    const int piece = piece_of(d, dv);
    return piece ? (dv + piece - 1) / piece : 0;
}

// The portions alone (single tokens: lia_mlstm_single).  qkv [n, ld] and out [n, heads dv] bfloat16; y [n, heads dv] 32-bit
// where lia_mlstm_tc_pieces is more than 1 (else it may be null); the rest as for lia_mlstm, chunks as lia_mlstm_tc_chunks says.
LIA_EXPORT int lia_mlstm_tc(const void* qkv, long long ld, const float* gates, long long ld_g, const float* i_bias,
                            const float* f_bias, float cap, float* state, long long slot_stride, const int* segments, int n_segments,
                            int max_chunks, const int* slots, const float* norm_weight, float eps, void* out, float* y, int heads,
                            int d, int dv, float* scratch, long long scratch_floats, cudaStream_t stream) {
    if (n_segments <= 0) return LIA_OK;
    const int pieces = lia_mlstm_tc_pieces(d, dv);
    if (pieces == 0 || heads <= 0 || heads > 65535 || !(cap > 0.f) || ld < (long long)heads * (2 * d + dv) || ld % 8 ||
        ld_g < (long long)heads * (dv + 2) || slot_stride < (long long)heads * ((long long)d * dv + d + 1) || max_chunks <= 0 ||
        !scratch || scratch_floats < mlstm_scratch_words(max_chunks, heads, d, dv) || (pieces > 1 && !y))
        return LIA_ERR_SIZE;
    if ((((uintptr_t)qkv | (uintptr_t)scratch | (uintptr_t)y | (uintptr_t)out) & 15u) || (((uintptr_t)gates | (uintptr_t)norm_weight) & 7u) || ld_g % 2)
        return LIA_ERR_ALIGN;
    MlstmArgs p = {};
    p.qkv = qkv; p.ld = ld; p.qkv_bf16 = 1; p.gates = gates; p.ld_g = ld_g; p.i_bias = i_bias; p.f_bias = f_bias; p.cap = cap;
    p.state = state; p.slot_stride = slot_stride; p.segments = segments; p.n_segments = n_segments; p.slots = slots;
    p.norm_weight = norm_weight; p.eps = eps; p.out = out; p.y = y; p.heads = heads; p.d = d; p.dv = dv; p.vec = 1;
    p.q_scale = 1.0f / sqrtf((float)d);
    mlstm_place_scratch(p, scratch, max_chunks);
    const bool four = slot_stride % 4 == 0 && ((uintptr_t)state & 15u) == 0;
    const int piece = piece_of(d, dv);
#define LIA_PORTIONS(TILES)                                                                                            \
    return piece == 16 * TILES && dv % piece == 0 ? launch_portions<TILES, true>(p, piece, max_chunks, four, stream)  \
                                                  : launch_portions<TILES, false>(p, piece, max_chunks, four, stream)
    if (piece <= 32) LIA_PORTIONS(2);
    if (piece <= 64) LIA_PORTIONS(4);
    LIA_PORTIONS(8);
#undef LIA_PORTIONS
}
