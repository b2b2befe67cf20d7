// The state-space recurrence's prompt portions on the tensor cores (bfloat16 x, B and C; see state_space.cu for the
// recurrence and for the three launches).  Chunks of 128 tokens; per (chunk, head)
//     sums    U[n, p] = sum_t B_t[n] x'_t[p],  x'_t = 2^(C_len - C_t) dt_t x_t
//     output  y_t = 2^(C_t) (C_t . S_in) + sum_(j<=t) a_tj x_j,  a_tj = (C_t . B_j) 2^(C_t - C_j) dt_j (+ D where j = t)
// B, C and x are bfloat16 as the convolution left them, so products of two of them are exact in the 32-bit accumulators.
// What is 32-bit, x', the weights a and the incoming state, enters a product as the sum of two bfloat16 numbers (the
// nearest one and the nearest one to what it misses; the rest is below 2^-17 of it), two products in place of one.  Steps,
// decays, their logarithms and powers, all sums and the state itself are 32-bit.
//
// `mma.sync` (16 x 8 x 16) and not tcgen05: the weights a are made of accumulators and used as operands at once, in the
// registers they lie in, and a head's matrices are 64 to 128 wide; eight warps own 16 rows each (tokens in the output,
// state rows in the sums) and meet nowhere after the loads.
#include "state_space.cuh"

namespace {
constexpr int TOKENS = 128, TC_THREADS = 256;

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
// two numbers as bfloat16 pairs: the nearest, and the nearest to what that misses
__device__ __forceinline__ void split_pair(float x, float y, uint32_t& hi, uint32_t& lo) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
    const __nv_bfloat162 l = __floats2bfloat162_rn(x - __low2float(h), y - __high2float(h));
    hi = *reinterpret_cast<const uint32_t*>(&h);
    lo = *reinterpret_cast<const uint32_t*>(&l);
}

// which portion and which of its chunks of TOKENS the CTA `index` serves: false when there is none
__device__ __forceinline__ bool find_tokens(const SsdArgs& p, int index, int* first_row, int* length) {
    for (int s = 0; s < p.n_segments; ++s) {
        const int count = p.segments[3 * s + 2], chunks = (count + TOKENS - 1) / TOKENS;
        if (index < chunks) {
            *first_row = p.segments[3 * s] + index * TOKENS;
            *length = min(TOKENS, count - index * TOKENS);
            return true;
        }
        index -= chunks;
    }
    return false;
}

// [TOKENS][width] of bfloat16 rows into shared memory (row stride width + 8: 16-byte aligned, an odd number of 16-byte
// pieces, so eight rows of a matrix lie in different banks), zeros behind `len` rows; asynchronous
__device__ __forceinline__ void bring_rows(__nv_bfloat16* dst, const __nv_bfloat16* src, long long ld, int len, int width) {
    const int pieces = width / 8;
    for (int e = threadIdx.x; e < TOKENS * pieces; e += TC_THREADS) {
        const int t = e / pieces, i = (e - t * pieces) * 8;
        const int bytes = t < len ? 16 : 0;
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(shared_address(dst + t * (width + 8) + i)),
                     "l"(src + (size_t)(t < len ? t : 0) * ld + i), "r"(bytes) : "memory");
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
}
__device__ __forceinline__ void rows_there() { asm volatile("cp.async.wait_group 0;" ::: "memory"); }

// steps [TOKENS] and the running sums [TOKENS] of the chunk's log2 decays, by the first four warps; `sums` [4] scratch.
// Every thread calls it; it ends with a barrier.
__device__ __forceinline__ void token_steps(const SsdArgs& p, int first, int len, int h, float* steps, float* logs, float* sums) {
    const int t = threadIdx.x, lane = t & 31, warp = t >> 5;
    float dt = 0.f, sum = 0.f;
    if (t < TOKENS) {
        if (t < len) dt = ring_softplus(p.dt[(size_t)(first + t) * p.ld_dt + h] + p.dt_bias[h]);
        sum = -p.rate[h] * dt * LOG2_E;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float before = __shfl_up_sync(0xffffffffu, sum, o);
            if (lane >= o) sum += before;
        }
        if (lane == 31) sums[warp] = sum;
    }
    __syncthreads();
    if (t < TOKENS) {
        for (int w = 0; w < warp; ++w) sum += sums[w];
        steps[t] = dt;
        logs[t] = sum;
    }
    __syncthreads();
}

template <int TILES>                                     // TILES: most 16-wide tiles of a head's size P
__global__ void __launch_bounds__(TC_THREADS)
ssd_sums_tc_kernel(SsdArgs p) {
    extern __shared__ __align__(16) uint8_t sums_raw[];  // B [TOKENS][N + 8], x [TOKENS][P + 8] (then x' near), x' rest [TOKENS][P + 8]
    __shared__ float steps[TOKENS], logs[TOKENS], scratch[4];
    pdl_launch_dependents();
    pdl_wait();
    int first, len;
    if (!find_tokens(p, blockIdx.x, &first, &len)) return;
    const int h = blockIdx.y, N = p.N, P = p.P, ns = N + 8, ps = P + 8;
    __nv_bfloat16* bs = reinterpret_cast<__nv_bfloat16*>(sums_raw);
    __nv_bfloat16* hi = bs + TOKENS * ns;
    __nv_bfloat16* lo = hi + TOKENS * ps;
    const __nv_bfloat16* rows = reinterpret_cast<const __nv_bfloat16*>(p.xbc) + (size_t)first * p.ld;
    const int g = h / (p.heads / p.groups);
    bring_rows(bs, rows + (size_t)p.heads * P + (size_t)g * N, p.ld, len, N);
    bring_rows(hi, rows + (size_t)h * P, p.ld, len, P);
    token_steps(p, first, len, h, steps, logs, scratch);
    const float total = logs[TOKENS - 1];                // (steps behind the chunk's end are zero)
    if (threadIdx.x == 0) p.totals[(size_t)blockIdx.x * p.heads + h] = total;
    rows_there();
    __syncthreads();
    for (int e = threadIdx.x; e < TOKENS * (P / 2); e += TC_THREADS) {
        const int t = e / (P / 2), i = (e - t * (P / 2)) * 2;
        const __nv_bfloat162 x = *reinterpret_cast<const __nv_bfloat162*>(hi + t * ps + i);
        const float w = steps[t] * pow2(total - logs[t]);
        uint32_t near, rest;
        split_pair(__low2float(x) * w, __high2float(x) * w, near, rest);
        *reinterpret_cast<uint32_t*>(hi + t * ps + i) = near;
        *reinterpret_cast<uint32_t*>(lo + t * ps + i) = rest;
    }
    __syncthreads();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gr = lane >> 2, tq = lane & 3;
    const int steps_k = (len + 15) / 16;
    float* U = p.sums + ((size_t)blockIdx.x * p.heads + h) * N * P;
    // a warp takes 16 state rows and (where the rows are fewer than the warps) a share of the head's columns
    const int row_tiles = N / 16, col_tiles = P / 16;
    const int shares = row_tiles >= TC_THREADS / 32 ? 1 : (TC_THREADS / 32) / row_tiles;
    const int per_share = (col_tiles + shares - 1) / shares;
    for (int unit = warp; unit < row_tiles * shares; unit += TC_THREADS / 32) {
        const int n0 = (unit % row_tiles) * 16, c_begin = (unit / row_tiles) * per_share, c_end = min(col_tiles, c_begin + per_share);
        if (c_begin >= c_end) continue;
        float acc[2 * TILES][4];
#pragma unroll
        for (int j = 0; j < 2 * TILES; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
        for (int k = 0; k < steps_k; ++k) {
            uint32_t a[4];
            ldsm4_trans(shared_address(bs + (k * 16 + (lane & 7) + (lane >> 4) * 8) * ns + n0 + ((lane >> 3) & 1) * 8), a);
#pragma unroll
            for (int c = 0; c < TILES; ++c) {
                if (c_begin + c >= c_end) break;
                uint32_t b[4], d[4];
                const int at = (k * 16 + (lane & 15)) * ps + (c_begin + c) * 16 + (lane >> 4) * 8;
                ldsm4_trans(shared_address(hi + at), b);
                ldsm4_trans(shared_address(lo + at), d);
                mma(acc[2 * c], a, b[0], b[1]);
                mma(acc[2 * c + 1], a, b[2], b[3]);
                mma(acc[2 * c], a, d[0], d[1]);
                mma(acc[2 * c + 1], a, d[2], d[3]);
            }
        }
#pragma unroll
        for (int c = 0; c < TILES; ++c) {
            if (c_begin + c >= c_end) break;
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int col = (c_begin + c) * 16 + e * 8 + tq * 2;
                *reinterpret_cast<float2*>(U + (size_t)(n0 + gr) * P + col) = make_float2(acc[2 * c + e][0], acc[2 * c + e][1]);
                *reinterpret_cast<float2*>(U + (size_t)(n0 + gr + 8) * P + col) = make_float2(acc[2 * c + e][2], acc[2 * c + e][3]);
            }
        }
    }
}

template <int TILES>
__global__ void __launch_bounds__(TC_THREADS)
ssd_output_tc_kernel(SsdArgs p) {
    // C [TOKENS][N + 8], x [TOKENS][P + 8], then B [TOKENS][N + 8] and, in the same room once the chunk's own tokens are done
    // with, the incoming state near and rest [N][P + 8] each: two CTAs an SM at the sizes of real models
    extern __shared__ __align__(16) uint8_t out_raw[];
    __shared__ float steps[TOKENS], logs[TOKENS], scratch[4];
    pdl_launch_dependents();
    pdl_wait();
    int first, len;
    if (!find_tokens(p, blockIdx.x, &first, &len)) return;
    const int h = blockIdx.y, N = p.N, P = p.P, ns = N + 8, ps = P + 8;
    __nv_bfloat16* cs = reinterpret_cast<__nv_bfloat16*>(out_raw);
    __nv_bfloat16* xs = cs + TOKENS * ns;
    __nv_bfloat16* bs = xs + TOKENS * ps;
    __nv_bfloat16* sh = bs;
    __nv_bfloat16* sl = sh + N * ps;
    const __nv_bfloat16* rows = reinterpret_cast<const __nv_bfloat16*>(p.xbc) + (size_t)first * p.ld;
    const int g = h / (p.heads / p.groups);
    bring_rows(cs, rows + (size_t)p.heads * P + (size_t)(p.groups + g) * N, p.ld, len, N);
    bring_rows(bs, rows + (size_t)p.heads * P + (size_t)g * N, p.ld, len, N);
    bring_rows(xs, rows + (size_t)h * P, p.ld, len, P);
    token_steps(p, first, len, h, steps, logs, scratch);
    rows_there();
    __syncthreads();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gr = lane >> 2, tq = lane & 3;
    const int r0 = warp * 16;
    const bool active = r0 < len;
    const int col_tiles = P / 16, k_tiles = N / 16;
    float acc[2 * TILES][4];
#pragma unroll
    for (int j = 0; j < 2 * TILES; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
    const uint32_t c_at = shared_address(cs + (r0 + (lane & 15)) * ns + (lane >> 4) * 8);
    const int t_low = r0 + gr, t_high = t_low + 8;
    const float log_low = logs[t_low], log_high = logs[t_high];
    // the chunk's own tokens up to this warp's, 32 at a time
    const float skip = p.skip[h];
    for (int j0 = 0; active && j0 < r0 + 16; j0 += 32) {
        float s[4][4];
#pragma unroll
        for (int q = 0; q < 4; ++q) s[q][0] = s[q][1] = s[q][2] = s[q][3] = 0.f;
        for (int k = 0; k < k_tiles; ++k) {
            uint32_t a[4], b[4], d[4];
            ldsm4(c_at + k * 32, a);
            const int at = (j0 + (lane & 7) + (lane >> 4) * 8) * ns + k * 16 + ((lane >> 3) & 1) * 8;
            ldsm4(shared_address(bs + at), b);
            ldsm4(shared_address(bs + at + 16 * ns), d);
            mma(s[0], a, b[0], b[1]);
            mma(s[1], a, b[2], b[3]);
            mma(s[2], a, d[0], d[1]);
            mma(s[3], a, d[2], d[3]);
        }
#pragma unroll
        for (int q = 0; q < 4; ++q)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int j = j0 + q * 8 + tq * 2 + e;
                const float step = steps[j], log_j = logs[j];
                s[q][e] = j > t_low ? 0.f : fmaf(s[q][e], step * pow2(log_low - log_j), j == t_low ? skip : 0.f);
                s[q][2 + e] = j > t_high ? 0.f : fmaf(s[q][2 + e], step * pow2(log_high - log_j), j == t_high ? skip : 0.f);
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
                if (c >= col_tiles) break;
                uint32_t b[4];
                ldsm4_trans(shared_address(xs + (j0 + half * 16 + (lane & 15)) * ps + c * 16 + (lane >> 4) * 8), b);
                mma(acc[2 * c], near, b[0], b[1]);
                mma(acc[2 * c + 1], near, b[2], b[3]);
                mma(acc[2 * c], rest, b[0], b[1]);
                mma(acc[2 * c + 1], rest, b[2], b[3]);
            }
        }
    }
    // what comes in from the chunk's start: C_t . S_in, decayed
    __syncthreads();
    const float* S = p.sums + ((size_t)blockIdx.x * p.heads + h) * N * P;
#pragma unroll 8
    for (int e = threadIdx.x; e < N * (P / 4); e += TC_THREADS) {
        const int n = e / (P / 4), i = (e - n * (P / 4)) * 4;
        const float4 v = *reinterpret_cast<const float4*>(S + (size_t)n * P + i);
        uint2 near, rest;
        split_pair(v.x, v.y, near.x, rest.x);
        split_pair(v.z, v.w, near.y, rest.y);
        *reinterpret_cast<uint2*>(sh + n * ps + i) = near;
        *reinterpret_cast<uint2*>(sl + n * ps + i) = rest;
    }
    __syncthreads();
    if (!active) return;
    const float w_low = pow2(log_low), w_high = pow2(log_high);
#pragma unroll
    for (int c = 0; c < TILES; ++c) {
        if (c >= col_tiles) break;
        float in[2][4] = {};
        for (int k = 0; k < k_tiles; ++k) {
            uint32_t a[4], b[4], d[4];
            ldsm4(c_at + k * 32, a);
            const int at = (k * 16 + (lane & 15)) * ps + c * 16 + (lane >> 4) * 8;
            ldsm4_trans(shared_address(sh + at), b);
            ldsm4_trans(shared_address(sl + at), d);
            mma(in[0], a, b[0], b[1]);
            mma(in[1], a, b[2], b[3]);
            mma(in[0], a, d[0], d[1]);
            mma(in[1], a, d[2], d[3]);
        }
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            acc[2 * c + e][0] = fmaf(w_low, in[e][0], acc[2 * c + e][0]);
            acc[2 * c + e][1] = fmaf(w_low, in[e][1], acc[2 * c + e][1]);
            acc[2 * c + e][2] = fmaf(w_high, in[e][2], acc[2 * c + e][2]);
            acc[2 * c + e][3] = fmaf(w_high, in[e][3], acc[2 * c + e][3]);
        }
    }
    float* y = p.y + (size_t)(first + r0) * p.heads * P + (size_t)h * P;
#pragma unroll
    for (int j = 0; j < 2 * TILES; ++j) {
        if (j >= 2 * col_tiles) break;
        const int col = j * 8 + tq * 2;
        if (t_low < len) *reinterpret_cast<float2*>(y + (size_t)gr * p.heads * P + col) = make_float2(acc[j][0], acc[j][1]);
        if (t_high < len) *reinterpret_cast<float2*>(y + (size_t)(gr + 8) * p.heads * P + col) = make_float2(acc[j][2], acc[j][3]);
    }
}

size_t sums_bytes(int N, int P) { return (size_t)TOKENS * ((N + 8) + 2 * (P + 8)) * 2; }
size_t output_bytes(int N, int P) {
    const size_t b = (size_t)TOKENS * (N + 8), state = (size_t)2 * N * (P + 8);
    return ((size_t)TOKENS * (N + 8 + P + 8) + (b > state ? b : state)) * 2;
}
constexpr size_t MOST_BYTES = 225 * 1024;

template <int TILES>
int launch_portions(const SsdArgs& p, int max_chunks, cudaStream_t stream) {
    static bool raised = false;
    if (!raised) {
        if (cudaFuncSetAttribute(ssd_sums_tc_kernel<TILES>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)MOST_BYTES) != cudaSuccess ||
            cudaFuncSetAttribute(ssd_output_tc_kernel<TILES>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)MOST_BYTES) != cudaSuccess)
            return LIA_ERR_LAUNCH;
        raised = true;
    }
    int code = lia_launch(ssd_sums_tc_kernel<TILES>, dim3(max_chunks, p.heads), dim3(TC_THREADS), sums_bytes(p.N, p.P), stream, p);
    if (code != LIA_OK) return code;
    const int parts = (p.N * p.P + SSD_THREADS - 1) / SSD_THREADS;
    code = lia_launch(ssd_carry_kernel, dim3(p.n_segments, p.heads, parts), dim3(SSD_THREADS), 0, stream, p, TOKENS);
    if (code != LIA_OK) return code;
    return lia_launch(ssd_output_tc_kernel<TILES>, dim3(max_chunks, p.heads), dim3(TC_THREADS), output_bytes(p.N, p.P), stream, p);
}
}  // namespace

// Most chunks that the portions of a step with `portion_tokens` tokens in `n_segments` portions are cut into.
LIA_EXPORT int lia_ssd_tc_chunks(int portion_tokens, int n_segments) {
    return n_segments > 0 ? portion_tokens / TOKENS + n_segments : 0;
}

// 1 if the kernels take these sizes: both multiples of 16, a head's size up to 128, the chunk's operands within shared memory.
LIA_EXPORT int lia_ssd_tc_accepts(int N, int P) {
    return N > 0 && P > 0 && N % 16 == 0 && P % 16 == 0 && P <= 128 && N <= SSD_MAX && output_bytes(N, P) <= MOST_BYTES ? 1 : 0;
}

// The portions alone (single tokens: lia_ssd_single).  xbc [n, ld] bfloat16, the rest as for lia_ssd; scratch:
// `lia_ssd_scratch_floats(max_chunks, ...)` words for the chunks that lia_ssd_tc_chunks gives.
LIA_EXPORT int lia_ssd_tc(const void* xbc, long long ld, const float* dt, long long ld_dt, const float* dt_bias,
                          const float* rate, const float* skip, float* state, long long slot_stride, const int* segments,
                          int n_segments, int max_chunks, const int* slots, float* y, int heads, int groups, int N, int P,
                          float* scratch, long long scratch_floats, cudaStream_t stream) {
    if (n_segments <= 0) return LIA_OK;
    if (heads <= 0 || groups <= 0 || heads % groups || !lia_ssd_tc_accepts(N, P) || ld % 8 || heads > 65535 || max_chunks <= 0 ||
        ld < (long long)heads * P + 2LL * groups * N || ld_dt < heads || slot_stride < (long long)heads * N * P || !scratch ||
        scratch_floats < (long long)max_chunks * heads * ((long long)N * P + 1))
        return LIA_ERR_SIZE;
    if (((uintptr_t)xbc | (uintptr_t)scratch | (uintptr_t)y) & 15u) return LIA_ERR_ALIGN;
    SsdArgs p = {(const float*)xbc, ld, dt, ld_dt, dt_bias, rate, skip, state, slot_stride, segments, n_segments, nullptr, slots, y,
                 scratch, scratch + (size_t)max_chunks * heads * N * P, heads, groups, N, P, 1};
    if (P <= 32) return launch_portions<2>(p, max_chunks, stream);
    if (P <= 64) return launch_portions<4>(p, max_chunks, stream);
    return launch_portions<8>(p, max_chunks, stream);
}
