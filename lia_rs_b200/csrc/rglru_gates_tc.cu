// The gates of the real-gated linear recurrent unit on the 5th-generation tensor cores (bfloat16 u and weights, 32-bit sums):
//     r = sigmoid(Wr_b u_b + br),  i = sigmoid(Wi_b u_b + bi)        for each of `blocks` equal parts of the channels
//     a = exp(-rate r),  inflow = sqrt(1 - a^2) i u
// A CTA owns 128 output channels of one part and `n_tile` tokens: two accumulators in TMEM (r's and i's), channels down the
// lanes, tokens across the columns, so that a thread has both gates of its channel and a warp's stores of a token are
// neighbours.  Warp 0 brings K blocks of 64 of both matrices and of u by TMA through a ring of two stages, warp 1 issues
// the MMAs, warps 2..9 (two a quarter of the lanes, each half of the tokens) turn the sums into a and the inflow.  Two CTAs
// share an SM: one's loads and MMAs run under the other's epilogue, which is what bounds the kernel (some fifty
// instructions an element).
// K beyond a part's size: the weights' rows end there (TMA fills zeros), so whatever u holds behind the part (the next
// part's channels, finite) counts for nothing.  Rows of a channel tile beyond the part are computed and not stored.
// 1 - a is taken as w = -expm1(log a) and 1 - a^2 as w (1 + a): no cancellation where a is close to one.
#include "conv_ring.cuh"
#include "tcgen05.cuh"

using namespace tc5;

namespace {
constexpr int EPILOGUE_WARPS = 8;
constexpr int GATES_THREADS = (2 + EPILOGUE_WARPS) * 32;
constexpr int GATES_STAGES = 2;

struct GatesArgs {
    const __nv_bfloat16* u;          // [n, width]
    const float* bias;               // [2, width]
    const float* rate;               // [width]
    const int* slots;
    float* a_out; float* inflow;     // [n, width]
    int n_tokens, width, size, n_tile, kblocks, tmem_cols;
    int* error_flag;
};

__device__ __forceinline__ float fast_sigmoid(float v) { return __fdividef(1.0f, 1.0f + __expf(-v)); }
// 1 - e^x for x <= 0: near zero the exponential's series to x^7 (what is left out is below 2^-28 of the sum), else as it stands
__device__ __forceinline__ float one_minus_exp(float x) {
    float s = fmaf(x, 1.0f / 7.0f, 1.0f);
    s = fmaf(x * s, 1.0f / 6.0f, 1.0f);
    s = fmaf(x * s, 0.2f, 1.0f);
    s = fmaf(x * s, 0.25f, 1.0f);
    s = fmaf(x * s, 1.0f / 3.0f, 1.0f);
    s = fmaf(x * s, 0.5f, 1.0f);
    return x > -0.25f ? -x * s : 1.0f - __expf(x);
}
__device__ __forceinline__ float fast_sqrt(float v) {
    float y;
    asm("sqrt.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(v));
    return y;
}

__global__ void __launch_bounds__(GATES_THREADS, 2)
rglru_gates_tc_kernel(const __grid_constant__ CUtensorMap map_r, const __grid_constant__ CUtensorMap map_i,
                      const __grid_constant__ CUtensorMap map_u, GatesArgs p) {
    extern __shared__ __align__(1024) uint8_t smem_raw[];
    __shared__ __align__(8) uint64_t full_bar[GATES_STAGES], empty_bar[GATES_STAGES], acc_full;
    __shared__ uint32_t tmem_base_slot;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    constexpr uint32_t W_BYTES = TILE_F * BLOCK_K * 2;
    const uint32_t stage_bytes = 2 * W_BYTES + (uint32_t)p.n_tile * BLOCK_K * 2;
    const uint32_t smem_base = (smem_u32(smem_raw) + 1023u) & ~1023u;
    const int t0 = blockIdx.x * p.n_tile, f0 = blockIdx.y * TILE_F, block = blockIdx.z;
    const int row0 = block * p.size + f0;                 // first row of the matrices, and first channel of the outputs

    if (warp == 0 && lane == 0) {
        for (int i = 0; i < GATES_STAGES; ++i) {
            mbar_init(smem_u32(&full_bar[i]), 1);
            mbar_init(smem_u32(&empty_bar[i]), 1);
        }
        mbar_init(smem_u32(&acc_full), 1);
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        fence_async_smem();
    }
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&tmem_base_slot)),
                     "r"((uint32_t)p.tmem_cols)
                     : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem_base = tmem_base_slot;
    pdl_launch_dependents();

    if (warp == 0 && lane == 0) {
        // ---- TMA producer: the first ring of weights is asked for before the kernel ahead has finished ----
        bool ok = true;
        const int ahead = p.kblocks < GATES_STAGES ? p.kblocks : GATES_STAGES;
        for (int kb = 0; kb < ahead; ++kb) {
            const uint32_t full = smem_u32(&full_bar[kb]), dst = smem_base + (uint32_t)kb * stage_bytes;
            mbar_expect_tx(full, stage_bytes);
            tma_load_2d(dst, &map_r, kb * BLOCK_K, row0, full);
            tma_load_2d(dst + W_BYTES, &map_i, kb * BLOCK_K, row0, full);
        }
        pdl_wait();
        int issued = 0;
        for (int kb = 0; kb < p.kblocks; ++kb) {
            const int st = kb % GATES_STAGES;
            const uint32_t full = smem_u32(&full_bar[st]), dst = smem_base + (uint32_t)st * stage_bytes;
            if (kb >= ahead) {
                if (!mbar_wait(smem_u32(&empty_bar[st]), ((uint32_t)(kb / GATES_STAGES) & 1u) ^ 1u)) { ok = false; break; }
                mbar_expect_tx(full, stage_bytes);
                tma_load_2d(dst, &map_r, kb * BLOCK_K, row0, full);
                tma_load_2d(dst + W_BYTES, &map_i, kb * BLOCK_K, row0, full);
            }
            // (the part's first column is a multiple of 8 elements, 16 bytes: the caller has checked the part's size)
            tma_load_2d(dst + 2 * W_BYTES, &map_u, block * p.size + kb * BLOCK_K, t0, full);
            issued = kb + 1;
        }
        if (!ok) {
            if (p.error_flag) atomicExch(p.error_flag, 3);
            for (int kb = max(0, issued - GATES_STAGES); kb < issued; ++kb)      // the copies that may still be in flight
                mbar_wait(smem_u32(&full_bar[kb % GATES_STAGES]), (uint32_t)(kb / GATES_STAGES) & 1u);
        }
    } else if (warp == 1 && lane == 0) {
        // ---- MMA issuer ----
        const uint32_t idesc = instr_desc(TILE_F, p.n_tile);
        const uint64_t desc_r0 = smem_desc(smem_base), desc_i0 = smem_desc(smem_base + W_BYTES), desc_u0 = smem_desc(smem_base + 2 * W_BYTES);
        bool ok = true;
        for (int kb = 0; kb < p.kblocks; ++kb) {
            const int st = kb % GATES_STAGES;
            if (!mbar_wait(smem_u32(&full_bar[st]), (uint32_t)(kb / GATES_STAGES) & 1u)) { ok = false; break; }
            tc_fence_after();
            const uint64_t stage = (uint64_t)((uint32_t)st * (stage_bytes >> 4));
#pragma unroll
            for (int k = 0; k < BLOCK_K / 16; ++k) {
                const uint32_t accumulate = (kb > 0 || k > 0) ? 1u : 0u;
                tc_mma(tmem_base, desc_r0 + stage + 2 * k, desc_u0 + stage + 2 * k, idesc, accumulate);
                tc_mma(tmem_base + (uint32_t)p.n_tile, desc_i0 + stage + 2 * k, desc_u0 + stage + 2 * k, idesc, accumulate);
            }
            tc_commit(smem_u32(&empty_bar[st]));
        }
        if (ok) tc_commit(smem_u32(&acc_full));
        else if (p.error_flag) atomicExch(p.error_flag, 3);
    } else if (warp >= 2) {
        // ---- epilogue: warp w reads TMEM lanes 32 * (w % 4) .. + 31 ----
        const int quarter = warp & 3, half = (warp - 2) >> 2;
        const int f = f0 + quarter * 32 + lane;
        const bool live = f < p.size;
        const int c = block * p.size + (live ? f : 0);
        const float rate = p.rate[c], br = p.bias[c], bi = p.bias[p.width + c];
        pdl_wait();
        if (mbar_wait(smem_u32(&acc_full), 0u)) {
            tc_fence_after();
            const uint32_t at = tmem_base + ((uint32_t)(quarter * 32) << 16);
            const int span = p.n_tile / 2;
            for (int c0 = half * span; c0 < (half + 1) * span; c0 += 16) {
                if (t0 + c0 >= p.n_tokens) break;
                float r[16], i[16];
                tmem_load16(at + (uint32_t)c0, r);
                tmem_load16(at + (uint32_t)(p.n_tile + c0), i);
                if (!live) continue;
                const int there = min(16, p.n_tokens - (t0 + c0));
                const size_t first = (size_t)(t0 + c0) * p.width + c;
                float u[16];
#pragma unroll
                for (int k = 0; k < 16; ++k) u[k] = k < there ? to_float(p.u[first + (size_t)k * p.width]) : 0.f;
#pragma unroll
                for (int k = 0; k < 16; ++k) {
                    const float w = one_minus_exp(-rate * fast_sigmoid(r[k] + br));
                    const float a = 1.0f - w;
                    r[k] = a;
                    i[k] = fast_sqrt(w * (1.0f + a)) * fast_sigmoid(i[k] + bi) * u[k];
                }
#pragma unroll
                for (int k = 0; k < 16; ++k)
                    if (k < there) {
                        p.a_out[first + (size_t)k * p.width] = r[k];
                        p.inflow[first + (size_t)k * p.width] = i[k];
                    }
            }
            tc_fence_before();
        } else if (lane == 0 && p.error_flag) {
            atomicExch(p.error_flag, 3);
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 1) {
        tc_fence_after();
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_base), "r"((uint32_t)p.tmem_cols) : "memory");
    }
}
}  // namespace

// 1 if the kernel takes parts of this size (16-byte aligned TMA boxes; u and the matrices 16-byte aligned).
LIA_EXPORT int lia_rglru_gates_tc_accepts(int width, int blocks) {
    if (width <= 0 || blocks <= 0 || width % blocks || blocks > 65535) return 0;
    return (width / blocks) % 8 == 0 ? 1 : 0;
}

// u [n, width] bf16; w_r, w_i [blocks * size, size] bf16 (rows: output channels); bias [2, width], rate [width] 32-bit;
// a_out, inflow [n, width] 32-bit.
LIA_EXPORT int lia_rglru_gates_tc(const void* u, const void* w_r, const void* w_i, const float* bias, const float* rate,
                                  const int* slots, float* a_out, float* inflow, int n_tokens, int width, int blocks,
                                  int sm_count, int* error_flag, cudaStream_t stream) {
    if (n_tokens <= 0) return LIA_OK;
    if (!lia_rglru_gates_tc_accepts(width, blocks) || sm_count <= 0) return LIA_ERR_SIZE;
    GatesArgs p;
    p.u = (const __nv_bfloat16*)u; p.bias = bias; p.rate = rate; p.slots = slots; p.a_out = a_out; p.inflow = inflow;
    p.n_tokens = n_tokens; p.width = width; p.size = width / blocks; p.error_flag = error_flag;
    p.kblocks = (p.size + BLOCK_K - 1) / BLOCK_K;
    const int f_tiles = (p.size + TILE_F - 1) / TILE_F;
    p.n_tile = 64;                                      // as wide as still gives every SM a CTA, 32 at least
    while (p.n_tile > 32 && (long long)((n_tokens + p.n_tile - 1) / p.n_tile) * f_tiles * blocks < sm_count) p.n_tile /= 2;
    p.tmem_cols = 2 * p.n_tile;                         // 64, 128 or 256: two CTAs an SM fit
    CUtensorMap mr, mi, mu;
    int rc;
    if ((rc = make_map(&mr, w_r, blocks * p.size, p.size, p.size, TILE_F)) != LIA_OK) return rc;
    if ((rc = make_map(&mi, w_i, blocks * p.size, p.size, p.size, TILE_F)) != LIA_OK) return rc;
    if ((rc = make_map(&mu, u, n_tokens, width, width, p.n_tile)) != LIA_OK) return rc;
    const size_t smem = (size_t)GATES_STAGES * (2 * TILE_F + p.n_tile) * BLOCK_K * 2 + 1024;
    static bool configured = false;
    if (!configured) {
        if (cudaFuncSetAttribute(rglru_gates_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 100 * 1024) != cudaSuccess)
            return LIA_ERR_LAUNCH;
        configured = true;
    }
    const dim3 grid((n_tokens + p.n_tile - 1) / p.n_tile, f_tiles, blocks);
    return lia_launch(rglru_gates_tc_kernel, grid, dim3(GATES_THREADS), smem, stream, mr, mi, mu, p);
}
