// The real-gated linear recurrent unit in a step of single tokens, from the input product's rows to the unit's output, in one
// kernel (bfloat16 weights and output): the short convolution over the ring, both gates' products, the decays, the state's
// step and the gate branch.  See rglru.cu for the recurrence and conv_ring.cuh for the ring.
//
// A CTA owns SLICE output channels of one part and up to 16 tokens.  Its rows of both gate matrices come into shared memory
// by asynchronous copies before the kernel ahead has finished (weights depend on no kernel); then it convolves the whole
// part's channels of its tokens (every slice of a part does: a few thousand multiply-adds), rounds them to bfloat16, and its
// eight warps multiply (mma.sync 16 x 8 x 16: 64 rows of the two matrices by 16 tokens).  Each slice stores its own channels'
// inputs in the ring: the row of a token's position is none of the rows that another CTA reads for it.
#include "conv_ring.cuh"

namespace {
constexpr int SLICE = 32, STEP_TOKENS = 16, STEP_THREADS = 256;

struct StepArgs {
    const float* y; const float* x; long long ld;            // the product's two branches, rows of `ld` columns
    const float* y_bias; const float* x_bias;
    const float* conv; const float* conv_bias;               // [taps, width], [width]
    const __nv_bfloat16* w_r; const __nv_bfloat16* w_i;      // [blocks, size, size], a row per output channel
    const float* bias; const float* rate;                    // [2, width], [width]
    float* ring; float* state; long long slot_stride;        // slot s: [taps, width] and [width]
    const int* positions; const int* slots;
    __nv_bfloat16* out;                                      // [n, width]
    int n_tokens, width, size, slices, taps;
};

__device__ __forceinline__ uint32_t step_address(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }

__global__ void __launch_bounds__(STEP_THREADS)
rglru_single_kernel(StepArgs p) {
    extern __shared__ __align__(16) uint8_t step_raw[];      // weights [2 SLICE][size + 8], u [STEP_TOKENS][size + 8]
    __shared__ float sums[2 * SLICE][STEP_TOKENS + 1];
    __shared__ int token_slot[STEP_TOKENS];
    __shared__ int ring_row[STEP_TOKENS][RING_MAX_TAPS];       // [j]: the ring's row of tap j's input, -1 before the start; [taps - 1]: the token's own row
    const int size = p.size, pitch = size + 8;
    __nv_bfloat16* ws = reinterpret_cast<__nv_bfloat16*>(step_raw);
    __nv_bfloat16* us = ws + 2 * SLICE * pitch;
    const int part = blockIdx.x / p.slices, o0 = (blockIdx.x % p.slices) * SLICE, t0 = blockIdx.y * STEP_TOKENS;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int pieces = size / 8;
    for (int e = tid; e < 2 * SLICE * pieces; e += STEP_THREADS) {
        const int row = e / pieces, k = (e - row * pieces) * 8, o = o0 + (row & (SLICE - 1));
        const bool there = o < size;
        const __nv_bfloat16* src = (row < SLICE ? p.w_r : p.w_i) + ((size_t)part * size + (there ? o : 0)) * size + k;
        const int bytes = there ? 16 : 0;
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(step_address(ws + row * pitch + k)), "l"(src), "r"(bytes) : "memory");
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
    if (tid < STEP_TOKENS) {                                 // (the step's metadata depends on no kernel of the step)
        const bool there = t0 + tid < p.n_tokens;
        const int pos = there ? p.positions[t0 + tid] : 0;
        token_slot[tid] = there ? p.slots[t0 + tid] : -1;
        for (int j = 0; j < p.taps; ++j) {
            const int at = pos - (p.taps - 1 - j);
            ring_row[tid][j] = at >= 0 ? at % p.taps : -1;
        }
    }
    pdl_launch_dependents();
    pdl_wait();
    __syncthreads();
    // this thread's two outputs: the state and the gate branch travel while the gates are made
    constexpr int OUTPUTS = STEP_TOKENS * SLICE / STEP_THREADS;
    float held[OUTPUTS], branch[OUTPUTS];
#pragma unroll
    for (int q = 0; q < OUTPUTS; ++q) {
        const int tok = (tid + q * STEP_THREADS) / SLICE, f = o0 + (tid & (SLICE - 1));
        const bool mine = token_slot[tok] >= 0 && f < size;
        const int c = part * size + (f < size ? f : 0);
        held[q] = mine ? p.state[(size_t)token_slot[tok] * p.slot_stride + c] : 0.f;
        branch[q] = mine ? p.y[(size_t)(t0 + tok) * p.ld + c] + p.y_bias[c] : 0.f;
    }
    // the part's convolution for these tokens, channels across the threads
    {
        const int across = size < STEP_THREADS ? size : STEP_THREADS, down = STEP_THREADS / across;
        const int row = tid / across;
        if (row < down) {
            for (int k = tid % across; k < size; k += across) {
                const int c = part * size + k;
                const float xb = p.x_bias[c], cb = p.conv_bias[c];
                float w[RING_MAX_TAPS - 1];
#pragma unroll
                for (int j = 0; j < RING_MAX_TAPS - 1; ++j) w[j] = j < p.taps - 1 ? p.conv[(size_t)j * p.width + c] : 0.f;
                const float w_own = p.conv[(size_t)(p.taps - 1) * p.width + c];
#pragma unroll 4
                for (int tok = row; tok < STEP_TOKENS; tok += down) {
                    const int slot = token_slot[tok];
                    float v = 0.f;
                    if (slot >= 0) {
                        float* ring = p.ring + (size_t)slot * p.slot_stride + c;
                        const float own = p.x[(size_t)(t0 + tok) * p.ld + c] + xb;
                        float earlier[RING_MAX_TAPS - 1];
#pragma unroll
                        for (int j = 0; j < RING_MAX_TAPS - 1; ++j) {
                            const int row = j < p.taps - 1 ? ring_row[tok][j] : -1;
                            earlier[j] = row >= 0 ? ring[(size_t)row * p.width] : 0.f;
                        }
                        v = cb;
#pragma unroll
                        for (int j = 0; j < RING_MAX_TAPS - 1; ++j) v = fmaf(j < p.taps - 1 ? w[j] : 0.f, earlier[j], v);
                        v = fmaf(w_own, own, v);
                        if (p.taps > 1 && k >= o0 && k < o0 + SLICE) ring[(size_t)ring_row[tok][p.taps - 1] * p.width] = own;
                    }
                    us[tok * pitch + k] = __float2bfloat16_rn(v);
                }
            }
        }
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    // 64 rows (r's channels, then i's) by 16 tokens: a warp 16 rows and 8 tokens
    {
        const int m0 = (warp & 3) * 16, n0 = (warp >> 2) * 8;
        float even[4] = {}, odd[4] = {};                     // two chains
        const uint32_t a_at = step_address(ws + (m0 + (lane & 15)) * pitch + (lane >> 4) * 8);
        const uint32_t b_at = step_address(us + (n0 + (lane & 7)) * pitch + ((lane >> 3) & 1) * 8);
        auto product = [&](int k, float (&c)[4]) {
            uint32_t a[4], b[2];
            asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(a[0]), "=r"(a[1]), "=r"(a[2]), "=r"(a[3]) : "r"(a_at + k * 32));
            asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0, %1}, [%2];" : "=r"(b[0]), "=r"(b[1]) : "r"(b_at + k * 32));
            asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                         : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b[0]), "r"(b[1]));
        };
        const int steps = size / 16;
#pragma unroll 2
        for (int k = 0; k + 1 < steps; k += 2) {
            product(k, even);
            product(k + 1, odd);
        }
        if (steps & 1) product(steps - 1, even);
        const int g = lane >> 2, t = (lane & 3) * 2;
        sums[m0 + g][n0 + t] = even[0] + odd[0];
        sums[m0 + g][n0 + t + 1] = even[1] + odd[1];
        sums[m0 + g + 8][n0 + t] = even[2] + odd[2];
        sums[m0 + g + 8][n0 + t + 1] = even[3] + odd[3];
    }
    __syncthreads();
#pragma unroll
    for (int q = 0; q < OUTPUTS; ++q) {
        const int tok = (tid + q * STEP_THREADS) / SLICE, channel = tid & (SLICE - 1), f = o0 + channel;
        const int slot = token_slot[tok];
        if (slot < 0 || f >= size) continue;
        const int c = part * size + f;
        const float w = -expm1f(-p.rate[c] * ring_sigmoid(sums[channel][tok] + p.bias[c]));      // 1 - a
        const float a = 1.0f - w;
        const float inflow = sqrtf(w * (1.0f + a)) * ring_sigmoid(sums[SLICE + channel][tok] + p.bias[p.width + c]) *
                             to_float(us[tok * pitch + f]);
        const float S = fmaf(a, held[q], inflow);
        p.state[(size_t)slot * p.slot_stride + c] = S;
        p.out[(size_t)(t0 + tok) * p.width + c] = __float2bfloat16_rn(S * ring_gelu_tanh(branch[q]));
    }
}

size_t step_bytes(int size) { return (size_t)(2 * SLICE + STEP_TOKENS) * (size + 8) * 2; }
}  // namespace

// 1 if the kernel takes parts of this size: a multiple of 16 whose rows fit in shared memory.
LIA_EXPORT int lia_rglru_single_accepts(int width, int blocks) {
    if (width <= 0 || blocks <= 0 || width % blocks) return 0;
    const int size = width / blocks;
    return size % 16 == 0 && step_bytes(size) <= 200 * 1024 ? 1 : 0;
}

// Every row of the step is a single token (or nobody's, slot negative).  y, x [n, ld] 32-bit, y_bias, x_bias, conv_bias, rate
// [width], conv [taps, width], bias [2, width] 32-bit; w_r, w_i bf16; ring and state: slot s at + s slot_stride; out [n, width]
// bf16.
LIA_EXPORT int lia_rglru_single(const float* y, const float* x, long long ld, const float* y_bias, const float* x_bias,
                                const float* conv, const float* conv_bias, const void* w_r, const void* w_i, const float* bias,
                                const float* rate, float* ring, float* state, long long slot_stride, const int* positions,
                                const int* slots, void* out, int n_tokens, int width, int blocks, int taps, cudaStream_t stream) {
    if (n_tokens <= 0) return LIA_OK;
    if (!lia_rglru_single_accepts(width, blocks) || taps < 1 || taps > RING_MAX_TAPS || ld < width || (taps > 1 && !ring)) return LIA_ERR_SIZE;
    if (((uintptr_t)w_r | (uintptr_t)w_i) & 15u) return LIA_ERR_ALIGN;
    const int size = width / blocks, slices = (size + SLICE - 1) / SLICE;
    StepArgs p = {y, x, ld, y_bias, x_bias, conv, conv_bias, (const __nv_bfloat16*)w_r, (const __nv_bfloat16*)w_i, bias, rate,
                  ring ? ring : state, state, slot_stride, positions, slots, (__nv_bfloat16*)out, n_tokens, width, size, slices, taps};
    static bool raised = false;
    if (!raised) {
        if (cudaFuncSetAttribute(rglru_single_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024) != cudaSuccess) return LIA_ERR_LAUNCH;
        raised = true;
    }
    const dim3 grid(blocks * slices, (n_tokens + STEP_TOKENS - 1) / STEP_TOKENS);
    if (grid.y > 65535) return LIA_ERR_SIZE;
    return lia_launch(rglru_single_kernel, grid, dim3(STEP_THREADS), step_bytes(size), stream, p);
}
