// A matrix memory with exponential gates per head (mLSTM of xLSTM); the recurrence and its form inside a chunk: mlstm.cuh.
//
//     log gates   i = cap tanh((W_i x + b_i) / cap),  f = log sigmoid(cap tanh((W_f x + b_f) / cap))
//     out_t = o_t / sqrt(mean(o_t^2) + eps) * w * sigmoid(g_t)      (per head over its dv elements; w [heads dv])
//
// q (times d^(-1/2)), k and v come as one set of rows [q | k | v], the output gate's and the two log gates' products as
// another [g | i | f], 32-bit (both may be columns of one product's rows).
//  * Single tokens (`mlstm_single`): one CTA per (token, head), or a cluster of CTAs that share the head's value columns
//    and meet for its norm, updates the memory in place and forms the output from it.
//  * Prompt portions are cut into chunks that run side by side, in three launches:
//      sums    U_c = sum_j exp(a_j - max a) k_j v_j^T of each chunk and the same sum of k_j, with F of the chunk and
//              max a + F (the largest exponent, counted from the chunk's end);
//      carry   along each portion: the memory that each chunk starts from takes U_c's place, the last goes to the state;
//      output  o_t from the chunk's start and from the chunk's own tokens, then the head's norm, its weight and the gate.
//    The kernels here have chunks of 32 tokens on the 32-bit pipes, any head sizes up to 512; mlstm_tc.cu has chunks of
//    128 tokens on the tensor cores.
// Gates, exponents, the memory, every sum and the norm are 32-bit (exponents of a chunk: two 32-bit numbers each).  A row
// whose slot is negative belongs to nobody and is skipped.
#include "linear_recurrence.cuh"
#include "mlstm.cuh"

namespace {
// the first 32 lanes' numbers of a chunk, shared
struct ChunkShared {
    float2 a[CHUNK], top[CHUNK];
    float weight[CHUNK], start[CHUNK], floor_[CHUNK], below[CHUNK];
    float total, highest;
};

__global__ void __launch_bounds__(MLSTM_THREADS)
mlstm_sums_kernel(MlstmArgs p) {
    extern __shared__ float mlstm_sums_shared[];          // k [CHUNK][dp], v [CHUNK][dvp] weighted
    __shared__ float weight[CHUNK];
    __shared__ double scratch[2];
    pdl_launch_dependents();
    pdl_wait();
    int first, len;
    bool last;
    if (!mlstm_find_chunk<CHUNK>(p, blockIdx.x, &first, &len, &last)) return;
    const int h = blockIdx.y, d = p.d, dv = p.dv, dp = (d + 3) & ~3, dvp = (dv + 3) & ~3;
    float* ks = mlstm_sums_shared;
    float* vs = ks + CHUNK * dp;
    const float* rows = reinterpret_cast<const float*>(p.qkv) + (size_t)first * p.ld;
    load_chunk(ks, dp, rows + (size_t)(p.heads + h) * d, p.ld, len, d, p.vec, false, 0.f);
    load_chunk(vs, dvp, rows + (size_t)2 * p.heads * d + (size_t)h * dv, p.ld, len, dv, p.vec, false, 0.f);
    const MlstmToken token = mlstm_tokens<CHUNK>(p, first, len, h, scratch);
    if (threadIdx.x < CHUNK) {
        const double highest = __shfl_sync(0xffffffffu, token.top, CHUNK - 1), total = __shfl_sync(0xffffffffu, token.total, CHUNK - 1);
        weight[threadIdx.x] = (int)threadIdx.x < len ? expf((float)(token.a - highest)) : 0.f;
        if (threadIdx.x == 0) {
            p.totals[(size_t)blockIdx.x * p.heads + h] = (float)total;
            p.tops[(size_t)blockIdx.x * p.heads + h] = (float)(highest + total);
        }
    }
    __syncthreads();
    float* U = p.sums + ((size_t)blockIdx.x * p.heads + h) * ((size_t)d * dv + d);
    for (int i = threadIdx.x; i < d; i += blockDim.x) {
        float sum = 0.f;
        for (int t = 0; t < len; ++t) sum = fmaf(weight[t], ks[t * dp + i], sum);
        U[(size_t)d * dv + i] = sum;
    }
    for (int e = threadIdx.x; e < len * dvp; e += blockDim.x) vs[e] *= weight[e / dvp];
    __syncthreads();
    const int tiles_j = dvp / 4, tiles = (dp / 4) * tiles_j;
    for (int tile = threadIdx.x; tile < tiles; tile += blockDim.x) {
        const int i0 = (tile / tiles_j) * 4, j0 = (tile % tiles_j) * 4;
        float acc[4][4] = {};
        for (int t = 0; t < len; ++t) {
            const float4 a = *reinterpret_cast<const float4*>(ks + t * dp + i0);
            const float4 b = *reinterpret_cast<const float4*>(vs + t * dvp + j0);
            const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
            for (int x = 0; x < 4; ++x)
#pragma unroll
                for (int y = 0; y < 4; ++y) acc[x][y] = fmaf(av[x], bv[y], acc[x][y]);
        }
#pragma unroll
        for (int x = 0; x < 4; ++x)
#pragma unroll
            for (int y = 0; y < 4; ++y)
                if (i0 + x < d && j0 + y < dv) U[(size_t)(i0 + x) * dv + j0 + y] = acc[x][y];
    }
}

template <typename TO>
__global__ void __launch_bounds__(MLSTM_THREADS)
mlstm_output_kernel(MlstmArgs p) {
    // q [CHUNK][ds], k [CHUNK][ds], v [CHUNK][dvp], A [CHUNK][CHUNK], o [CHUNK][dvp]; ds = dp + 4: rows four floats apart from a
    // multiple of 32, so that 32 lanes reading four floats each of 32 different rows meet no bank twice
    extern __shared__ float mlstm_out_shared[];
    __shared__ ChunkShared c;
    __shared__ double scratch[2];
    pdl_launch_dependents();
    pdl_wait();
    int first, len;
    bool last;
    if (!mlstm_find_chunk<CHUNK>(p, blockIdx.x, &first, &len, &last)) return;
    const int slot = p.slots[first];
    if (slot < 0) return;
    const int h = blockIdx.y, d = p.d, dv = p.dv, dp = (d + 3) & ~3, dvp = (dv + 3) & ~3, ds = dp + 4;
    float* qs = mlstm_out_shared;
    float* ks = qs + CHUNK * ds;
    float* vs = ks + CHUNK * ds;
    float* A = vs + CHUNK * dvp;
    float* os = dvp <= ds ? ks : A + CHUNK * CHUNK;       // (in the keys' room where it fits: they are done with once A is made)
    const float* rows = reinterpret_cast<const float*>(p.qkv) + (size_t)first * p.ld;
    load_chunk(qs, ds, rows + (size_t)h * d, p.ld, len, d, p.vec, false, 0.f);
    load_chunk(ks, ds, rows + (size_t)(p.heads + h) * d, p.ld, len, d, p.vec, false, 0.f);
    load_chunk(vs, dvp, rows + (size_t)2 * p.heads * d + (size_t)h * dv, p.ld, len, dv, p.vec, false, 0.f);
    const size_t at = (size_t)blockIdx.x * p.heads + h;
    const float m0 = p.starts[at];
    const MlstmToken token = mlstm_tokens<CHUNK>(p, first, len, h, scratch);
    if (threadIdx.x < CHUNK) {
        const int t = threadIdx.x;
        const double top = fmax((double)m0, token.top);
        c.a[t] = mlstm_pair(token.a);
        c.top[t] = mlstm_pair(top);
        c.start[t] = expf((float)((double)m0 - top)) * p.q_scale;
        c.floor_[t] = expf(-(float)(token.total + top));
        if (last && t == len - 1)
            p.state[(size_t)slot * p.slot_stride + (size_t)p.heads * ((size_t)d * dv + d) + h] = fmaxf(m0 + p.totals[at], p.tops[at]);
    }
    __syncthreads();
    // A[t][j] = (q_t . k_j) d^(-1/2) exp(a_j - M_t) for j <= t: a warp one j, a lane a token t
    for (int e = threadIdx.x; e < CHUNK * CHUNK; e += blockDim.x) {
        const int j = e / CHUNK, t = e - j * CHUNK;
        float acc = 0.f;
        if (j <= t && t < len) {
            const float4* q4 = reinterpret_cast<const float4*>(qs + t * ds);
            const float4* k4 = reinterpret_cast<const float4*>(ks + j * ds);
            for (int i = 0; i < dp / 4; ++i) {
                const float4 q = q4[i], k = k4[i];
                acc = fmaf(q.x, k.x, acc);
                acc = fmaf(q.y, k.y, acc);
                acc = fmaf(q.z, k.z, acc);
                acc = fmaf(q.w, k.w, acc);
            }
            acc *= p.q_scale * expf(mlstm_difference(c.a[j], c.top[t]));
        }
        A[t * CHUNK + j] = acc;
    }
    __syncthreads();
    const int unit = d * dv + d;
    const float* S = p.sums + at * unit;
    const float* n_in = S + (size_t)d * dv;
    // n_t . q_t from the start and from the chunk's own tokens, and with it what o_t is divided by: a warp a token
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    for (int t = warp; t < len; t += MLSTM_THREADS / 32) {
        float sum = 0.f;
        for (int i = lane; i < d; i += 32) sum = fmaf(qs[t * ds + i], n_in[i], sum);
        sum = warp_sum(fmaf(c.start[t], sum, A[t * CHUNK + lane]));
        if (lane == 0) c.below[t] = fmaxf(fabsf(sum), c.floor_[t]) + 1e-6f;
    }
    __syncthreads();
    const int tiles_j = dvp / 4, tiles = (CHUNK / 4) * tiles_j;
    const bool aligned = (dv & 3) == 0 && (unit & 3) == 0 && p.vec;
    for (int tile = threadIdx.x; tile < tiles; tile += blockDim.x) {
        const int t0 = (tile / tiles_j) * 4, j0 = (tile % tiles_j) * 4;
        float acc[4][4] = {};
#pragma unroll 8
        for (int i = 0; i < d; ++i) {
            float bv[4];
            if (aligned) {
                const float4 b = __ldg(reinterpret_cast<const float4*>(S + (size_t)i * dv + j0));
                bv[0] = b.x, bv[1] = b.y, bv[2] = b.z, bv[3] = b.w;
            } else {
#pragma unroll
                for (int y = 0; y < 4; ++y) bv[y] = j0 + y < dv ? __ldg(S + (size_t)i * dv + j0 + y) : 0.f;
            }
#pragma unroll
            for (int x = 0; x < 4; ++x) {
                const float a = qs[(t0 + x) * ds + i];
#pragma unroll
                for (int y = 0; y < 4; ++y) acc[x][y] = fmaf(a, bv[y], acc[x][y]);
            }
        }
#pragma unroll
        for (int x = 0; x < 4; ++x) {
            const float w = c.start[t0 + x];
#pragma unroll
            for (int y = 0; y < 4; ++y) acc[x][y] *= w;
        }
        for (int jj = 0; jj < len; ++jj) {
            const float4 b = *reinterpret_cast<const float4*>(vs + jj * dvp + j0);
            const float bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
            for (int x = 0; x < 4; ++x) {
                const float w = A[(t0 + x) * CHUNK + jj];
#pragma unroll
                for (int y = 0; y < 4; ++y) acc[x][y] = fmaf(w, bv[y], acc[x][y]);
            }
        }
#pragma unroll
        for (int x = 0; x < 4; ++x)
#pragma unroll
            for (int y = 0; y < 4; ++y) os[(t0 + x) * dvp + j0 + y] = acc[x][y] / (t0 + x < len ? c.below[t0 + x] : 1.f);
    }
    __syncthreads();
    // the head's norm over its dv elements, its weight and the gate: a warp a token
    for (int t = warp; t < len; t += MLSTM_THREADS / 32) {
        float sum = 0.f;
        for (int j = lane; j < dv; j += 32) sum = fmaf(os[t * dvp + j], os[t * dvp + j], sum);
        sum = warp_sum(sum);
        const float inv = 1.0f / sqrtf(sum / (float)dv + p.eps);
        const float* g = p.gates + (size_t)(first + t) * p.ld_g + (size_t)h * dv;
        TO* dst = reinterpret_cast<TO*>(p.out) + ((size_t)(first + t) * p.heads + h) * dv;
        for (int j = lane; j < dv; j += 32)
            dst[j] = from_float<TO>(os[t * dvp + j] * inv * p.norm_weight[(size_t)h * dv + j] * mlstm_sigmoid(g[j]));
    }
}

size_t output_shared_bytes(int d, int dv) {
    const int dp = (d + 3) & ~3, dvp = (dv + 3) & ~3;
    return ((size_t)2 * CHUNK * (dp + 4) + (size_t)(dvp <= dp + 4 ? 1 : 2) * CHUNK * dvp + CHUNK * CHUNK) * sizeof(float);
}

__device__ __forceinline__ float qkv_at(const MlstmArgs& p, size_t index, int round16) {
    if (p.qkv_bf16) return to_float(reinterpret_cast<const __nv_bfloat16*>(p.qkv)[index]);
    const float v = reinterpret_cast<const float*>(p.qkv)[index];
    return round16 ? to_float(__float2bfloat16_rn(v)) : v;
}
__device__ __forceinline__ void mlstm_cluster_sync() {
    asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
    asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory");
}
__device__ __forceinline__ float mlstm_cluster_load(const float* mine, uint32_t rank) {
    uint32_t remote;
    const uint32_t at = (uint32_t)__cvta_generic_to_shared(mine);
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(remote) : "r"(at), "r"(rank));
    float v;
    asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(remote) : "memory");
    return v;
}

// VEC: value columns of the memory that a thread takes side by side (4 where sizes and addresses allow it).  gridDim.z CTAs
// (a cluster, where more than one) share a head's columns; all of them keep n and m for themselves and the first writes them
// back once all have read them.
template <typename TO, int VEC>
__global__ void __launch_bounds__(MLSTM_THREADS, 4)
mlstm_single_kernel(MlstmArgs p, int round16) {
    extern __shared__ float mlstm_single_shared[];        // q [d], k [d], n [d], partial sums [rows][columns]
    __shared__ float scratch[32], squares;
    pdl_launch_dependents();
    // (the step's metadata and the state as the step before left it depend on no kernel of this step)
    const int t = p.single_rows[blockIdx.x], h = blockIdx.y;
    const int slot = t >= 0 ? p.slots[t] : -1;
    if (slot < 0) return;                                 // (a cluster serves one token: all its CTAs leave)
    const int d = p.d, dv = p.dv, unit = d * dv + d, columns = dv / gridDim.z, c0 = blockIdx.z * columns;
    float* base = p.state + (size_t)slot * p.slot_stride;
    float* S = base + (size_t)h * d * dv + c0;
    float* n_state = base + (size_t)p.heads * d * dv + (size_t)h * d;
    float* m_state = base + (size_t)p.heads * unit + h;
    const int lanes = min(columns / VEC, MLSTM_THREADS), rows = MLSTM_THREADS / lanes;
    const int group = threadIdx.x / lanes, lane_j = (threadIdx.x % lanes) * VEC;
    constexpr int AHEAD = 8;                              // (eight rows of the memory at a time: their loads are in flight together)
    float held[AHEAD][VEC];
    auto load = [&](int i0, int j) {
#pragma unroll
        for (int k = 0; k < AHEAD; ++k) {
            const int i = i0 + k * rows;
            if (group < rows && i < d) {
                if constexpr (VEC == 4) {
                    const float4 v = *reinterpret_cast<const float4*>(S + (size_t)i * dv + j);
                    held[k][0] = v.x, held[k][1] = v.y, held[k][2] = v.z, held[k][3] = v.w;
                } else {
                    held[k][0] = S[(size_t)i * dv + j];
                }
            }
        }
    };
    load(group, lane_j);
    const float m_before = *m_state;
    pdl_wait();
    float* qs = mlstm_single_shared;
    float* ks = qs + d;
    float* ns = ks + d;
    float* partial = ns + d;
    float i_gate, f_gate;
    mlstm_log_gates(p, t, h, i_gate, f_gate);
    const float kept = f_gate + m_before, m = fmaxf(kept, i_gate);
    const float keep = expf(kept - m), put = expf(i_gate - m);
    const size_t row = (size_t)t * p.ld;
    float dot = 0.f;
    for (int i = threadIdx.x; i < d; i += MLSTM_THREADS) {
        const float q = qkv_at(p, row + (size_t)h * d + i, round16) * p.q_scale;
        const float k = qkv_at(p, row + (size_t)(p.heads + h) * d + i, round16) * put;
        const float n = fmaf(keep, n_state[i], k);
        qs[i] = q;
        ks[i] = k;
        ns[i] = n;
        dot = fmaf(n, q, dot);
    }
    dot = block_sum(dot, scratch);                        // (its barriers also publish q and k)
    const float below = fmaxf(fabsf(dot), expf(-m)) + 1e-6f;
    if (group < rows) {
        for (int j = lane_j; j < columns; j += lanes * VEC) {
            float vj[VEC], acc[VEC];
#pragma unroll
            for (int v = 0; v < VEC; ++v) {
                vj[v] = qkv_at(p, row + (size_t)2 * p.heads * d + (size_t)h * dv + c0 + j + v, round16);
                acc[v] = 0.f;
            }
            for (int i0 = group; i0 < d; i0 += rows * AHEAD) {
                if (i0 != group || j != lane_j) load(i0, j);
#pragma unroll
                for (int k = 0; k < AHEAD; ++k) {
                    const int i = i0 + k * rows;
                    if (i >= d) break;
#pragma unroll
                    for (int v = 0; v < VEC; ++v) {
                        held[k][v] = fmaf(keep, held[k][v], ks[i] * vj[v]);
                        acc[v] = fmaf(held[k][v], qs[i], acc[v]);
                    }
                    if constexpr (VEC == 4)
                        *reinterpret_cast<float4*>(S + (size_t)i * dv + j) = make_float4(held[k][0], held[k][1], held[k][2], held[k][3]);
                    else
                        S[(size_t)i * dv + j] = held[k][0];
                }
            }
#pragma unroll
            for (int v = 0; v < VEC; ++v) partial[group * columns + j + v] = acc[v];
        }
    }
    __syncthreads();
    float sum = 0.f;
    for (int j = threadIdx.x; j < columns; j += MLSTM_THREADS) {
        float o = partial[j];
        for (int r = 1; r < rows; ++r) o += partial[r * columns + j];
        o /= below;
        partial[j] = o;                                   // (only this thread touches column j)
        sum = fmaf(o, o, sum);
    }
    sum = block_sum(sum, scratch);
    if (gridDim.z > 1) {
        if (threadIdx.x == 0) squares = sum;
        mlstm_cluster_sync();                             // every CTA's squares are there, and everyone has read n and m
        sum = 0.f;
        for (uint32_t r = 0; r < gridDim.z; ++r) sum += mlstm_cluster_load(&squares, r);
    }
    if (blockIdx.z == 0) {
        for (int i = threadIdx.x; i < d; i += MLSTM_THREADS) n_state[i] = ns[i];
        if (threadIdx.x == 0) *m_state = m;
    }
    const float inv = 1.0f / sqrtf(sum / (float)dv + p.eps);
    const float* g = p.gates + (size_t)t * p.ld_g + (size_t)h * dv + c0;
    const float* w = p.norm_weight + (size_t)h * dv + c0;
    TO* dst = reinterpret_cast<TO*>(p.out) + ((size_t)t * p.heads + h) * dv + c0;
    for (int j = threadIdx.x; j < columns; j += MLSTM_THREADS) dst[j] = from_float<TO>(partial[j] * inv * w[j] * mlstm_sigmoid(g[j]));
    if (gridDim.z > 1) mlstm_cluster_sync();              // nobody leaves while a neighbour may still read its shared memory
}

template <typename TO, int VEC>
int launch_single(const MlstmArgs& p, int n_single, int share, int round16, cudaStream_t stream) {
    const int columns = p.dv / share, lanes = columns / VEC < MLSTM_THREADS ? columns / VEC : MLSTM_THREADS;
    const size_t bytes = ((size_t)3 * p.d + (size_t)(MLSTM_THREADS / lanes) * columns) * sizeof(float);
    cudaLaunchConfig_t config = {};
    config.gridDim = dim3(n_single, p.heads, share);
    config.blockDim = dim3(MLSTM_THREADS);
    config.dynamicSmemBytes = bytes;
    config.stream = stream;
    cudaLaunchAttribute attributes[2];
    attributes[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attributes[0].val.programmaticStreamSerializationAllowed = 1;
    attributes[1].id = cudaLaunchAttributeClusterDimension;
    attributes[1].val.clusterDim.x = 1;
    attributes[1].val.clusterDim.y = 1;
    attributes[1].val.clusterDim.z = (unsigned)share;
    const bool pdl = lia_pdl_enabled.load(std::memory_order_relaxed) != 0;
    config.attrs = pdl ? attributes : attributes + 1;
    config.numAttrs = (pdl ? 1 : 0) + (share > 1 ? 1 : 0);
    lia_launch_counter.fetch_add(1, std::memory_order_relaxed);
    if (cudaLaunchKernelEx(&config, mlstm_single_kernel<TO, VEC>, p, round16) != cudaSuccess) {
        cudaGetLastError();
        return LIA_ERR_LAUNCH;
    }
    return cudaGetLastError() == cudaSuccess ? LIA_OK : LIA_ERR_LAUNCH;
}
}  // namespace

// Words of 32-bit scratch for `chunks` chunks.
LIA_EXPORT long long lia_mlstm_scratch_floats(int chunks, int heads, int d, int dv) { return mlstm_scratch_words(chunks, heads, d, dv); }

// The portions of a step on the 32-bit pipes.  qkv [n, ld] = [q: heads d | k: heads d | v: heads dv] and gates [n, ld_g] =
// [g: heads dv | i: heads | f: heads], 32-bit; i_bias, f_bias [heads], norm_weight [heads dv] 32-bit; state: slot s at
// + s slot_stride: S [heads, d, dv], n [heads, d], m [heads]; `segments` [n_segments, 3] (first batch index, first position,
// count); out [n, heads dv] of out_dtype; scratch: lia_mlstm_scratch_floats(max_chunks, ...) words.
LIA_EXPORT int lia_mlstm(const float* qkv, long long ld, const float* gates, long long ld_g, const float* i_bias,
                         const float* f_bias, float cap, float* state, long long slot_stride, const int* segments, int n_segments,
                         int max_chunks, const int* slots, const float* norm_weight, float eps, void* out, int out_dtype, int heads,
                         int d, int dv, float* scratch, long long scratch_floats, cudaStream_t stream) {
    if (n_segments <= 0) return LIA_OK;
    if (heads <= 0 || heads > 65535 || d <= 0 || dv <= 0 || d > MLSTM_MAX || dv > MLSTM_MAX || !(cap > 0.f) ||
        ld < (long long)heads * (2 * d + dv) || ld_g < (long long)heads * (dv + 2) ||
        slot_stride < (long long)heads * ((long long)d * dv + d + 1) || max_chunks <= 0 || !scratch ||
        scratch_floats < mlstm_scratch_words(max_chunks, heads, d, dv))
        return LIA_ERR_SIZE;
    if (out_dtype != LIA_F32 && out_dtype != LIA_BF16) return LIA_ERR_DTYPE;
    MlstmArgs p = {};
    p.qkv = qkv; p.ld = ld; p.gates = gates; p.ld_g = ld_g; p.i_bias = i_bias; p.f_bias = f_bias; p.cap = cap;
    p.state = state; p.slot_stride = slot_stride; p.segments = segments; p.n_segments = n_segments; p.slots = slots;
    p.norm_weight = norm_weight; p.eps = eps; p.out = out; p.heads = heads; p.d = d; p.dv = dv;
    p.q_scale = 1.0f / sqrtf((float)d);
    mlstm_place_scratch(p, scratch, max_chunks);
    p.vec = ((d | dv) & 3) == 0 && (ld & 3) == 0 && (((uintptr_t)qkv | (uintptr_t)scratch) & 15u) == 0 ? 1 : 0;
    const bool four = p.vec && slot_stride % 4 == 0 && ((uintptr_t)state & 15u) == 0;
    const int dp = (d + 3) & ~3, dvp = (dv + 3) & ~3;
    static bool raised = false;
    if (!raised) {
        if (cudaFuncSetAttribute(mlstm_sums_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024) != cudaSuccess ||
            cudaFuncSetAttribute(mlstm_output_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024) != cudaSuccess ||
            cudaFuncSetAttribute(mlstm_output_kernel<__nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024) != cudaSuccess)
            return LIA_ERR_LAUNCH;
        raised = true;
    }
    int code = lia_launch(mlstm_sums_kernel, dim3(max_chunks, heads), dim3(MLSTM_THREADS), (size_t)CHUNK * (dp + dvp) * sizeof(float), stream, p);
    if (code != LIA_OK) return code;
    code = mlstm_launch_carry(p, CHUNK, four, stream);
    if (code != LIA_OK) return code;
    const size_t bytes = output_shared_bytes(d, dv);
    if (out_dtype == LIA_F32) return lia_launch(mlstm_output_kernel<float>, dim3(max_chunks, heads), dim3(MLSTM_THREADS), bytes, stream, p);
    return lia_launch(mlstm_output_kernel<__nv_bfloat16>, dim3(max_chunks, heads), dim3(MLSTM_THREADS), bytes, stream, p);
}

// The single tokens alone (batch indices `single_rows`): qkv of qkv_dtype (round16: 32-bit rows are rounded to bfloat16 as
// they are read), the other arguments as for lia_mlstm.  `wanted_ctas`: a head's columns are shared by up to 8 CTAs while there
// are fewer CTAs than this and a CTA's share of the memory is 128 KB or more (a cluster costs about 2 us: smaller heads stay whole).
LIA_EXPORT int lia_mlstm_single(const void* qkv, int qkv_dtype, long long ld, int round16, const float* gates, long long ld_g,
                                const float* i_bias, const float* f_bias, float cap, float* state, long long slot_stride,
                                const int* single_rows, int n_single, const int* slots, const float* norm_weight, float eps,
                                void* out, int out_dtype, int heads, int d, int dv, int wanted_ctas, cudaStream_t stream) {
    if (n_single <= 0) return LIA_OK;
    if (heads <= 0 || heads > 65535 || d <= 0 || dv <= 0 || d > MLSTM_MAX || dv > MLSTM_MAX || !(cap > 0.f) ||
        ld < (long long)heads * (2 * d + dv) || ld_g < (long long)heads * (dv + 2) ||
        slot_stride < (long long)heads * ((long long)d * dv + d + 1))
        return LIA_ERR_SIZE;
    if ((qkv_dtype != LIA_F32 && qkv_dtype != LIA_BF16) || (out_dtype != LIA_F32 && out_dtype != LIA_BF16)) return LIA_ERR_DTYPE;
    MlstmArgs p = {};
    p.qkv = qkv; p.ld = ld; p.qkv_bf16 = qkv_dtype == LIA_BF16; p.gates = gates; p.ld_g = ld_g; p.i_bias = i_bias; p.f_bias = f_bias;
    p.cap = cap; p.state = state; p.slot_stride = slot_stride; p.single_rows = single_rows; p.slots = slots;
    p.norm_weight = norm_weight; p.eps = eps; p.out = out; p.heads = heads; p.d = d; p.dv = dv;
    p.q_scale = 1.0f / sqrtf((float)d);
    const bool four = dv % 4 == 0 && slot_stride % 4 == 0 && ((uintptr_t)state & 15u) == 0;
    int share = 1;
    while (four && share < 8 && dv % (share * 2 * 32) == 0 && (long long)d * dv >= 32768LL * share && (long long)n_single * heads * share < wanted_ctas)
        share *= 2;
    if (out_dtype == LIA_F32)
        return four ? launch_single<float, 4>(p, n_single, share, round16, stream) : launch_single<float, 1>(p, n_single, 1, round16, stream);
    return four ? launch_single<__nv_bfloat16, 4>(p, n_single, share, round16, stream)
                : launch_single<__nv_bfloat16, 1>(p, n_single, 1, round16, stream);
}
