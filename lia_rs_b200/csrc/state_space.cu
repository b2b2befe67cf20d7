// A linear recurrence per head with one decay per token and head (state-space duality, Mamba-2).  Head h of `heads` reads
// group g = h / (heads / groups) of B and C:
//     dt = softplus(raw + dt_bias_h),   S_t = exp(-exp(A_log_h) dt) S_(t-1) + dt B_t x_t^T      (S [N, P], 32-bit)
//     y_t = S_t^T C_t + D_h x_t
// x, B and C come as rows [x: heads P | B: groups N | C: groups N] out of the convolution, dt raw from the input product.
//  * Single tokens (`ssd_single`): one CTA per (token, head) updates the state in place and forms y from it.
//  * Prompt portions are cut into chunks of CHUNK tokens that run side by side, in three launches; with
//    L_t = -exp(A_log) dt_t log2(e) and C_t = L_1 + ... + L_t inside the chunk (every exponent below is <= 0):
//      sums    U_c = sum_j 2^(C_len - C_j) dt_j B_j x_j^T of each chunk, from zero, and C_len beside it;
//      carry   along each portion: the state that each chunk starts from takes U_c's place in scratch,
//              S <- 2^C_len S + U_c, and the last S goes back to the request's state;
//      output  y_t = 2^C_t S_in^T C_t + sum_(j<=t) (C_t . B_j) 2^(C_t - C_j) dt_j x_j + D x_t.
//    The recurrence is linear in the state, so this is the recurrence itself in another order of additions.
//  * `gated_group_norm`: y * silu(z), in `groups` equal parts of a row each over its own root mean square, times a weight.
// Everything is 32-bit; only the normed rows have the compute element type.  A row whose slot is negative belongs to nobody
// and is skipped.
#include "linear_recurrence.cuh"
#include "state_space.cuh"

namespace {
// Where a single token's x, B and C come from: the convolution's rows (`raw` null), or the input product's rows, and the
// kernel does the convolution of the channels that its head reads itself (a step of single tokens alone: no other row of
// the step is an earlier input of a token, all of them lie in its ring).
struct SingleInput {
    const float* raw; long long ld_raw;       // [n, ld_raw] [x | B | C] ahead of the convolution
    const float* weight; const float* bias;   // [taps, channels], [channels] or null
    float* ring; long long ring_stride;       // slot s: [taps, channels]
    const int* positions;
    int taps, channels, round16;              // round16: the convolution's result is rounded to bfloat16, as its rows would be
    const void* rows; int rows_bf16;          // [n, ld] out of the convolution
};

template <int VEC>                            // columns of the state that a thread takes (4: P and the addresses allow it)
__global__ void __launch_bounds__(SSD_THREADS, 4)
ssd_single_kernel(SsdArgs p, SingleInput in) {
    extern __shared__ float ssd_single_shared[];          // B [N], C [N], x [P], partial sums [SSD_THREADS VEC]
    pdl_launch_dependents();
    // (the step's metadata depends on no kernel of the step)
    const int t = p.single_rows[blockIdx.x], h = blockIdx.y;
    const int slot = t >= 0 ? p.slots[t] : -1;
    const int pos = in.raw && t >= 0 ? in.positions[t] : 0;
    pdl_wait();
    if (slot < 0) return;
    const int N = p.N, P = p.P;
    float* S = p.state + (size_t)slot * p.slot_stride + (size_t)h * N * P;
    const int lanes = P / VEC, rows = SSD_THREADS / lanes;
    const int group = threadIdx.x / lanes, j = (threadIdx.x % lanes) * VEC;
    constexpr int AHEAD = 8;                              // (eight rows of the state at a time: their loads are in flight together)
    float held[AHEAD][VEC];
    auto load = [&](int i0) {
#pragma unroll
        for (int k = 0; k < AHEAD; ++k) {
            const int i = i0 + k * rows;
            if (group < rows && i < N) {
                if constexpr (VEC == 4) {
                    const float4 v = *reinterpret_cast<const float4*>(S + (size_t)i * P + j);
                    held[k][0] = v.x, held[k][1] = v.y, held[k][2] = v.z, held[k][3] = v.w;
                } else {
                    held[k][0] = S[(size_t)i * P + j];
                }
            }
        }
    };
    load(group);                                          // (under way while x, B and C arrive)
    float* bs = ssd_single_shared;
    float* cs = bs + N;
    float* xs = cs + N;
    float* partial = xs + P;
    const int per_group = p.heads / p.groups, g = h / per_group;
    const int b_at = p.heads * P + g * N, c_at = p.heads * P + (p.groups + g) * N;
    float* ring = in.ring ? in.ring + (size_t)slot * in.ring_stride : nullptr;
    for (int e = threadIdx.x; e < 2 * N + P; e += SSD_THREADS) {
        const int c = e < N ? b_at + e : e < 2 * N ? c_at + e - N : h * P + e - 2 * N;
        float v;
        if (in.raw) {
            const float own = in.raw[(size_t)t * in.ld_raw + c];
            v = in.bias ? in.bias[c] : 0.f;
            for (int j = 0; j < in.taps - 1; ++j) {
                const int k = in.taps - 1 - j;
                const float earlier = pos - k >= 0 ? ring[(size_t)((pos - k) % in.taps) * in.channels + c] : 0.f;
                v = fmaf(in.weight[(size_t)j * in.channels + c], earlier, v);
            }
            v = ring_silu(fmaf(in.weight[(size_t)(in.taps - 1) * in.channels + c], own, v));
            if (in.round16) v = to_float(from_float<__nv_bfloat16>(v));
            // the head's own channels, and the group's by its first head (the row written is none of those read)
            if (in.taps > 1 && (e >= 2 * N || h == g * per_group)) ring[(size_t)(pos % in.taps) * in.channels + c] = own;
        } else if (in.rows_bf16) {
            v = to_float(reinterpret_cast<const __nv_bfloat16*>(in.rows)[(size_t)t * p.ld + c]);
        } else {
            v = reinterpret_cast<const float*>(in.rows)[(size_t)t * p.ld + c];
        }
        bs[e] = v;
    }
    const float dt = ring_softplus(p.dt[(size_t)t * p.ld_dt + h] + p.dt_bias[h]);
    const float decay = expf(-p.rate[h] * dt);
    __syncthreads();
    if (group < rows) {
        float xj[VEC], acc[VEC];
#pragma unroll
        for (int v = 0; v < VEC; ++v) xj[v] = dt * xs[j + v], acc[v] = 0.f;
        for (int i0 = group; i0 < N; i0 += rows * AHEAD) {
            if (i0 != group) load(i0);
#pragma unroll
            for (int k = 0; k < AHEAD; ++k) {
                const int i = i0 + k * rows;
                if (i >= N) break;
#pragma unroll
                for (int v = 0; v < VEC; ++v) {
                    held[k][v] = fmaf(decay, held[k][v], bs[i] * xj[v]);
                    acc[v] = fmaf(held[k][v], cs[i], acc[v]);
                }
                if constexpr (VEC == 4)
                    *reinterpret_cast<float4*>(S + (size_t)i * P + j) = make_float4(held[k][0], held[k][1], held[k][2], held[k][3]);
                else
                    S[(size_t)i * P + j] = held[k][0];
            }
        }
#pragma unroll
        for (int v = 0; v < VEC; ++v) partial[group * P + j + v] = acc[v];
    }
    __syncthreads();
    for (int c = threadIdx.x; c < P; c += SSD_THREADS) {
        float o = partial[c];
        for (int r = 1; r < rows; ++r) o += partial[r * P + c];
        p.y[(size_t)t * p.heads * P + (size_t)h * P + c] = fmaf(p.skip[h], xs[c], o);
    }
}

// steps [CHUNK] and the running sums [CHUNK] of the chunk's log2 decays, by the first warp (CHUNK lanes)
__device__ __forceinline__ void chunk_steps(const SsdArgs& p, int first, int len, int h, float* steps, float* logs) {
    static_assert(CHUNK == 32, "a lane a token");
    if (threadIdx.x < 32) {
        const int lane = threadIdx.x;
        const float dt = lane < len ? ring_softplus(p.dt[(size_t)(first + lane) * p.ld_dt + h] + p.dt_bias[h]) : 0.f;
        float sum = -p.rate[h] * dt * LOG2_E;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float before = __shfl_up_sync(0xffffffffu, sum, o);
            if (lane >= o) sum += before;
        }
        steps[lane] = dt;
        logs[lane] = sum;
    }
}

__global__ void __launch_bounds__(SSD_THREADS)
ssd_sums_kernel(SsdArgs p) {
    extern __shared__ float ssd_sums_shared[];            // B [CHUNK][np], x [CHUNK][pp] weighted
    __shared__ float steps[CHUNK], logs[CHUNK];
    pdl_launch_dependents();
    pdl_wait();
    int first, len, segment, chunk;
    if (!find_chunk(p.segments, p.n_segments, blockIdx.x, &first, &len, &segment, &chunk)) return;
    const int h = blockIdx.y, N = p.N, P = p.P, np = (N + 3) & ~3, pp = (P + 3) & ~3;
    float* bs = ssd_sums_shared;
    float* xs = bs + CHUNK * np;
    const float* rows = p.xbc + (size_t)first * p.ld;
    const int g = h / (p.heads / p.groups);
    load_chunk(bs, np, rows + (size_t)p.heads * P + (size_t)g * N, p.ld, len, N, p.vec, false, 0.f);
    load_chunk(xs, pp, rows + (size_t)h * P, p.ld, len, P, p.vec, false, 0.f);
    chunk_steps(p, first, len, h, steps, logs);
    __syncthreads();
    const float total = logs[len - 1];
    for (int e = threadIdx.x; e < len * pp; e += blockDim.x) {
        const int t = e / pp;
        xs[e] *= steps[t] * exp2f(total - logs[t]);
    }
    if (threadIdx.x == 0) p.totals[(size_t)blockIdx.x * p.heads + h] = total;
    __syncthreads();
    float* U = p.sums + ((size_t)blockIdx.x * p.heads + h) * N * P;
    const int tiles_j = pp / 4, tiles = (np / 4) * tiles_j;
    for (int tile = threadIdx.x; tile < tiles; tile += blockDim.x) {
        const int i0 = (tile / tiles_j) * 4, j0 = (tile % tiles_j) * 4;
        float acc[4][4] = {};
        for (int t = 0; t < len; ++t) {
            const float4 a = *reinterpret_cast<const float4*>(bs + t * np + i0);
            const float4 b = *reinterpret_cast<const float4*>(xs + t * pp + j0);
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
                if (i0 + x < N && j0 + y < P) U[(size_t)(i0 + x) * P + j0 + y] = acc[x][y];
    }
}

__global__ void __launch_bounds__(SSD_THREADS)
ssd_output_kernel(SsdArgs p) {
    // C [CHUNK][ns], B [CHUNK][ns], x [CHUNK][pp], A [CHUNK][CHUNK]; ns = np + 4: rows four floats apart from a multiple of
    // 32, so that 32 lanes reading four floats each of 32 different rows meet no bank twice
    extern __shared__ float ssd_out_shared[];
    __shared__ float steps[CHUNK], logs[CHUNK];
    pdl_launch_dependents();
    pdl_wait();
    int first, len, segment, chunk;
    if (!find_chunk(p.segments, p.n_segments, blockIdx.x, &first, &len, &segment, &chunk)) return;
    const int h = blockIdx.y, N = p.N, P = p.P, np = (N + 3) & ~3, pp = (P + 3) & ~3, ns = np + 4;
    float* cs = ssd_out_shared;
    float* bs = cs + CHUNK * ns;
    float* xs = bs + CHUNK * ns;
    float* A = xs + CHUNK * pp;
    const float* rows = p.xbc + (size_t)first * p.ld;
    const int g = h / (p.heads / p.groups);
    load_chunk(bs, ns, rows + (size_t)p.heads * P + (size_t)g * N, p.ld, len, N, p.vec, false, 0.f);
    load_chunk(cs, ns, rows + (size_t)p.heads * P + (size_t)(p.groups + g) * N, p.ld, len, N, p.vec, false, 0.f);
    load_chunk(xs, pp, rows + (size_t)h * P, p.ld, len, P, p.vec, false, 0.f);
    chunk_steps(p, first, len, h, steps, logs);
    __syncthreads();
    // A[t][j] = (C_t . B_j) 2^(C_t - C_j) dt_j for j <= t (and D on the diagonal): a warp one j, a lane a token t
    for (int e = threadIdx.x; e < CHUNK * CHUNK; e += blockDim.x) {
        const int j = e / CHUNK, t = e - j * CHUNK;
        float acc = 0.f;
        if (j <= t && t < len) {
            const float4* c4 = reinterpret_cast<const float4*>(cs + t * ns);
            const float4* b4 = reinterpret_cast<const float4*>(bs + j * ns);
            for (int i = 0; i < np / 4; ++i) {
                const float4 c = c4[i], b = b4[i];
                acc = fmaf(c.x, b.x, acc);
                acc = fmaf(c.y, b.y, acc);
                acc = fmaf(c.z, b.z, acc);
                acc = fmaf(c.w, b.w, acc);
            }
            acc *= exp2f(logs[t] - logs[j]) * steps[j];
            if (j == t) acc += p.skip[h];
        }
        A[t * CHUNK + j] = acc;
    }
    __syncthreads();
    const float* S = p.sums + ((size_t)blockIdx.x * p.heads + h) * N * P;
    const int tiles_j = pp / 4, tiles = (CHUNK / 4) * tiles_j;
    const bool aligned = (P & 3) == 0 && p.vec;
    for (int tile = threadIdx.x; tile < tiles; tile += blockDim.x) {
        const int t0 = (tile / tiles_j) * 4, j0 = (tile % tiles_j) * 4;
        float acc[4][4] = {};
#pragma unroll 8
        for (int i = 0; i < N; ++i) {
            float bv[4];
            if (aligned) {
                const float4 b = __ldg(reinterpret_cast<const float4*>(S + (size_t)i * P + j0));
                bv[0] = b.x, bv[1] = b.y, bv[2] = b.z, bv[3] = b.w;
            } else {
#pragma unroll
                for (int y = 0; y < 4; ++y) bv[y] = j0 + y < P ? __ldg(S + (size_t)i * P + j0 + y) : 0.f;
            }
#pragma unroll
            for (int x = 0; x < 4; ++x) {
                const float a = cs[(t0 + x) * ns + i];
#pragma unroll
                for (int y = 0; y < 4; ++y) acc[x][y] = fmaf(a, bv[y], acc[x][y]);
            }
        }
#pragma unroll
        for (int x = 0; x < 4; ++x) {
            const float w = exp2f(logs[t0 + x]);
#pragma unroll
            for (int y = 0; y < 4; ++y) acc[x][y] *= w;
        }
        for (int jj = 0; jj < len; ++jj) {
            const float4 b = *reinterpret_cast<const float4*>(xs + jj * pp + j0);
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
            for (int y = 0; y < 4; ++y)
                if (t0 + x < len && j0 + y < P)
                    p.y[(size_t)(first + t0 + x) * p.heads * P + (size_t)h * P + j0 + y] = acc[x][y];
    }
}

// out[t, part] = rms(y * silu(z)) * weight over each of `groups` parts of `size` elements: a CTA a (token, part)
template <typename TO, int PER>                  // PER: quads a thread keeps in registers; 0: any size, the row read twice
__global__ void gated_group_norm_kernel(const float* __restrict__ y, const float* __restrict__ z, long long ld_z,
                                        const float* __restrict__ weight, const int* __restrict__ slots, TO* __restrict__ out,
                                        int groups, int size, float eps) {
    __shared__ float scratch[32];
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x, g = blockIdx.y;
    if (slots[t] < 0) return;
    const float* yr = y + (size_t)t * groups * size + (size_t)g * size;
    const float* zr = z + (size_t)t * ld_z + (size_t)g * size;
    TO* dst = out + (size_t)t * groups * size + (size_t)g * size;
    const float* w = weight + (size_t)g * size;
    float sum = 0.f;
    if constexpr (PER > 0) {
        const int quads = size / 4;
        float4 v[PER], gate[PER];
#pragma unroll
        for (int i = 0; i < PER; ++i) {
            const int q = threadIdx.x + i * blockDim.x;
            v[i] = q < quads ? reinterpret_cast<const float4*>(yr)[q] : make_float4(0.f, 0.f, 0.f, 0.f);
            gate[i] = q < quads ? reinterpret_cast<const float4*>(zr)[q] : make_float4(0.f, 0.f, 0.f, 0.f);
        }
#pragma unroll
        for (int i = 0; i < PER; ++i) {
            v[i].x *= ring_silu(gate[i].x), v[i].y *= ring_silu(gate[i].y);
            v[i].z *= ring_silu(gate[i].z), v[i].w *= ring_silu(gate[i].w);
            sum = fmaf(v[i].x, v[i].x, sum), sum = fmaf(v[i].y, v[i].y, sum);
            sum = fmaf(v[i].z, v[i].z, sum), sum = fmaf(v[i].w, v[i].w, sum);
        }
        const float inv = 1.0f / sqrtf(block_sum(sum, scratch) / (float)size + eps);
#pragma unroll
        for (int i = 0; i < PER; ++i) {
            const int q = threadIdx.x + i * blockDim.x;
            if (q >= quads) break;
            const float4 f = reinterpret_cast<const float4*>(w)[q];
            const float r[4] = {v[i].x * inv * f.x, v[i].y * inv * f.y, v[i].z * inv * f.z, v[i].w * inv * f.w};
            if constexpr (sizeof(TO) == 4) {
                *reinterpret_cast<float4*>(dst + 4 * q) = make_float4(r[0], r[1], r[2], r[3]);
            } else {
                const __nv_bfloat162 lo = __floats2bfloat162_rn(r[0], r[1]), hi = __floats2bfloat162_rn(r[2], r[3]);
                *reinterpret_cast<uint2*>(dst + 4 * q) = make_uint2(*reinterpret_cast<const uint32_t*>(&lo), *reinterpret_cast<const uint32_t*>(&hi));
            }
        }
    } else {
        for (int i = threadIdx.x; i < size; i += blockDim.x) {
            const float v = yr[i] * ring_silu(zr[i]);
            sum = fmaf(v, v, sum);
        }
        const float inv = 1.0f / sqrtf(block_sum(sum, scratch) / (float)size + eps);
        for (int i = threadIdx.x; i < size; i += blockDim.x) dst[i] = from_float<TO>(yr[i] * ring_silu(zr[i]) * inv * w[i]);
    }
}

// the last inputs of every run's convolution into the slot's ring: a CTA a row, rows further than `taps` from their run's end skip
__global__ void ring_store_kernel(const float* __restrict__ x, long long ld, const float* __restrict__ in_bias,
                                  float* __restrict__ ring, long long ring_stride, const int* __restrict__ positions,
                                  const int* __restrict__ slots, int n_tokens, int channels, int taps) {
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x, slot = slots[t];
    if (slot < 0) return;
    const int pos = positions[t];
    if (t + taps < n_tokens && slots[t + taps] == slot && positions[t + taps] == pos + taps) return;
    float* row = ring + (size_t)slot * ring_stride + (size_t)(pos % taps) * channels;
    for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < channels; c += gridDim.y * blockDim.x)
        row[c] = x[(size_t)t * ld + c] + (in_bias ? in_bias[c] : 0.f);
}
}  // namespace

// x [n, ld] 32-bit, in_bias [channels] or null: the inputs of every run's last `taps` tokens go to the slot's ring (slot s
// at ring + s ring_stride: [taps, channels]).
LIA_EXPORT int lia_ring_store(const float* x, long long ld, const float* in_bias, float* ring, long long ring_stride,
                              const int* positions, const int* slots, int n_tokens, int channels, int taps,
                              cudaStream_t stream) {
    if (n_tokens <= 0 || taps <= 1) return LIA_OK;
    if (channels <= 0 || taps > RING_MAX_TAPS || ld < channels || !ring) return LIA_ERR_SIZE;
    const dim3 grid(n_tokens, n_tokens >= 512 ? 1 : min(16, (channels + 127) / 128));
    return lia_launch(ring_store_kernel, grid, dim3(128), 0, stream, x, ld, in_bias, ring, ring_stride, positions, slots,
                      n_tokens, channels, taps);
}

// Words of 32-bit scratch for `chunks` chunks (the chunks' sums and, behind them, their summed log decays).
LIA_EXPORT long long lia_ssd_scratch_floats(int chunks, int heads, int N, int P) {
    return (long long)chunks * heads * ((long long)N * P + 1);
}

// xbc [n, ld] = [x: heads P | B: groups N | C: groups N], dt [n, ld_dt] (heads columns), dt_bias, rate, skip [heads], state
// (slot s at + s slot_stride: [heads, N, P]), y [n, heads P], scratch: `lia_ssd_scratch_floats(max_chunks, ...)` words: all
// 32-bit.  `segments` [n_segments, 3] names the step's portions; single tokens go to lia_ssd_single.
LIA_EXPORT int lia_ssd(const float* xbc, long long ld, const float* dt, long long ld_dt, const float* dt_bias,
                       const float* rate, const float* skip, float* state, long long slot_stride, const int* segments,
                       int n_segments, int max_chunks, const int* slots, float* y,
                       int heads, int groups, int N, int P, float* scratch, long long scratch_floats, cudaStream_t stream) {
    if (heads <= 0 || groups <= 0 || heads % groups || N <= 0 || P <= 0 || N > SSD_MAX || P > SSD_MAX ||
        ld < (long long)heads * P + 2LL * groups * N || ld_dt < heads || slot_stride < (long long)heads * N * P || heads > 65535)
        return LIA_ERR_SIZE;
    SsdArgs p = {xbc, ld, dt, ld_dt, dt_bias, rate, skip, state, slot_stride, segments, n_segments, nullptr, slots, y,
                 scratch, nullptr, heads, groups, N, P, 0};
    int code = LIA_OK;
    if (n_segments > 0) {
        if (max_chunks <= 0 || !scratch || scratch_floats < lia_ssd_scratch_floats(max_chunks, heads, N, P)) return LIA_ERR_SIZE;
        p.totals = scratch + (size_t)max_chunks * heads * N * P;
        p.vec = ((N | P) & 3) == 0 && (ld & 3) == 0 && (((uintptr_t)xbc | (uintptr_t)scratch) & 15u) == 0 ? 1 : 0;
        const int np = (N + 3) & ~3, pp = (P + 3) & ~3;
        const size_t sums_bytes = (size_t)CHUNK * (np + pp) * sizeof(float);
        const size_t out_bytes = ((size_t)CHUNK * (2 * (np + 4) + pp) + CHUNK * CHUNK) * sizeof(float);
        static bool raised = false;
        if (!raised) {
            cudaFuncSetAttribute(ssd_sums_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
            cudaFuncSetAttribute(ssd_output_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
            raised = true;
        }
        code = lia_launch(ssd_sums_kernel, dim3(max_chunks, heads), dim3(SSD_THREADS), sums_bytes, stream, p);
        if (code != LIA_OK) return code;
        const int parts = (N * P + SSD_THREADS - 1) / SSD_THREADS;
        code = lia_launch(ssd_carry_kernel, dim3(n_segments, heads, parts), dim3(SSD_THREADS), 0, stream, p, CHUNK);
        if (code != LIA_OK) return code;
        code = lia_launch(ssd_output_kernel, dim3(max_chunks, heads), dim3(SSD_THREADS), out_bytes, stream, p);
        if (code != LIA_OK) return code;
    }
    return code;
}

// The single tokens alone.  With `raw` (the input product's rows [n, ld_raw]; a step of single tokens alone): the kernel does
// the convolution (weight [taps, channels], bias [channels] or null, ring as for lia_ring_conv) and leaves each token's inputs
// in its ring; `round16`: x, B and C are rounded to bfloat16.  Else xbc [n, ld] of xbc_dtype comes from the convolution.
// The other arguments as for lia_ssd.
LIA_EXPORT int lia_ssd_single(const void* xbc, int xbc_dtype, long long ld, const float* raw, long long ld_raw,
                              const float* weight, const float* bias, float* ring, long long ring_stride, const int* positions,
                              int taps, int round16, const float* dt, long long ld_dt, const float* dt_bias, const float* rate,
                              const float* skip, float* state, long long slot_stride, const int* single_rows, int n_single,
                              const int* slots, float* y, int heads, int groups, int N, int P, cudaStream_t stream) {
    if (n_single <= 0) return LIA_OK;
    const long long channels = (long long)heads * P + 2LL * groups * N;
    if (heads <= 0 || groups <= 0 || heads % groups || N <= 0 || P <= 0 || N > SSD_MAX || P > SSD_MAX || ld_dt < heads ||
        slot_stride < (long long)heads * N * P || heads > 65535 || channels > 2147483647LL)
        return LIA_ERR_SIZE;
    if (raw ? (taps < 1 || taps > RING_MAX_TAPS || ld_raw < channels || !weight || !positions || (taps > 1 && !ring)) : (!xbc || ld < channels))
        return LIA_ERR_SIZE;
    if (!raw && xbc_dtype != LIA_F32 && xbc_dtype != LIA_BF16) return LIA_ERR_DTYPE;
    SsdArgs p = {nullptr, ld, dt, ld_dt, dt_bias, rate, skip, state, slot_stride, nullptr, 0, single_rows, slots, y,
                 nullptr, nullptr, heads, groups, N, P, 0};
    SingleInput in = {raw, ld_raw, weight, bias, ring, ring_stride, positions, taps, (int)channels, round16, xbc, xbc_dtype == LIA_BF16};
    const bool four = P % 4 == 0 && slot_stride % 4 == 0 && ((uintptr_t)state & 15u) == 0;
    const size_t bytes = ((size_t)2 * N + P + SSD_THREADS * (four ? 4 : 1)) * sizeof(float);
    if (four) return lia_launch(ssd_single_kernel<4>, dim3(n_single, heads), dim3(SSD_THREADS), bytes, stream, p, in);
    return lia_launch(ssd_single_kernel<1>, dim3(n_single, heads), dim3(SSD_THREADS), bytes, stream, p, in);
}

// y [n, groups size] and z [n, ld_z] 32-bit, weight [groups size] 32-bit, out [n, groups size] of out_dtype.
LIA_EXPORT int lia_gated_group_norm(const float* y, const float* z, long long ld_z, const float* weight, const int* slots,
                                    void* out, int out_dtype, int n_tokens, int groups, int size, float eps,
                                    cudaStream_t stream) {
    if (n_tokens <= 0) return LIA_OK;
    if (groups <= 0 || groups > 65535 || size <= 0 || ld_z < (long long)groups * size) return LIA_ERR_SIZE;
    const uintptr_t bits = (uintptr_t)y | (uintptr_t)z | (uintptr_t)weight | (uintptr_t)out;
    int per = 0, threads = size >= 1024 ? 256 : 128;
    if (size % 4 == 0 && ld_z % 4 == 0 && (bits & 15u) == 0 && size <= 8192) {
        const int quads = size / 4;
        threads = quads <= 32 ? 32 : quads <= 64 ? 64 : quads <= 128 ? 128 : quads <= 256 ? 256 : 512;
        per = (quads + threads - 1) / threads;
        per = per > 2 ? 4 : per;
    }
#define LIA_GATED(TO, PER)                                                                                                    \
    return lia_launch(gated_group_norm_kernel<TO, PER>, dim3(n_tokens, groups), dim3(threads), 0, stream, y, z, ld_z, weight, \
                      slots, (TO*)out, groups, size, eps)
#define LIA_GATED_PER(TO)                    \
    {                                        \
        if (per == 1) LIA_GATED(TO, 1);      \
        if (per == 2) LIA_GATED(TO, 2);      \
        if (per == 4) LIA_GATED(TO, 4);      \
        LIA_GATED(TO, 0);                    \
    }
    if (out_dtype == LIA_F32) LIA_GATED_PER(float)
    if (out_dtype == LIA_BF16) LIA_GATED_PER(__nv_bfloat16)
#undef LIA_GATED_PER
#undef LIA_GATED
    return LIA_ERR_DTYPE;
}
