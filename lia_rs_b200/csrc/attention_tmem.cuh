// Device helpers shared by the tcgen05 attention kernels (attention_prefill_tc.cu, sigmoid_attention_tc.cu): fast
// exponentials and paired 32-bit arithmetic, cp.async with zero fill, loads and stores of tensor memory, the MMA with
// its first operand in tensor memory, and the 128-byte-swizzled shared-memory tile with its two descriptors.
#pragma once
#include "tcgen05.cuh"

namespace tc5 {
__device__ __forceinline__ float ex2_approx(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
// Two 32-bit floats in one 64-bit register, and the instructions that work on both at once.
__device__ __forceinline__ uint64_t pack_f32x2(float lo, float hi) {
    uint64_t d;
    asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(lo), "f"(hi));
    return d;
}
__device__ __forceinline__ void unpack_f32x2(uint64_t v, float& lo, float& hi) {
    asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v));
}
__device__ __forceinline__ uint64_t fma_f32x2(uint64_t a, uint64_t b, uint64_t c) {
    uint64_t d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
__device__ __forceinline__ uint64_t add_f32x2(uint64_t a, uint64_t b) {
    uint64_t d;
    asm("add.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}
__device__ __forceinline__ uint64_t mul_f32x2(uint64_t a, uint64_t b) {
    uint64_t d;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}
// tanh as 1 - 2 / (1 + exp(2x)): absolute error about 2^-22, any x
__device__ __forceinline__ float tanh_by_exponential(float x) {
    return 1.0f - __fdividef(2.0f, 1.0f + ex2_approx(x * 2.8853900817779268f));
}
// tanh of two numbers within [-1, 1] or [-1/2, 1/2]: x P(x^2), P the polynomial of degree 5 (3) that agrees with
// tanh(sqrt(u)) / sqrt(u) at the six (four) Chebyshev nodes of [0, 1] ([0, 1/4]); absolute error below 2^-20 in both.  They run
// on the multiply-add pipes, beside the exponentials.
__device__ __forceinline__ uint64_t tanh_within_one(uint64_t x) {
    const uint64_t u = mul_f32x2(x, x);
    uint64_t r = pack_f32x2(-0.00305822904f, -0.00305822904f);
    r = fma_f32x2(r, u, pack_f32x2(0.0167208552f, 0.0167208552f));
    r = fma_f32x2(r, u, pack_f32x2(-0.0515859884f, -0.0515859884f));
    r = fma_f32x2(r, u, pack_f32x2(0.132807206f, 0.132807206f));
    r = fma_f32x2(r, u, pack_f32x2(-0.333289514f, -0.333289514f));
    r = fma_f32x2(r, u, pack_f32x2(0.999999395f, 0.999999395f));
    return mul_f32x2(r, x);
}
__device__ __forceinline__ uint64_t tanh_within_half(uint64_t x) {
    const uint64_t u = mul_f32x2(x, x);
    uint64_t r = pack_f32x2(-0.0443927384f, -0.0443927384f);
    r = fma_f32x2(r, u, pack_f32x2(0.131899394f, 0.131899394f));
    r = fma_f32x2(r, u, pack_f32x2(-0.333262842f, -0.333262842f));
    r = fma_f32x2(r, u, pack_f32x2(0.999999451f, 0.999999451f));
    return mul_f32x2(r, x);
}
__device__ __forceinline__ float exp2_whole(float n) {       // 2^n for a whole number n <= 0 (or -infinity), exactly
    return n < -126.f ? 0.f : __int_as_float(((int)n + 127) << 23);
}
__device__ __forceinline__ void cp_async_16(uint32_t dst, const void* src, bool valid) {
    const int bytes = valid ? 16 : 0;        // 0: the 16 bytes are filled with zeros
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
__device__ __forceinline__ void cp_async_wait_all() { asm volatile("cp.async.wait_group 0;" ::: "memory"); }
// 16 consecutive columns of this warp's 32 TMEM lanes, written from registers.
__device__ __forceinline__ void tmem_store16(uint32_t addr, const float* v) {
    asm volatile(
        "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], {%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16};"
        ::"r"(addr), "r"(__float_as_uint(v[0])), "r"(__float_as_uint(v[1])), "r"(__float_as_uint(v[2])), "r"(__float_as_uint(v[3])),
          "r"(__float_as_uint(v[4])), "r"(__float_as_uint(v[5])), "r"(__float_as_uint(v[6])), "r"(__float_as_uint(v[7])),
          "r"(__float_as_uint(v[8])), "r"(__float_as_uint(v[9])), "r"(__float_as_uint(v[10])), "r"(__float_as_uint(v[11])),
          "r"(__float_as_uint(v[12])), "r"(__float_as_uint(v[13])), "r"(__float_as_uint(v[14])), "r"(__float_as_uint(v[15]))
        : "memory");
}
// 64 consecutive columns of this warp's 32 TMEM lanes into registers; the caller waits (tc5::tmem_load_wait) before use.
__device__ __forceinline__ void tmem_load64_nowait(uint32_t addr, uint32_t* r) {
    asm volatile(
        "tcgen05.ld.sync.aligned.32x32b.x64.b32 {%0, %1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16, %17, %18, %19, %20, %21, %22, %23, %24, %25, %26, %27, %28, %29, %30, %31, %32, %33, %34, %35, %36, %37, %38, %39, %40, %41, %42, %43, %44, %45, %46, %47, %48, %49, %50, %51, %52, %53, %54, %55, %56, %57, %58, %59, %60, %61, %62, %63}, [%64];"
        : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]), "=r"(r[9]), "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15]), "=r"(r[16]), "=r"(r[17]), "=r"(r[18]), "=r"(r[19]), "=r"(r[20]), "=r"(r[21]), "=r"(r[22]), "=r"(r[23]), "=r"(r[24]), "=r"(r[25]), "=r"(r[26]), "=r"(r[27]), "=r"(r[28]), "=r"(r[29]), "=r"(r[30]), "=r"(r[31]), "=r"(r[32]), "=r"(r[33]), "=r"(r[34]), "=r"(r[35]), "=r"(r[36]), "=r"(r[37]), "=r"(r[38]), "=r"(r[39]), "=r"(r[40]), "=r"(r[41]), "=r"(r[42]), "=r"(r[43]), "=r"(r[44]), "=r"(r[45]), "=r"(r[46]), "=r"(r[47]), "=r"(r[48]), "=r"(r[49]), "=r"(r[50]), "=r"(r[51]), "=r"(r[52]), "=r"(r[53]), "=r"(r[54]), "=r"(r[55]), "=r"(r[56]), "=r"(r[57]), "=r"(r[58]), "=r"(r[59]), "=r"(r[60]), "=r"(r[61]), "=r"(r[62]), "=r"(r[63])
        : "r"(addr));
}
// 32 consecutive columns of this warp's 32 TMEM lanes, written from registers.
__device__ __forceinline__ void tmem_store32(uint32_t addr, const uint32_t* r) {
    asm volatile(
        "tcgen05.st.sync.aligned.32x32b.x32.b32 [%0], {%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16, %17, %18, %19, %20, %21, %22, %23, %24, %25, %26, %27, %28, %29, %30, %31, %32};"
        ::"r"(addr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]), "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15]), "r"(r[16]), "r"(r[17]), "r"(r[18]), "r"(r[19]), "r"(r[20]), "r"(r[21]), "r"(r[22]), "r"(r[23]), "r"(r[24]), "r"(r[25]), "r"(r[26]), "r"(r[27]), "r"(r[28]), "r"(r[29]), "r"(r[30]), "r"(r[31])
        : "memory");
}
// D (+)= A B with A from tensor memory (rows = lanes, two 16-bit elements of K per 32-bit column, the lower index in
// the lower half) and B from shared memory.
__device__ __forceinline__ void tc_mma_ts(uint32_t tmem_d, uint32_t tmem_a, uint64_t desc_b, uint32_t idesc, uint32_t accumulate) {
    asm volatile(
        "{\n\t.reg .pred p;\n\t"
        "setp.ne.b32 p, %4, 0;\n\t"
        "tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n\t}"
        ::"r"(tmem_d), "r"(tmem_a), "l"(desc_b), "r"(idesc), "r"(accumulate)
        : "memory");
}
__device__ __forceinline__ void tmem_store_wait() { asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory"); }

// A tile of `rows` rows x D elements as the tensor cores want a K-major operand (and, read with the other
// descriptor, an MN-major one): blocks of 64 elements (128 bytes) per row, 128-byte swizzle, 8 rows per 1024
// bytes, the blocks of one row `rows` * 128 bytes apart.  Byte offset of the 16-byte piece `piece` of row `row`.
template <int TILE_ROWS>
__device__ __forceinline__ uint32_t tile_offset(int row, int piece) {
    return (uint32_t)((piece >> 3) * (TILE_ROWS * 128) + (row >> 3) * 1024 + (row & 7) * 128 + (((piece & 7) ^ (row & 7)) << 4));
}
// K-major operand: see smem_desc in tcgen05.cuh.  MN-major operand with 128-byte swizzle: leading offset = the
// distance between two 64-element blocks of the MN dimension, stride offset = the distance between two groups
// of 8 rows of K.
__device__ __forceinline__ uint64_t smem_desc_mn(uint32_t addr, uint32_t leading_bytes, uint32_t stride_bytes) {
    uint64_t d = 0;
    d |= (uint64_t)((addr & 0x3FFFFu) >> 4);
    d |= (uint64_t)((leading_bytes >> 4) & 0x3FFFu) << 16;
    d |= (uint64_t)((stride_bytes >> 4) & 0x3FFFu) << 32;
    d |= (uint64_t)1 << 46;
    d |= (uint64_t)2 << 61;
    return d;
}
// Instruction descriptor as instr_desc(), with B taken MN-major.
__device__ __forceinline__ uint32_t instr_desc_b_mn(int m, int n) { return instr_desc(m, n) | (1u << 16); }
}  // namespace tc5
