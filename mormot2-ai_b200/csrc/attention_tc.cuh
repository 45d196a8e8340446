// Pieces that the attention kernels on tcgen05 share: descriptors of value tiles, tensor-memory
// loads and stores of a row, packed arithmetic for the softmax.
#pragma once
#include "tc_common.cuh"

// Operand descriptor of an MN-major tile written by TMA with the 128-byte swizzle: rows of 64
// values (128 bytes) are consecutive values of the K dimension (here: keys), 8 rows make a
// swizzle atom of 1024 bytes, the atoms of further keys follow one another (stride byte
// offset 1024); a second block of 64 values along N would lie `lbo` bytes on (unused here:
// every MMA takes 64 values of N).
__device__ __forceinline__ uint64_t umma_desc_mn128(uint32_t smem_addr, uint32_t lbo) {
  uint64_t d = 0;
  d |= (uint64_t)((smem_addr >> 4) & 0x3FFF);
  d |= (uint64_t)((lbo >> 4) & 0x3FFF) << 16;
  d |= (uint64_t)(1024 >> 4) << 32;
  d |= (uint64_t)1 << 46;
  d |= (uint64_t)2 << 61;
  return d;
}

__device__ __forceinline__ void tmem_st16(uint32_t taddr, const float* v) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], "
      "{%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16};\n"
      ::"r"(taddr), "r"(__float_as_uint(v[0])), "r"(__float_as_uint(v[1])),
        "r"(__float_as_uint(v[2])), "r"(__float_as_uint(v[3])), "r"(__float_as_uint(v[4])),
        "r"(__float_as_uint(v[5])), "r"(__float_as_uint(v[6])), "r"(__float_as_uint(v[7])),
        "r"(__float_as_uint(v[8])), "r"(__float_as_uint(v[9])), "r"(__float_as_uint(v[10])),
        "r"(__float_as_uint(v[11])), "r"(__float_as_uint(v[12])), "r"(__float_as_uint(v[13])),
        "r"(__float_as_uint(v[14])), "r"(__float_as_uint(v[15]))
      : "memory");
}
__device__ __forceinline__ void tmem_wait_st() {
  asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
}
// 2^x by the special-function unit (x <= 8 here; -inf gives 0)
__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// two float32 values in one 64-bit register, and arithmetic on both at once
__device__ __forceinline__ unsigned long long pack2(float a, float b) {
  unsigned long long r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
  return r;
}
__device__ __forceinline__ void unpack2(unsigned long long r, float& a, float& b) {
  asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(r));
}
__device__ __forceinline__ unsigned long long fma2(unsigned long long a, unsigned long long b,
                                                   unsigned long long c) {
  unsigned long long r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
__device__ __forceinline__ unsigned long long add2(unsigned long long a, unsigned long long b) {
  unsigned long long r;
  asm("add.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}
// the largest of three in one instruction
__device__ __forceinline__ float max3(float a, float b, float c) {
  float y;
  asm("max.f32 %0, %1, %2, %3;" : "=f"(y) : "f"(a), "f"(b), "f"(c));
  return y;
}
__device__ __forceinline__ void fence_async_smem() {
  asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
}

// 64 consecutive float32 columns of this thread's TMEM lane: four loads in flight, one wait.
// The loaded registers pass through the wait (and through empty statements after it) so that
// no use of them can be scheduled before it.
#define AT_LD16(R, OFF)                                                                          \
  asm volatile(                                                                                  \
      "tcgen05.ld.sync.aligned.32x32b.x16.b32"                                                   \
      "{%0, %1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15}, [%16];\n"         \
      : "=r"(R[0]), "=r"(R[1]), "=r"(R[2]), "=r"(R[3]), "=r"(R[4]), "=r"(R[5]), "=r"(R[6]),      \
        "=r"(R[7]), "=r"(R[8]), "=r"(R[9]), "=r"(R[10]), "=r"(R[11]), "=r"(R[12]), "=r"(R[13]),  \
        "=r"(R[14]), "=r"(R[15])                                                                 \
      : "r"(taddr + OFF))
#define AT_HOLD16(TEXT, R)                                                                       \
  asm volatile(TEXT                                                                              \
               : "+r"(R[0]), "+r"(R[1]), "+r"(R[2]), "+r"(R[3]), "+r"(R[4]), "+r"(R[5]),         \
                 "+r"(R[6]), "+r"(R[7]), "+r"(R[8]), "+r"(R[9]), "+r"(R[10]), "+r"(R[11]),       \
                 "+r"(R[12]), "+r"(R[13]), "+r"(R[14]), "+r"(R[15])                              \
               :                                                                                 \
               : "memory")
__device__ __forceinline__ void tmem_ld64(uint32_t taddr, float* v) {
  uint32_t a[16], b[16], c[16], d[16];
  AT_LD16(a, 0);
  AT_LD16(b, 16);
  AT_LD16(c, 32);
  AT_LD16(d, 48);
  AT_HOLD16("tcgen05.wait::ld.sync.aligned;", a);
  AT_HOLD16("", b);
  AT_HOLD16("", c);
  AT_HOLD16("", d);
#pragma unroll
  for (int i = 0; i < 16; ++i) {
    v[i] = __uint_as_float(a[i]);
    v[16 + i] = __uint_as_float(b[i]);
    v[32 + i] = __uint_as_float(c[i]);
    v[48 + i] = __uint_as_float(d[i]);
  }
}

// 16 packed words (32 bfloat16 values) into this thread's TMEM lane
__device__ __forceinline__ void tmem_st16_u32(uint32_t taddr, const uint32_t* w) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], "
      "{%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16};\n"
      ::"r"(taddr), "r"(w[0]), "r"(w[1]), "r"(w[2]), "r"(w[3]), "r"(w[4]), "r"(w[5]), "r"(w[6]),
        "r"(w[7]), "r"(w[8]), "r"(w[9]), "r"(w[10]), "r"(w[11]), "r"(w[12]), "r"(w[13]),
        "r"(w[14]), "r"(w[15])
      : "memory");
}

// D[tmem] (+)= A[tmem] · B[smem]: the first operand (128 rows x 16 bfloat16 values, two values
// a 32-bit column, 8 columns) lies in tensor memory. Issued by one thread.
__device__ __forceinline__ void umma_bf16_ts(uint32_t tmem_d, uint32_t tmem_a, uint64_t desc_b,
                                             uint32_t idesc, uint32_t accumulate) {
  asm volatile(
      "{\n\t.reg .pred p;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n\t}\n"
      ::"r"(tmem_d), "r"(tmem_a), "l"(desc_b), "r"(idesc), "r"(accumulate)
      : "memory");
}
