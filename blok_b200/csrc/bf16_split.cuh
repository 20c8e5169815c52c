// fp32 values as operands of bf16 tensor-core products: v = hi + mid + lo with each part a bf16 value.  Three parts carry
// 24 mantissa bits, so a product with a bf16 operand accumulated in fp32 is what fp32 arithmetic gives: attention weights,
// decayed keys and recurrent states go through it.
#pragma once
#include "common.cuh"

namespace blok {

constexpr int kSplitParts = 3;

// Both values rounded to nearest even, a in the low half, in one instruction.
__device__ __forceinline__ uint32_t pack_pair(float a, float b) {
  uint32_t r;
  asm("cvt.rn.bf16x2.f32 %0, %1, %2;" : "=r"(r) : "f"(b), "f"(a));
  return r;
}
// Parts of the pair (a, b) as packed bf16 pairs, a in the low half.
__device__ __forceinline__ void split_pair(float a, float b, uint32_t (&parts)[kSplitParts]) {
#pragma unroll
  for (int p = 0; p < kSplitParts; ++p) {
    const uint32_t v = pack_pair(a, b);
    parts[p] = v;
    a -= bf16lo(v);
    b -= bf16hi(v);
  }
}
__device__ __forceinline__ void ldsm4(uint32_t addr, uint32_t &r0, uint32_t &r1, uint32_t &r2, uint32_t &r3) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldsm4_t(uint32_t addr, uint32_t &r0, uint32_t &r1, uint32_t &r2, uint32_t &r3) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3)
               : "r"(addr)
               : "memory");
}
__device__ __forceinline__ void cp_async16(uint32_t dst, const void *src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}
// Fragment addresses in a row-major bf16 tile of `pitch` bytes per row, lane `lane`:
// A operand, rows m0.. and columns k0..: the four 8 x 8 blocks (m, k), (m + 8, k), (m, k + 8), (m + 8, k + 8)
__device__ __forceinline__ uint32_t frag_a(uint32_t base, int m0, int k0, int pitch, int lane) {
  return base + (uint32_t)((m0 + (lane & 15)) * pitch + (k0 + (lane >> 4) * 8) * 2);
}
// A operand from a tile stored transposed (row = k, column = m), read with ldsm4_t
__device__ __forceinline__ uint32_t frag_a_t(uint32_t base, int m0, int k0, int pitch, int lane) {
  return base + (uint32_t)((k0 + (lane & 7) + ((lane >> 4) << 3)) * pitch + (m0 + ((lane >> 3) & 1) * 8) * 2);
}
// B operand of two n8 tiles from a tile with row = n, column = k: (r0, r1) the first tile, (r2, r3) the second
__device__ __forceinline__ uint32_t frag_b(uint32_t base, int n0, int k0, int pitch, int lane) {
  return base + (uint32_t)((n0 + (lane & 7) + ((lane >> 4) << 3)) * pitch + (k0 + ((lane >> 3) & 1) * 8) * 2);
}
// B operand of two n8 tiles from a tile with row = k, column = n, read with ldsm4_t
__device__ __forceinline__ uint32_t frag_b_t(uint32_t base, int n0, int k0, int pitch, int lane) {
  return base + (uint32_t)((k0 + (lane & 15)) * pitch + (n0 + (lane >> 4) * 8) * 2);
}

}  // namespace blok
