// Helpers of a TMA-fed tcgen05 pipeline: bounded mbarrier waits, tile copies, shared-memory descriptors, the MMA and its
// commit.  No copy here is multicast.
#pragma once
#include <cuda.h>

#include "common.cuh"
#include "tmem_io.cuh"

namespace blok {

constexpr unsigned kTpSpinLimit = 1u << 21;

__device__ __forceinline__ void tp_mbar_init(uint32_t mbar, uint32_t count) {
  asm volatile("mbarrier.init.shared::cta.b64 [%0], %1;" ::"r"(mbar), "r"(count) : "memory");
}
__device__ __forceinline__ void tp_mbar_init_fence() { asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory"); }
__device__ __forceinline__ void tp_expect_tx(uint32_t mbar, uint32_t bytes) {
  asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(mbar), "r"(bytes) : "memory");
}
__device__ __forceinline__ void tp_arrive(uint32_t mbar) {
  asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(mbar) : "memory");
}
// Waits for the phase of the given parity; false when the limit ran out.
__device__ __forceinline__ bool tp_wait(uint32_t mbar, uint32_t parity) {
  for (unsigned it = 0; it < kTpSpinLimit; ++it) {
    uint32_t ok;
    asm volatile(
        "{\n\t"
        ".reg .pred p;\n\t"
        "mbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2;\n\t"
        "selp.u32 %0, 1, 0, p;\n\t"
        "}\n"
        : "=r"(ok)
        : "r"(mbar), "r"(parity)
        : "memory");
    if (ok) return true;
    if (it > 64) __nanosleep(64);
  }
  return false;
}
// True in one lane of a converged warp.
__device__ __forceinline__ bool tp_elect() {
  uint32_t is;
  asm volatile(
      "{\n\t"
      ".reg .pred p;\n\t"
      "elect.sync _|p, 0xffffffff;\n\t"
      "selp.u32 %0, 1, 0, p;\n\t"
      "}\n"
      : "=r"(is));
  return is != 0;
}
// One box of a 2-D tensor map (x: column in elements, 16-byte aligned; y: row) into shared memory, counted on the mbarrier.
__device__ __forceinline__ void tp_load_2d(uint32_t dst, const CUtensorMap *map, int x, int y, uint32_t mbar) {
  asm volatile("cp.async.bulk.tensor.2d.shared::cluster.global.tile.mbarrier::complete_tx::bytes [%0], [%1, {%2, %3}], [%4];" ::"r"(dst),
               "l"(map), "r"(x), "r"(y), "r"(mbar)
               : "memory");
}
// K-major operand in the 128-byte swizzle: rows of 128 bytes (64 bf16), 1,024 bytes between 8-row groups.  A K = 16 step
// inside the row advances the start address by 32 bytes.
__device__ __forceinline__ uint64_t tp_desc_k_sw128(uint32_t saddr) {
  return (uint64_t)((saddr & 0x3FFFFu) >> 4) | (1ull << 16) | ((uint64_t)(1024 >> 4) << 32) | (1ull << 46) | (2ull << 61);
}
// MN-major operand in the 128-byte swizzle: 64 contiguous elements of M or N per row, `lead` bytes between 64-element chunks,
// 1,024 bytes between groups of 8 along K (a K = 16 step advances by 2,048).
__device__ __forceinline__ uint64_t tp_desc_mn_sw128(uint32_t saddr, uint32_t lead) {
  return (uint64_t)((saddr & 0x3FFFFu) >> 4) | ((uint64_t)(lead >> 4) << 16) | ((uint64_t)(1024 >> 4) << 32) | (1ull << 46) | (2ull << 61);
}
// bf16 x bf16 -> fp32, M = 128, both operands K-major.
__host__ __device__ constexpr uint32_t tp_idesc_bf16(int n) {
  return (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(n >> 3) << 17) | ((128u >> 4) << 24);
}
__device__ __forceinline__ void tp_mma(uint32_t tmem_d, uint64_t adesc, uint64_t bdesc, uint32_t idesc, uint32_t accumulate) {
  asm volatile(
      "{\n\t"
      ".reg .pred p;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n\t"
      "}\n" ::"r"(tmem_d), "l"(adesc), "l"(bdesc), "r"(idesc), "r"(accumulate)
      : "memory");
}
// A from tensor memory (lane = row, two bf16 per 32-bit column, 8 columns per K = 16 step).
__device__ __forceinline__ void tp_mma_ts(uint32_t tmem_d, uint32_t tmem_a, uint64_t bdesc, uint32_t idesc, uint32_t accumulate) {
  asm volatile(
      "{\n\t"
      ".reg .pred p;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n\t"
      "}\n" ::"r"(tmem_d), "r"(tmem_a), "l"(bdesc), "r"(idesc), "r"(accumulate)
      : "memory");
}
__device__ __forceinline__ void tp_commit(uint32_t mbar) {
  asm volatile("tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];" ::"r"(mbar) : "memory");
}
__device__ __forceinline__ void tp_tmem_alloc(uint32_t smem_word, uint32_t cols) {
  asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_word), "r"(cols) : "memory");
  asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
}
__device__ __forceinline__ void tp_tmem_free(uint32_t tmem, uint32_t cols) {
  asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(cols) : "memory");
}

}  // namespace blok
