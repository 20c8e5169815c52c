// Seeded synthetic weights on the device: a counter-based generator, one value per element.
#pragma once
#include "common.cuh"

namespace blok {

__device__ __forceinline__ uint64_t mix64(uint64_t z) {
  z += 0x9e3779b97f4a7c15ull;
  z = (z ^ (z >> 30)) * 0xbf58476d1ce4e5b9ull;
  z = (z ^ (z >> 27)) * 0x94d049bb133111ebull;
  return z ^ (z >> 31);
}
__device__ __forceinline__ float unit_normal(uint64_t key, uint64_t i) {
  uint64_t r = mix64(key ^ mix64(i));
  float u1 = ((uint32_t)(r >> 40) + 1.0f) * (1.0f / 16777217.0f);  // (0, 1)
  float u2 = (uint32_t)(r & 0xffffff) * (1.0f / 16777216.0f);
  return sqrtf(-2.0f * logf(u1)) * cosf(6.28318530718f * u2);
}

// `first` is the index, in the whole tensor, of the first element generated: a rank's shard of the experts holds exactly
// the values the unsharded tensor has at those positions.
static __global__ void fill_words_kernel(uint32_t *p, size_t n, uint64_t key, size_t first) {
  size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i < n) p[i] = (uint32_t)mix64(key ^ mix64(i + first));
}
// mode 0: N(0, std); mode 1: |N(0, std)|; mode 2: constant std
static __global__ void fill_bf16_kernel(uint16_t *p, size_t n, uint64_t key, float std, int mode, size_t first) {
  size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= n) return;
  float v = mode == 2 ? std : unit_normal(key, i + first) * std;
  if (mode == 1) v = fabsf(v);
  p[i] = f32_to_bf16_bits(v);
}
static __global__ void fill_f32_kernel(float *p, size_t n, uint64_t key, float std) {
  size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i < n) p[i] = unit_normal(key, i) * std;
}

}  // namespace blok
