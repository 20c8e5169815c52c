// Routing by a table of token ids, and the experts of a few tokens.  The table fixes a layer's routing before the layer
// runs, so one launch plans every layer of a step: assignments in expert order, in tiles of up to 128 rows for the grouped
// GEMM (gemm_tma.cu).  Few assignments skip the plan: a mat-vec kernel reads each assignment's expert from the table.
#include "common.cuh"
#include "gemm_tma.h"
#include "stack_kernels.h"

namespace blok {

constexpr int kEpThreads = 1024;

__global__ void __launch_bounds__(kEpThreads) expert_plan_kernel(const ExpertPlanArgs *__restrict__ layers, const uint32_t *__restrict__ ids,
                                                                 int vocab, int T) {
  extern __shared__ int s_count[];  // [experts] assignments, then the next free row
  __shared__ int s_rows[kEpThreads], s_tiles[kEpThreads];
  const ExpertPlanArgs L = layers[blockIdx.x];
  const int tid = threadIdx.x, A = T * L.top;
  for (int e = tid; e < L.experts; e += kEpThreads) s_count[e] = 0;
  __syncthreads();
  auto expert = [&](int a) {
    const uint32_t id = min(ids[a / L.top], (uint32_t)vocab - 1);
    return L.table[(size_t)id * L.top + a % L.top];
  };
  for (int a = tid; a < A; a += kEpThreads) atomicAdd(&s_count[expert(a)], 1);
  __syncthreads();
  // every thread sums a range of experts, the block scans the sums
  const int per = (L.experts + kEpThreads - 1) / kEpThreads;
  const int e0 = min(tid * per, L.experts), e1 = min(e0 + per, L.experts);
  int rows = 0, tiles = 0;
  for (int e = e0; e < e1; ++e) rows += s_count[e], tiles += (s_count[e] + kGtTileRows - 1) / kGtTileRows;
  s_rows[tid] = rows;
  s_tiles[tid] = tiles;
  __syncthreads();
  for (int o = 1; o < kEpThreads; o <<= 1) {
    const int r = tid >= o ? s_rows[tid - o] : 0, t = tid >= o ? s_tiles[tid - o] : 0;
    __syncthreads();
    s_rows[tid] += r;
    s_tiles[tid] += t;
    __syncthreads();
  }
  int row = s_rows[tid] - rows, tile = s_tiles[tid] - tiles;
  for (int e = e0; e < e1; ++e) {
    const int n = s_count[e];
    for (int at = 0; at < n; at += kGtTileRows, ++tile) {
      L.plan.tile_expert[tile] = e;
      L.plan.tile_start[tile] = row + at;
      L.plan.tile_count[tile] = min(kGtTileRows, n - at);
    }
    s_count[e] = row;
    row += n;
  }
  if (tid == kEpThreads - 1) *L.plan.num_tiles = s_tiles[tid];
  __syncthreads();
  for (int a = tid; a < A; a += kEpThreads) L.plan.at[a] = atomicAdd(&s_count[expert(a)], 1);
}

int expert_plan_max_tiles(int assignments, int experts) {
  const int groups = assignments < experts ? assignments : experts;  // experts with at least one row
  return assignments / kGtTileRows + groups;
}

int launch_expert_plan(const ExpertPlanArgs *layers, int n_layers, const uint32_t *ids, int vocab, int T, cudaStream_t stream) {
  expert_plan_kernel<<<n_layers, kEpThreads, kMaxTableExperts * sizeof(int), stream>>>(layers, ids, vocab, T);
  return launch_status("expert_plan_kernel");
}

// A warp owns kEgRows weight rows; lanes take 16 bytes (8 weights) at a time, x comes from shared memory.
constexpr int kEgWarps = 8, kEgRows = 2;

template <bool XF32>
__device__ __forceinline__ void eg_fetch(const unsigned char *xs, int k, float (&x)[8]) {
  if (XF32) {
    const float4 a = *reinterpret_cast<const float4 *>(xs + (size_t)k * 4), b = *reinterpret_cast<const float4 *>(xs + (size_t)k * 4 + 16);
    x[0] = a.x, x[1] = a.y, x[2] = a.z, x[3] = a.w, x[4] = b.x, x[5] = b.y, x[6] = b.z, x[7] = b.w;
  } else {
    const uint4 v = *reinterpret_cast<const uint4 *>(xs + (size_t)k * 2);
    x[0] = bf16lo(v.x), x[1] = bf16hi(v.x), x[2] = bf16lo(v.y), x[3] = bf16hi(v.y);
    x[4] = bf16lo(v.z), x[5] = bf16hi(v.z), x[6] = bf16lo(v.w), x[7] = bf16hi(v.w);
  }
}
__device__ __forceinline__ float eg_dot(uint4 w, const float (&x)[8], float acc) {
  acc = fmaf(bf16lo(w.x), x[0], acc);
  acc = fmaf(bf16hi(w.x), x[1], acc);
  acc = fmaf(bf16lo(w.y), x[2], acc);
  acc = fmaf(bf16hi(w.y), x[3], acc);
  acc = fmaf(bf16lo(w.z), x[4], acc);
  acc = fmaf(bf16hi(w.z), x[5], acc);
  acc = fmaf(bf16lo(w.w), x[6], acc);
  return fmaf(bf16hi(w.w), x[7], acc);
}

template <bool XF32>
__global__ void __launch_bounds__(kEgWarps * 32)
    expert_gemv_kernel(const uint16_t *__restrict__ w, int R, int K, const int *__restrict__ table, const uint32_t *__restrict__ ids, int vocab, int top,
                       const void *__restrict__ x, int shared_x, int relu2, void *__restrict__ y, int y_f32) {
  extern __shared__ __align__(16) unsigned char xs[];
  const int a = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const uint32_t id = min(ids[a / top], (uint32_t)vocab - 1);
  const int e = table[(size_t)id * top + a % top];
  const size_t xbytes = (size_t)K * (XF32 ? 4 : 2);
  const uint4 *xsrc = reinterpret_cast<const uint4 *>(static_cast<const unsigned char *>(x) + (size_t)(shared_x ? a / top : a) * xbytes);
  for (int i = tid; i < (int)(xbytes / 16); i += blockDim.x) reinterpret_cast<uint4 *>(xs)[i] = xsrc[i];
  const int r0 = (blockIdx.y * kEgWarps + warp) * kEgRows;
  const int units = K / 8;
  const uint4 *wr[kEgRows];
#pragma unroll
  for (int j = 0; j < kEgRows; ++j) wr[j] = reinterpret_cast<const uint4 *>(w + ((size_t)e * R + min(r0 + j, R - 1)) * K);
  __syncthreads();
  if (r0 >= R) return;
  float acc[kEgRows] = {};
  int u = lane;
  for (; u + 96 < units; u += 128) {  // four loads of each row in flight
    uint4 v[kEgRows][4];
#pragma unroll
    for (int q = 0; q < 4; ++q)
#pragma unroll
      for (int j = 0; j < kEgRows; ++j) v[j][q] = ldg_stream(wr[j] + u + 32 * q);
#pragma unroll
    for (int q = 0; q < 4; ++q) {
      float xv[8];
      eg_fetch<XF32>(xs, (u + 32 * q) * 8, xv);
#pragma unroll
      for (int j = 0; j < kEgRows; ++j) acc[j] = eg_dot(v[j][q], xv, acc[j]);
    }
  }
  for (; u < units; u += 32) {
    float xv[8];
    eg_fetch<XF32>(xs, u * 8, xv);
#pragma unroll
    for (int j = 0; j < kEgRows; ++j) acc[j] = eg_dot(ldg_stream(wr[j] + u), xv, acc[j]);
  }
#pragma unroll
  for (int j = 0; j < kEgRows; ++j) {
    float v = warp_sum(acc[j]);
    if (lane == 0 && r0 + j < R) {
      if (relu2) {
        v = fmaxf(v, 0.f);
        v *= v;
      }
      const size_t o = (size_t)a * R + r0 + j;
      if (y_f32) static_cast<float *>(y)[o] = v;
      else static_cast<uint16_t *>(y)[o] = f32_to_bf16_bits(v);
    }
  }
}

int launch_expert_gemv(const uint16_t *w, int R, int K, const int *table, const uint32_t *ids, int vocab, int top, int T, const void *x, bool x_f32,
                       bool shared_x, bool relu2, void *y, bool y_f32, cudaStream_t stream) {
  const size_t smem = (size_t)K * (x_f32 ? 4 : 2);
  BLOK_REQUIRE(K % 8 == 0 && smem <= 200 * 1024, BLOK_ERR_SHAPE, "expert mat-vec: %d columns", K);
  const dim3 grid(T * top, (R + kEgWarps * kEgRows - 1) / (kEgWarps * kEgRows));
  if (x_f32) {
    if (smem > 48 * 1024) BLOK_CUDA(cudaFuncSetAttribute(expert_gemv_kernel<true>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    expert_gemv_kernel<true><<<grid, kEgWarps * 32, smem, stream>>>(w, R, K, table, ids, vocab, top, x, shared_x, relu2, y, y_f32);
  } else {
    if (smem > 48 * 1024) BLOK_CUDA(cudaFuncSetAttribute(expert_gemv_kernel<false>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    expert_gemv_kernel<false><<<grid, kEgWarps * 32, smem, stream>>>(w, R, K, table, ids, vocab, top, x, shared_x, relu2, y, y_f32);
  }
  return launch_status("expert_gemv_kernel");
}

}  // namespace blok
