// The merge behind the split-context attention cores (mla.cu, latent_attn.cu, grouped_attn.cu).
#pragma once
#include "common.cuh"

namespace blok {

// ---------------------------------------------------------------------------
// Merge of the split-KV partial results.  grid = (heads, B), 128 threads.
//   part_o fp32 [B, splits, heads, kv_rank] unnormalised, part_ml fp32 [B, splits, heads, 2] = (max, sum)
// Rows of o_lat are ldo values apart (0: heads * kv_rank).  gate, optional: bf16 [B, ld_gate]; head h's output times
// sigmoid(gate[b][h]).
// ---------------------------------------------------------------------------
static __global__ void mla_merge_kernel(const float *__restrict__ part_o, const float *__restrict__ part_ml, int splits,
                                 int heads, int kv_rank, uint16_t *__restrict__ o_lat, int ldo = 0,
                                 const uint16_t *__restrict__ gate = nullptr, int ld_gate = 0) {
  extern __shared__ float s_wt[];  // [splits] weight of every split: exp(m_s - M), 0 for an empty split
  __shared__ float s_red[2][4];
  const int h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x;
  const float *ml = part_ml + ((size_t)b * splits * heads + h) * 2;  // split s at + s * heads * 2
  float M = -INFINITY;
  for (int s = tid; s < splits; s += blockDim.x) M = fmaxf(M, ml[(size_t)s * heads * 2]);
  M = warp_max(M);
  if ((tid & 31) == 0) s_red[0][tid >> 5] = M;
  __syncthreads();
  M = fmaxf(fmaxf(s_red[0][0], s_red[0][1]), fmaxf(s_red[0][2], s_red[0][3]));
  float L = 0.f;
  for (int s = tid; s < splits; s += blockDim.x) {
    const float m = ml[(size_t)s * heads * 2];
    const float wt = m != -INFINITY ? expf(m - M) : 0.f;
    s_wt[s] = wt;
    L += wt * ml[(size_t)s * heads * 2 + 1];
  }
  L = warp_sum(L);
  if ((tid & 31) == 0) s_red[1][tid >> 5] = L;
  __syncthreads();
  L = (s_red[1][0] + s_red[1][1]) + (s_red[1][2] + s_red[1][3]);
  float inv = L > 0.f ? 1.0f / L : 0.f;
  if (gate) inv *= 1.0f / (1.0f + expf(-bf16_bits_to_f32(gate[(size_t)b * ld_gate + h])));
  if (!ldo) ldo = heads * kv_rank;
  const float *po = part_o + ((size_t)b * splits * heads + h) * kv_rank;  // split s at + s * heads * kv_rank
  // four columns per thread, eight splits' worth of loads in flight per thread: the partial results (B x splits x 128 KB)
  // come from L2 or HBM, and the kernel is as fast as it keeps bytes in flight.  Each column still adds its splits in
  // ascending order.
  const float4 *po4 = reinterpret_cast<const float4 *>(po);
  const size_t stride4 = (size_t)heads * kv_rank / 4;
  for (int j4 = tid; j4 < kv_rank / 4; j4 += blockDim.x) {
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
    int s = 0;
    for (; s + 8 <= splits; s += 8) {
      float4 v[8];
#pragma unroll
      for (int i = 0; i < 8; ++i) v[i] = __ldg(po4 + (size_t)(s + i) * stride4 + j4);
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const float wt = s_wt[s + i];
        acc.x = fmaf(wt, v[i].x, acc.x);
        acc.y = fmaf(wt, v[i].y, acc.y);
        acc.z = fmaf(wt, v[i].z, acc.z);
        acc.w = fmaf(wt, v[i].w, acc.w);
      }
    }
    for (; s < splits; ++s) {
      const float4 v = __ldg(po4 + (size_t)s * stride4 + j4);
      const float wt = s_wt[s];
      acc.x = fmaf(wt, v.x, acc.x);
      acc.y = fmaf(wt, v.y, acc.y);
      acc.z = fmaf(wt, v.z, acc.z);
      acc.w = fmaf(wt, v.w, acc.w);
    }
    uint2 o;
    o.x = pack_bf16x2(acc.x * inv, acc.y * inv);
    o.y = pack_bf16x2(acc.z * inv, acc.w * inv);
    *reinterpret_cast<uint2 *>(o_lat + (size_t)b * ldo + (size_t)h * kv_rank + (size_t)j4 * 4) = o;
  }
}

}  // namespace blok
