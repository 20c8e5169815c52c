// Hyper-connected residual streams and the Dynamic-Tanh norm, in one elementwise pass between two sublayers: the streams
// take in the sublayer's output (mixing among themselves), the next sublayer's input is combined from the new streams,
// normed and written where the next product reads it.  A Dynamic Tanh needs no mean, so nothing here waits for a
// reduction: a thread owns four columns of one token in every stream.  All of it is fp32; h alone is rounded.
#include "common.cuh"
#include "stack_kernels.h"

namespace blok {

__device__ __forceinline__ float4 rs_fma(float a, float4 x, float4 y) {
  return make_float4(fmaf(a, x.x, y.x), fmaf(a, x.y, y.y), fmaf(a, x.z, y.z), fmaf(a, x.w, y.w));
}

// MAXS: streams kept in registers (a.streams <= MAXS).
template <int MAXS>
__global__ void __launch_bounds__(128) streams_step_kernel(const StreamsStep a) {
  __shared__ float s_mix[MAXS * MAXS], s_out[MAXS], s_in[MAXS];
  const int S = a.streams;
  for (int i = threadIdx.x; i < S * S; i += blockDim.x) s_mix[i] = a.mix ? a.mix[i] : 0.f;
  if (threadIdx.x < S) {
    s_out[threadIdx.x] = a.out ? a.out[threadIdx.x] : 0.f;
    s_in[threadIdx.x] = a.in ? a.in[threadIdx.x] : 1.f;
  }
  __syncthreads();
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * 4;
  if (c >= a.width) return;
  const int i = blockIdx.y, t = a.rows ? a.rows[i] : i;
  float *xt = a.x + (size_t)t * S * a.width + c;
  float4 x[MAXS];
  if (a.ids) {
    const uint32_t id = min(a.ids[t], (uint32_t)a.vocab - 1);
    const uint2 e = *reinterpret_cast<const uint2 *>(a.embed + (size_t)id * a.width + c);
    const float4 v = make_float4(bf16lo(e.x), bf16hi(e.x), bf16lo(e.y), bf16hi(e.y));
#pragma unroll
    for (int s = 0; s < MAXS; ++s) x[s] = v;
  } else {
    float4 old[MAXS];
#pragma unroll
    for (int s = 0; s < MAXS; ++s)
      if (s < S) old[s] = *reinterpret_cast<const float4 *>(xt + (size_t)s * a.width);
    if (a.y_rows) {
      float4 y = make_float4(0.f, 0.f, 0.f, 0.f);
      for (int k = 0; k < a.parts; ++k) {
        const int at = t * a.parts + k;
        const float4 v = *reinterpret_cast<const float4 *>(a.y_rows + (size_t)(a.part_at ? a.part_at[at] : at) * a.width + c);
        y = make_float4(y.x + v.x, y.y + v.y, y.z + v.z, y.w + v.w);
      }
      y = make_float4(y.x * a.part_scale, y.y * a.part_scale, y.z * a.part_scale, y.w * a.part_scale);
#pragma unroll
      for (int to = 0; to < MAXS; ++to)
        if (to < S) {
          x[to] = make_float4(s_out[to] * y.x, s_out[to] * y.y, s_out[to] * y.z, s_out[to] * y.w);
#pragma unroll
          for (int s = 0; s < MAXS; ++s)
            if (s < S) x[to] = rs_fma(s_mix[s * S + to], old[s], x[to]);
        }
    } else {
#pragma unroll
      for (int s = 0; s < MAXS; ++s) x[s] = old[s];
    }
  }
  if (a.store_x && (a.ids || a.y_rows)) {
#pragma unroll
    for (int s = 0; s < MAXS; ++s)
      if (s < S) *reinterpret_cast<float4 *>(xt + (size_t)s * a.width) = x[s];
  }
  if (a.sum) {
    float4 u = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int s = 0; s < MAXS; ++s)
      if (s < S) u = rs_fma(1.f, x[s], u);
    const float v[4] = {u.x, u.y, u.z, u.w};
    for (int j = 0; j < 4; ++j)
      if (c + j < a.true_width) a.sum[(size_t)t * a.true_width + c + j] = v[j];
  }
  if (a.norm_w) {
    float4 u = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int s = 0; s < MAXS; ++s)
      if (s < S) u = rs_fma(s_in[s], x[s], u);
    const float4 w = *reinterpret_cast<const float4 *>(a.norm_w + c), b = *reinterpret_cast<const float4 *>(a.norm_b + c);
    const float4 h = make_float4(fmaf(tanhf(a.alpha * u.x), w.x, b.x), fmaf(tanhf(a.alpha * u.y), w.y, b.y),
                                 fmaf(tanhf(a.alpha * u.z), w.z, b.z), fmaf(tanhf(a.alpha * u.w), w.w, b.w));
    for (int k = 0; k < a.copies; ++k) {
      const size_t at = (size_t)(a.copy_at ? a.copy_at[i * a.copies + k] : i) * a.width + c;
      if (a.h_f32) *reinterpret_cast<float4 *>(static_cast<float *>(a.h) + at) = h;
      else *reinterpret_cast<uint2 *>(static_cast<uint16_t *>(a.h) + at) = make_uint2(pack_bf16x2(h.x, h.y), pack_bf16x2(h.z, h.w));
    }
  }
}

int launch_streams_step(const StreamsStep &a, cudaStream_t stream) {
  BLOK_REQUIRE(a.T >= 1 && a.width % 4 == 0 && a.streams >= 1 && a.streams <= kMaxStreams, BLOK_ERR_SHAPE, "streams step: T %d, width %d, streams %d",
               a.T, a.width, a.streams);
  const dim3 grid((a.width / 4 + 127) / 128, a.T);
  if (a.streams == 1) streams_step_kernel<1><<<grid, 128, 0, stream>>>(a);
  else if (a.streams == 2) streams_step_kernel<2><<<grid, 128, 0, stream>>>(a);
  else if (a.streams <= 4) streams_step_kernel<4><<<grid, 128, 0, stream>>>(a);
  else streams_step_kernel<kMaxStreams><<<grid, 128, 0, stream>>>(a);
  return launch_status("streams_step_kernel");
}

}  // namespace blok
