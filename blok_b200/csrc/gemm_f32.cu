// Products in true fp32 (fused multiply-add on the CUDA cores) for models opened with BLOK_DTYPE_F32: bf16 weight values,
// fp32 activations.  64 x 64 tiles, 4 x 4 outputs per thread.
#include "common.cuh"
#include "stack_kernels.h"

namespace blok {

constexpr int kGfTile = 64, kGfStep = 16;

__global__ void __launch_bounds__(256) gemm_f32_kernel(const GemmF32 g) {
  __shared__ float xs[kGfStep][kGfTile + 4], ws[kGfStep][kGfTile + 4];
  const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
  const int r0 = blockIdx.x * kGfTile, t0 = blockIdx.y * kGfTile;
  const uint16_t *w = g.w + (size_t)blockIdx.z * g.w_stride;
  const float *x = g.x + (size_t)blockIdx.z * g.x_stride;
  float *y = g.y + (size_t)blockIdx.z * g.y_stride;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < g.K; k0 += kGfStep) {
    for (int i = tid; i < kGfTile * kGfStep; i += 256) {
      const int row = i / kGfStep, k = i % kGfStep;
      const bool in_k = k0 + k < g.K;
      xs[k][row] = in_k && t0 + row < g.T ? x[(size_t)(t0 + row) * g.ldx + k0 + k] : 0.f;
      ws[k][row] = in_k && r0 + row < g.R ? bf16_bits_to_f32(w[(size_t)(r0 + row) * g.ldw + k0 + k]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kGfStep; ++k) {
      float a[4], b[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) a[i] = xs[k][ty * 4 + i], b[i] = ws[k][tx * 4 + i];
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
    }
    __syncthreads();
  }
  for (int i = 0; i < 4; ++i)
    for (int j = 0; j < 4; ++j) {
      const int t = t0 + ty * 4 + i, r = r0 + tx * 4 + j;
      if (t < g.T && r < g.R) y[(size_t)t * g.ldy + r] = acc[i][j];
    }
}

int launch_gemm_f32(const GemmF32 &g, cudaStream_t stream) {
  BLOK_REQUIRE(g.R >= 1 && g.K >= 1 && g.T >= 1 && g.batch >= 1, BLOK_ERR_SHAPE, "fp32 product: T %d, R %d, K %d", g.T, g.R, g.K);
  gemm_f32_kernel<<<dim3((g.R + kGfTile - 1) / kGfTile, (g.T + kGfTile - 1) / kGfTile, g.batch), 256, 0, stream>>>(g);
  return launch_status("gemm_f32_kernel");
}

// out[t, r] = silu(x[t, r]) * x[t, cols + r]
__global__ void __launch_bounds__(256) swiglu_f32_kernel(const float *__restrict__ x, float *__restrict__ out, int cols, long n) {
  const long i = (long)blockIdx.x * 256 + threadIdx.x;
  if (i >= n) return;
  const float *p = x + i / cols * 2 * cols + i % cols;
  const float z = p[0];
  out[i] = z / (1.0f + expf(-z)) * p[cols];
}

int launch_swiglu_f32(const float *x, float *out, int cols, int T, cudaStream_t stream) {
  const long n = (long)cols * T;
  swiglu_f32_kernel<<<(unsigned)((n + 255) / 256), 256, 0, stream>>>(x, out, cols, n);
  return launch_status("swiglu_f32_kernel");
}

}  // namespace blok
