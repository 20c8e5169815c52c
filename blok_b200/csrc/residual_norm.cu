// One residual between sandwiched sublayers, in one pass over a token's row: the sublayer's output is normed, scaled and
// added to the residual, the new residual is normed again into the next sublayer's input.  Both are layer norms without a
// bias (mean, then the mean of the squared deviations, from registers).  The first pass of a step makes the residual from the
// embeddings instead.  All of it is fp32; h alone is rounded.  One CTA per token.
#include "common.cuh"
#include "stack_kernels.h"

namespace blok {

// The CTA's sum; s_red has one word per warp and serves one call.
template <int WARPS>
__device__ __forceinline__ float rn_sum(float v, float *s_red) {
  v = warp_sum(v);
  if ((threadIdx.x & 31) == 0) s_red[threadIdx.x >> 5] = v;
  __syncthreads();
  v = s_red[0];
#pragma unroll
  for (int w = 1; w < WARPS; ++w) v += s_red[w];
  return v;
}

// v <- (v - mean) / sqrt(variance + eps) over the row's true columns (the thread's are 4 (tid + THREADS k) + j); columns of
// the padding become 0.
template <int THREADS, int KEEP>
__device__ __forceinline__ void rn_layer_norm(float4 (&v)[KEEP], int width, float eps, float (*s_red)[THREADS / 32]) {
  auto each = [&](auto f) {
#pragma unroll
    for (int k = 0; k < KEEP; ++k) {
      const int c = 4 * ((int)threadIdx.x + THREADS * k);
      f(c < width, v[k].x), f(c + 1 < width, v[k].y), f(c + 2 < width, v[k].z), f(c + 3 < width, v[k].w);
    }
  };
  float s = 0.f;
  each([&](bool in, float &x) { s += in ? x : 0.f; });
  const float mean = rn_sum<THREADS / 32>(s, s_red[0]) / (float)width;
  s = 0.f;
  each([&](bool in, float &x) {
    x = in ? x - mean : 0.f;
    s = fmaf(x, x, s);
  });
  const float r = 1.0f / sqrtf(rn_sum<THREADS / 32>(s, s_red[1]) / (float)width + eps);
  each([&](bool, float &x) { x *= r; });
}

__device__ __forceinline__ float4 rn_bf16x4(const uint16_t *p) {
  const uint2 v = *reinterpret_cast<const uint2 *>(p);
  return make_float4(bf16lo(v.x), bf16hi(v.x), bf16lo(v.y), bf16hi(v.y));
}

template <int THREADS, int KEEP>
__global__ void __launch_bounds__(THREADS) residual_norm_kernel(const ResidualNorm a) {
  __shared__ float s_red[4][THREADS / 32];
  const int t = blockIdx.x, tid = threadIdx.x;
  float *xr = a.x + (size_t)t * a.width;
  float4 x[KEEP], w[KEEP];
  if (a.norm_w) {  // on their way before the reductions
#pragma unroll
    for (int k = 0; k < KEEP; ++k) {
      const int c = 4 * (tid + THREADS * k);
      if (c < a.width) w[k] = *reinterpret_cast<const float4 *>(a.norm_w + c);
    }
  }
  if (a.ids) {
    const uint32_t last = (uint32_t)a.vocab - 1, id = min(a.ids[t], last);
    const int pos = a.pos ? a.pos[t] : 0;
    const uint16_t *pair = nullptr;
    if (a.bigram) {
      size_t row = (size_t)a.buckets;
      if (pos > 0) {
        const uint32_t prev = min(a.chunk && t > 0 ? a.ids[t - 1] : a.last_ids[a.slot_of[t]], last);
        row = (size_t)(((uint64_t)prev * (uint64_t)a.mul_prev + (uint64_t)id * (uint64_t)a.mul_cur) % (uint64_t)a.buckets);
      }
      pair = a.bigram + row * a.width;
    }
#pragma unroll
    for (int k = 0; k < KEEP; ++k) {
      const int c = 4 * (tid + THREADS * k);
      if (c >= a.width) continue;
      float4 v = rn_bf16x4(a.embed + (size_t)id * a.width + c);
      v = make_float4(v.x * a.embed_scale, v.y * a.embed_scale, v.z * a.embed_scale, v.w * a.embed_scale);
      if (pair) {
        const float4 p = rn_bf16x4(pair + c);
        v = make_float4(v.x + p.x, v.y + p.y, v.z + p.z, v.w + p.w);
      }
      if (a.turns) {
        // a pair's sine and cosine, the angle reduced to one turn in double
        float p[4];
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          const double full = (double)pos * a.turns[c / 2 + i];
          sincospif((float)(2.0 * (full - floor(full))), &p[2 * i], &p[2 * i + 1]);
        }
        const float keep[4] = {c < a.true_width ? p[0] : 0.f, c + 1 < a.true_width ? p[1] : 0.f, c + 2 < a.true_width ? p[2] : 0.f,
                               c + 3 < a.true_width ? p[3] : 0.f};
        v = make_float4(v.x + keep[0], v.y + keep[1], v.z + keep[2], v.w + keep[3]);
      }
      x[k] = v;
      *reinterpret_cast<float4 *>(xr + c) = v;
    }
  } else {
#pragma unroll
    for (int k = 0; k < KEEP; ++k) {
      const int c = 4 * (tid + THREADS * k);
      if (c < a.width) x[k] = *reinterpret_cast<const float4 *>(xr + c);
    }
    if (a.y) {
      float4 y[KEEP], p[KEEP];
#pragma unroll
      for (int k = 0; k < KEEP; ++k) {
        const int c = 4 * (tid + THREADS * k);
        y[k] = c < a.width ? *reinterpret_cast<const float4 *>(a.y + (size_t)t * a.width + c) : make_float4(0.f, 0.f, 0.f, 0.f);
        p[k] = a.post_w && c < a.width ? *reinterpret_cast<const float4 *>(a.post_w + c) : make_float4(1.f, 1.f, 1.f, 1.f);
      }
      if (a.post_w) rn_layer_norm<THREADS, KEEP>(y, a.true_width, a.eps, s_red);
#pragma unroll
      for (int k = 0; k < KEEP; ++k) {
        const int c = 4 * (tid + THREADS * k);
        if (c >= a.width) continue;
        x[k] = make_float4(fmaf(a.mult, y[k].x * p[k].x, x[k].x), fmaf(a.mult, y[k].y * p[k].y, x[k].y), fmaf(a.mult, y[k].z * p[k].z, x[k].z),
                           fmaf(a.mult, y[k].w * p[k].w, x[k].w));
        *reinterpret_cast<float4 *>(xr + c) = x[k];
      }
    }
  }
  if (a.copy) {
#pragma unroll
    for (int k = 0; k < KEEP; ++k) {
      const int c = 4 * (tid + THREADS * k);
      const float v[4] = {x[k].x, x[k].y, x[k].z, x[k].w};
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (c + j < a.true_width) a.copy[(size_t)t * a.true_width + c + j] = v[j];
    }
  }
  if (a.norm_w) {
    rn_layer_norm<THREADS, KEEP>(x, a.true_width, a.eps, s_red + 2);
#pragma unroll
    for (int k = 0; k < KEEP; ++k) {
      const int c = 4 * (tid + THREADS * k);
      if (c >= a.width) continue;
      const float4 h = make_float4(x[k].x * w[k].x, x[k].y * w[k].y, x[k].z * w[k].z, x[k].w * w[k].w);
      const size_t at = (size_t)t * a.width + c;
      if (a.h_f32) *reinterpret_cast<float4 *>(static_cast<float *>(a.h) + at) = h;
      else *reinterpret_cast<uint2 *>(static_cast<uint16_t *>(a.h) + at) = make_uint2(pack_bf16x2(h.x, h.y), pack_bf16x2(h.z, h.w));
    }
  }
  // a sequence's newest token, kept for the pair at its next call
  if (a.keep_ids && tid == 0 && (!a.chunk || t == a.T - 1)) a.last_ids[a.slot_of[t]] = a.keep_ids[t];
}

int launch_residual_norm(const ResidualNorm &a, cudaStream_t stream) {
  BLOK_REQUIRE(a.T >= 1 && a.width % 4 == 0 && a.true_width >= 1 && a.true_width <= a.width && a.width <= kMaxNormWidth, BLOK_ERR_SHAPE,
               "residual norm: T %d, width %d (at most %d)", a.T, a.width, kMaxNormWidth);
  if (a.width <= 512) residual_norm_kernel<128, 1><<<a.T, 128, 0, stream>>>(a);
  else if (a.width <= 1024) residual_norm_kernel<256, 1><<<a.T, 256, 0, stream>>>(a);
  else if (a.width <= 2048) residual_norm_kernel<256, 2><<<a.T, 256, 0, stream>>>(a);
  else if (a.width <= 4096) residual_norm_kernel<512, 2><<<a.T, 512, 0, stream>>>(a);
  else if (a.width <= 8192) residual_norm_kernel<512, 4><<<a.T, 512, 0, stream>>>(a);
  else residual_norm_kernel<1024, 8><<<a.T, 1024, 0, stream>>>(a);
  return launch_status("residual_norm_kernel");
}

}  // namespace blok
