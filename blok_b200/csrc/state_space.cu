// What a selective state space (Mamba-2) feeds its recurrence with, and what follows it: the causal convolution per channel
// with SiLU, step sizes and decays, and the gate with a norm over parts.  The recurrence itself is linear_attn.cu.
//
// A sequence's last inputs of the convolution live in a ring of `taps` rows, position p at p % taps: a token reads taps - 1
// rows that it does not write, so a decode step reads and writes the ring in one launch.  A prompt reads the ring for its
// first tokens and writes it in the launch after that.
#include "common.cuh"
#include "stack_kernels.h"

namespace blok {

constexpr int kSiThreads = 256, kSiTokens = 8;  // tokens per thread of the convolution

template <typename Act>
struct Si8 {  // eight channels
  float v[8];
  __device__ __forceinline__ void load(const Act *p) {
    if constexpr (sizeof(Act) == 2) {
      const uint4 u = *reinterpret_cast<const uint4 *>(p);
      const uint32_t w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
      for (int j = 0; j < 4; ++j) v[2 * j] = bf16lo(w[j]), v[2 * j + 1] = bf16hi(w[j]);
    } else {
      const float4 a = *reinterpret_cast<const float4 *>(p), b = *reinterpret_cast<const float4 *>(p + 4);
      v[0] = a.x, v[1] = a.y, v[2] = a.z, v[3] = a.w, v[4] = b.x, v[5] = b.y, v[6] = b.z, v[7] = b.w;
    }
  }
  __device__ __forceinline__ void store(Act *p) const {
    if constexpr (sizeof(Act) == 2) {
      *reinterpret_cast<uint4 *>(p) = make_uint4(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]), pack_bf16x2(v[4], v[5]), pack_bf16x2(v[6], v[7]));
    } else {
      *reinterpret_cast<float4 *>(p) = make_float4(v[0], v[1], v[2], v[3]);
      *reinterpret_cast<float4 *>(p + 4) = make_float4(v[4], v[5], v[6], v[7]);
    }
  }
};
template <typename Act>
__device__ __forceinline__ void si_copy8(Act *dst, const Act *src) {
  *reinterpret_cast<uint4 *>(dst) = *reinterpret_cast<const uint4 *>(src);
  if constexpr (sizeof(Act) == 4) *reinterpret_cast<uint4 *>(dst + 4) = *reinterpret_cast<const uint4 *>(src + 4);
}

// Channels [c, c + 8) of tokens t0 .. t0 + n - 1.
template <typename Act>
__device__ __forceinline__ void si_conv(const StateInputs &a, const StackRows &r, int c, int t0, int n, bool chunk) {
  const Act *x = static_cast<const Act *>(a.proj) + a.first + c;
  Act *ring = static_cast<Act *>(a.ring) + c;
  Si8<Act> bias;
#pragma unroll
  for (int i = 0; i < 8; ++i) bias.v[i] = a.conv_b[c + i];
  Si8<Act> acc[kSiTokens];
#pragma unroll
  for (int q = 0; q < kSiTokens; ++q) acc[q] = bias;
  for (int j = a.taps - 1; j >= 0; --j) {  // the input j tokens back
    float w[8];
    const float4 w0 = *reinterpret_cast<const float4 *>(a.conv_w + (size_t)(a.taps - 1 - j) * a.channels + c),
                 w1 = *reinterpret_cast<const float4 *>(a.conv_w + (size_t)(a.taps - 1 - j) * a.channels + c + 4);
    w[0] = w0.x, w[1] = w0.y, w[2] = w0.z, w[3] = w0.w, w[4] = w1.x, w[5] = w1.y, w[6] = w1.z, w[7] = w1.w;
#pragma unroll
    for (int q = 0; q < kSiTokens; ++q) {
      const int t = t0 + q;
      if (q >= n) break;
      Si8<Act> in;
      if (j == 0 || (chunk && t >= j)) {
        in.load(x + (size_t)(t - j) * a.ld);
      } else {
        const int p = r.pos[t] - j;
        if (p < 0) continue;  // zeros before the start
        in.load(ring + ((size_t)r.slot_of[t] * a.taps + p % a.taps) * a.channels);
      }
#pragma unroll
      for (int i = 0; i < 8; ++i) acc[q].v[i] = fmaf(w[i], in.v[i], acc[q].v[i]);
    }
  }
#pragma unroll
  for (int q = 0; q < kSiTokens; ++q) {
    if (q >= n) break;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const float z = acc[q].v[i];
      acc[q].v[i] = sizeof(Act) == 2 ? __fdividef(z, 1.0f + __expf(-z)) : z / (1.0f + expf(-z));  // bf16: rounded right away
    }
    acc[q].store(static_cast<Act *>(a.out) + (size_t)(t0 + q) * a.channels + c);
  }
  if (!chunk)
    for (int q = 0; q < n; ++q)
      si_copy8(ring + ((size_t)r.slot_of[t0 + q] * a.taps + r.pos[t0 + q] % a.taps) * a.channels, x + (size_t)(t0 + q) * a.ld);
}

// 32 heads (one per lane), the 64 tokens of chunk `chunk_index` (eight per warp): step, log decay, running sum.
template <typename Act>
__device__ __forceinline__ void si_steps(const StateInputs &a, int head0, int chunk_index, int T) {
  __shared__ double s_sum[kSiThreads / 32][32];
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, h = head0 + lane, t0 = chunk_index * kLinChunk + warp * 8;
  const bool in = h < a.heads;
  float dt[8], lg[8];
  double sum = 0;
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    float z = 0.f;
    if (in && t0 + i < T) {
      const Act *p = static_cast<const Act *>(a.proj) + (size_t)(t0 + i) * a.ld + a.dt_at + h;
      if constexpr (sizeof(Act) == 2) z = bf16_bits_to_f32(*p);
      else z = *p;
      z += a.dt_bias[h];
      dt[i] = fmaxf(z, 0.f) + log1pf(expf(-fabsf(z)));
      lg[i] = a.rate[h] * dt[i];
    } else {
      dt[i] = lg[i] = 0.f;
    }
    sum += (double)lg[i];
  }
  s_sum[warp][lane] = sum;
  __syncthreads();
  sum = 0;
  for (int w = 0; w < warp; ++w) sum += s_sum[w][lane];
  if (!in) return;
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    sum += (double)lg[i];
    const float hi = (float)sum;
    if (t0 + i < T) a.token[(size_t)h * a.token_ld + t0 + i] = make_float4(dt[i], lg[i], hi, (float)(sum - (double)hi));
  }
}

// Blocks 0 .. conv_blocks - 1: convolution; then `ring_blocks` that write the ring; then the steps.
template <typename Act>
__global__ void __launch_bounds__(kSiThreads) state_inputs_kernel(const StateInputs a, const StackRows r, int T, int chunk, int per_thread,
                                                                  int conv_blocks, int ring_blocks) {
  const int per = a.channels / 8;
  int b = blockIdx.x;
  if (b < conv_blocks) {
    const long u = (long)b * kSiThreads + threadIdx.x;
    const int c = (int)(u % per) * 8, t0 = (int)(u / per) * per_thread;
    if (t0 < T) si_conv<Act>(a, r, c, t0, min(per_thread, T - t0), chunk != 0);
    return;
  }
  b -= conv_blocks;
  if (b < ring_blocks) {  // the last `taps` inputs of a prompt's portion
    const int n = min(T, a.taps);
    const long u = (long)b * kSiThreads + threadIdx.x;
    const int c = (int)(u % per) * 8, i = (int)(u / per);
    if (i < n) {
      const int t = T - n + i;
      si_copy8(static_cast<Act *>(a.ring) + ((size_t)r.slot_of[t] * a.taps + r.pos[t] % a.taps) * a.channels + c,
               static_cast<const Act *>(a.proj) + (size_t)t * a.ld + a.first + c);
    }
    return;
  }
  b -= ring_blocks;
  const int groups = (a.heads + 31) / 32;
  si_steps<Act>(a, b % groups * 32, b / groups, T);
}

template <typename Act>
static int state_inputs(const StateInputs &a, const StackRows &r, int T, bool chunk, cudaStream_t stream) {
  const long per = a.channels / 8;
  // several tokens per thread where that leaves enough threads: neighbours share most inputs
  const int per_thread = chunk && per * T >= (long)kSiTokens * sm_count() * kSiThreads ? kSiTokens : chunk && per * T >= 2l * sm_count() * kSiThreads ? 2 : 1;
  const auto blocks = [&](long units) { return (int)((units + kSiThreads - 1) / kSiThreads); };
  const int conv = blocks(per * ((T + per_thread - 1) / per_thread)), ring = blocks(per * (T < a.taps ? T : a.taps));
  const int steps = (a.heads + 31) / 32 * ((T + kLinChunk - 1) / kLinChunk);
  if (!chunk) {
    state_inputs_kernel<Act><<<conv + steps, kSiThreads, 0, stream>>>(a, r, T, 0, per_thread, conv, 0);
    return launch_status("state_inputs_kernel");
  }
  state_inputs_kernel<Act><<<conv, kSiThreads, 0, stream>>>(a, r, T, 1, per_thread, conv, 0);
  if (int rc = launch_status("state_inputs_kernel")) return rc;
  state_inputs_kernel<Act><<<ring + steps, kSiThreads, 0, stream>>>(a, r, T, 1, 1, 0, ring);
  return launch_status("state_inputs_kernel");
}

int launch_state_inputs(const StateInputs &a, const StackRows &r, int T, bool chunk, cudaStream_t stream) {
  BLOK_REQUIRE(a.heads >= 1 && a.channels % 16 == 0 && a.taps >= 1 && a.ld % 8 == 0 && a.first % 8 == 0 && T >= 1 && T <= a.token_ld, BLOK_ERR_SHAPE,
               "state space: %d heads, %d channels, %d taps", a.heads, a.channels, a.taps);
  return a.f32 ? state_inputs<float>(a, r, T, chunk, stream) : state_inputs<uint16_t>(a, r, T, chunk, stream);
}

// ---- gate, then a norm over equal parts of the true columns.  grid = (T, parts) ----
constexpr int kGnKeep = 8;

// VEC 4: no padding and parts in multiples of four; 1: any.
template <typename Act, int VEC>
__global__ void __launch_bounds__(256) gate_then_norm_kernel(const GatedNorm a, int part_len) {
  __shared__ float s_red[8];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, from = blockIdx.y * part_len, n = a.heads * a.vdim;
  const float *o = a.o + (size_t)blockIdx.x * n;
  const Act *g = static_cast<const Act *>(a.g) + (size_t)blockIdx.x * a.ldg;
  Act *out = static_cast<Act *>(a.out) + (size_t)blockIdx.x * a.ldo;
  auto column = [&](int i) { return VEC == 4 ? from + i : (from + i) / a.true_vdim * a.vdim + (from + i) % a.true_vdim; };
  auto gated = [&](int i, float *v) {
    const int c = column(i);
    float z[VEC];
    if constexpr (VEC == 4) {
      const float4 u = *reinterpret_cast<const float4 *>(o + c);
      v[0] = u.x, v[1] = u.y, v[2] = u.z, v[3] = u.w;
      if constexpr (sizeof(Act) == 2) {
        const uint2 w = *reinterpret_cast<const uint2 *>(g + c);
        z[0] = bf16lo(w.x), z[1] = bf16hi(w.x), z[2] = bf16lo(w.y), z[3] = bf16hi(w.y);
      } else {
        const float4 w = *reinterpret_cast<const float4 *>(g + c);
        z[0] = w.x, z[1] = w.y, z[2] = w.z, z[3] = w.w;
      }
    } else {
      v[0] = o[c];
      if constexpr (sizeof(Act) == 2) z[0] = bf16_bits_to_f32(g[c]);
      else z[0] = g[c];
    }
#pragma unroll
    for (int j = 0; j < VEC; ++j) v[j] *= z[j] / (1.0f + expf(-z[j]));
  };
  float keep[kGnKeep][VEC], s = 0.f;
  auto square = [&](const float *v) {
#pragma unroll
    for (int j = 0; j < VEC; ++j) s = fmaf(v[j], v[j], s);
  };
#pragma unroll
  for (int k = 0; k < kGnKeep; ++k) {
    const int i = (tid + 256 * k) * VEC;
    if (i < part_len) gated(i, keep[k]), square(keep[k]);
  }
  for (int i = (tid + 256 * kGnKeep) * VEC; i < part_len; i += 256 * VEC) {
    float v[VEC];
    gated(i, v), square(v);
  }
  s = warp_sum(s);
  if (lane == 0) s_red[warp] = s;
  __syncthreads();
  s = 0.f;
#pragma unroll
  for (int w = 0; w < 8; ++w) s += s_red[w];
  const float scale = 1.0f / sqrtf(s / (float)part_len + a.eps);
  auto write = [&](int i, const float *v) {
    const int c = column(i);
    float r[VEC];
#pragma unroll
    for (int j = 0; j < VEC; ++j) r[j] = v[j] * scale * (a.w ? a.w[c + j] : 1.f);
    if constexpr (VEC == 4) {
      if constexpr (sizeof(Act) == 2) *reinterpret_cast<uint2 *>(out + c) = make_uint2(pack_bf16x2(r[0], r[1]), pack_bf16x2(r[2], r[3]));
      else *reinterpret_cast<float4 *>(out + c) = make_float4(r[0], r[1], r[2], r[3]);
    } else {
      if constexpr (sizeof(Act) == 2) out[c] = f32_to_bf16_bits(r[0]);
      else out[c] = r[0];
    }
  };
#pragma unroll
  for (int k = 0; k < kGnKeep; ++k) {
    const int i = (tid + 256 * k) * VEC;
    if (i < part_len) write(i, keep[k]);
  }
  for (int i = (tid + 256 * kGnKeep) * VEC; i < part_len; i += 256 * VEC) {
    float v[VEC];
    gated(i, v);
    write(i, v);
  }
  if (blockIdx.y == 0) {  // the padding
    if (a.true_vdim < a.vdim) {
      const int pad = a.vdim - a.true_vdim;
      for (int i = tid; i < a.heads * pad; i += 256) out[i / pad * a.vdim + a.true_vdim + i % pad] = Act(0);
    }
    for (int i = n + tid; i < a.ldo; i += 256) out[i] = Act(0);
  }
}

int launch_gate_then_norm(const GatedNorm &a, int parts, int T, cudaStream_t stream) {
  BLOK_REQUIRE(parts >= 1 && a.heads * a.true_vdim % parts == 0, BLOK_ERR_SHAPE, "gated norm: %d parts of %d columns", parts, a.heads * a.true_vdim);
  const int len = a.heads * a.true_vdim / parts;
  const dim3 grid(T, parts);
  const bool wide = a.true_vdim == a.vdim && len % 4 == 0 && a.ldg % 4 == 0 && a.ldo % 4 == 0;
  if (a.f32 && wide) gate_then_norm_kernel<float, 4><<<grid, 256, 0, stream>>>(a, len);
  else if (a.f32) gate_then_norm_kernel<float, 1><<<grid, 256, 0, stream>>>(a, len);
  else if (wide) gate_then_norm_kernel<uint16_t, 4><<<grid, 256, 0, stream>>>(a, len);
  else gate_then_norm_kernel<uint16_t, 1><<<grid, 256, 0, stream>>>(a, len);
  return launch_status("gate_then_norm_kernel");
}

}  // namespace blok
