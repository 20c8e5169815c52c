// What a selective state space (Mamba-2) feeds its recurrence with, and what follows it: the causal convolution per channel
// with SiLU, step sizes and decays, and the gate with a norm over parts.  The recurrence itself is linear_attn.cu.
//
// A sequence's last inputs of the convolution live in a ring of `taps` rows, position p at p % taps.  Every channel of a ring is
// read and written by one thread: the one that has the sequence's first tokens of the call, taps - 1 of them at least.
#include "common.cuh"
#include "stack_kernels.h"

namespace blok {

constexpr int kSiThreads = 256, kSiTokens = 4;  // tokens per thread of a long prompt's convolution

// Eight channels of a row, as they are stored.
template <typename Act>
struct Si8 {
  static constexpr int kWords = sizeof(Act) * 2;
  uint32_t w[kWords];
  __device__ __forceinline__ void clear() {
#pragma unroll
    for (int i = 0; i < kWords; ++i) w[i] = 0;
  }
  __device__ __forceinline__ void load(const Act *p) {
#pragma unroll
    for (int i = 0; i < kWords; i += 4) {
      const uint4 u = *reinterpret_cast<const uint4 *>(reinterpret_cast<const uint32_t *>(p) + i);
      w[i] = u.x, w[i + 1] = u.y, w[i + 2] = u.z, w[i + 3] = u.w;
    }
  }
  __device__ __forceinline__ float value(int i) const {
    if constexpr (sizeof(Act) == 2) return i & 1 ? bf16hi(w[i / 2]) : bf16lo(w[i / 2]);
    else return __uint_as_float(w[i]);
  }
};
template <typename Act>
__device__ __forceinline__ void si_copy8(Act *dst, const Act *src) {
  *reinterpret_cast<uint4 *>(dst) = *reinterpret_cast<const uint4 *>(src);
  if constexpr (sizeof(Act) == 4) *reinterpret_cast<uint4 *>(dst + 4) = *reinterpret_cast<const uint4 *>(src + 4);
}

// Channels [c, c + 8) of tokens t0 .. t0 + n - 1, n <= TOKENS.  TAPS: a.taps if it is known (every load is on its way before the
// first use then), or 0.
template <typename Act, int TAPS, int TOKENS>
__device__ __forceinline__ void si_conv(const StateInputs &a, const StackRows &r, int c, int t0, int n, bool chunk) {
  const Act *x = static_cast<const Act *>(a.proj) + a.first + c;
  const Act *ring = static_cast<const Act *>(a.ring) + c;
  // the input of token t0 + q, q possibly negative: of this call, of the ring (a step's tokens have rings of their own), or zeros
  auto input = [&](int t, int back, Si8<Act> *in) {
    if (back == 0 || (chunk && t >= back)) {
      in->load(x + (size_t)(t - back) * a.ld);
      return;
    }
    const int p = r.pos[t] - back;
    if (p >= 0) in->load(ring + ((size_t)r.slot_of[t] * a.taps + p % a.taps) * a.channels);
    else in->clear();
  };
  Si8<float> bias;
  bias.load(a.conv_b + c);
  float acc[TOKENS][8];
#pragma unroll
  for (int q = 0; q < TOKENS; ++q)
#pragma unroll
    for (int i = 0; i < 8; ++i) acc[q][i] = bias.value(i);
  auto add = [&](const Si8<float> &w, const Si8<Act> &in, float (&to)[8]) {
#pragma unroll
    for (int i = 0; i < 8; ++i) to[i] = fmaf(w.value(i), in.value(i), to[i]);
  };
  if constexpr (TAPS > 0) {
    Si8<float> w[TAPS];
    Si8<Act> in[TOKENS + TAPS - 1];
#pragma unroll
    for (int j = 0; j < TAPS; ++j) w[j].load(a.conv_w + (size_t)j * a.channels + c);
#pragma unroll
    for (int k = 0; k < TOKENS + TAPS - 1; ++k) {
      const int q = k - (TAPS - 1);  // token t0 + q, seen from token t0 if it lies in front of it
      if (q < n) input(q < 0 ? t0 : t0 + q, q < 0 ? -q : 0, &in[k]);
    }
#pragma unroll
    for (int q = 0; q < TOKENS; ++q)
#pragma unroll
      for (int j = 0; j < TAPS; ++j)
        if (q < n) add(w[j], in[q + j], acc[q]);
  } else {
    for (int j = 0; j < a.taps; ++j) {
      Si8<float> w;
      w.load(a.conv_w + (size_t)j * a.channels + c);
#pragma unroll
      for (int q = 0; q < TOKENS; ++q) {
        if (q >= n) break;
        Si8<Act> in;
        input(t0 + q, a.taps - 1 - j, &in);
        add(w, in, acc[q]);
      }
    }
  }
#pragma unroll
  for (int q = 0; q < TOKENS; ++q) {
    if (q >= n) break;
    float v[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const float z = acc[q][i];
      v[i] = sizeof(Act) == 2 ? __fdividef(z, 1.0f + __expf(-z)) : z / (1.0f + expf(-z));  // bf16: rounded right away
    }
    Act *out = static_cast<Act *>(a.out) + (size_t)(t0 + q) * a.channels + c;
    if constexpr (sizeof(Act) == 2) {
      *reinterpret_cast<uint4 *>(out) = make_uint4(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]), pack_bf16x2(v[4], v[5]), pack_bf16x2(v[6], v[7]));
    } else {
      *reinterpret_cast<float4 *>(out) = make_float4(v[0], v[1], v[2], v[3]);
      *reinterpret_cast<float4 *>(out + 4) = make_float4(v[4], v[5], v[6], v[7]);
    }
  }
}

// The newest inputs of a call go into the ring: rows t0 .. t0 + n - 1.
template <typename Act>
__device__ __forceinline__ void si_keep(const StateInputs &a, const StackRows &r, int c, int t0, int n) {
  for (int t = t0; t < t0 + n; ++t)
    si_copy8(static_cast<Act *>(a.ring) + ((size_t)r.slot_of[t] * a.taps + r.pos[t] % a.taps) * a.channels + c,
             static_cast<const Act *>(a.proj) + (size_t)t * a.ld + a.first + c);
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

// The steps in the first `step_blocks` blocks, then the convolution: unit 0 of a chunk has its first `lead` tokens.
template <typename Act, int TAPS, int TOKENS>
__global__ void __launch_bounds__(kSiThreads, sizeof(Act) == 2 ? 2 : 1) state_inputs_kernel(const StateInputs a, const StackRows r, int T, int chunk, int lead, int step_blocks) {
  const int b = (int)blockIdx.x - step_blocks;
  if (b < 0) {
    const int groups = (a.heads + 31) / 32;
    si_steps<Act>(a, (int)blockIdx.x % groups * 32, (int)blockIdx.x / groups, T);
    return;
  }
  const int per = a.channels / 8, u = b * kSiThreads + (int)threadIdx.x, i = u / per, c = (u - i * per) * 8;
  if (!chunk) {
    if (i >= T) return;
    si_conv<Act, TAPS, 1>(a, r, c, i, 1, false);
    si_keep<Act>(a, r, c, i, 1);
    return;
  }
  int t0 = i == 0 ? 0 : lead + (i - 1) * TOKENS;
  const int end = min(T, i == 0 ? lead : t0 + TOKENS);
  for (; t0 < end; t0 += TOKENS) si_conv<Act, TAPS, TOKENS>(a, r, c, t0, min(TOKENS, end - t0), true);
  if (i == 0) {
    const int n = min(T, a.taps);
    si_keep<Act>(a, r, c, T - n, n);
  }
}

template <typename Act, int TAPS, int TOKENS>
static int state_inputs(const StateInputs &a, const StackRows &r, int T, bool chunk, cudaStream_t stream) {
  const int lead = chunk && a.taps > 1 ? a.taps - 1 : 1;
  const long units = chunk ? 1 + (T > lead ? (T - lead + TOKENS - 1) / TOKENS : 0) : T, threads = a.channels / 8 * units;
  const int steps = (a.heads + 31) / 32 * ((T + kLinChunk - 1) / kLinChunk);
  BLOK_REQUIRE(threads < (1l << 30), BLOK_ERR_SHAPE, "state space: %d channels of %d tokens", a.channels, T);
  state_inputs_kernel<Act, TAPS, TOKENS><<<steps + (int)((threads + kSiThreads - 1) / kSiThreads), kSiThreads, 0, stream>>>(a, r, T, chunk, lead, steps);
  return launch_status("state_inputs_kernel");
}
template <typename Act>
static int state_inputs_of(const StateInputs &a, const StackRows &r, int T, bool chunk, cudaStream_t stream) {
  // several tokens per thread where that leaves enough threads: neighbours share most inputs
  const bool many = (long)a.channels / 8 * T / kSiTokens >= 512l * sm_count();
  if (a.taps != 4) return many ? state_inputs<Act, 0, kSiTokens>(a, r, T, chunk, stream) : state_inputs<Act, 0, 1>(a, r, T, chunk, stream);
  return many ? state_inputs<Act, 4, kSiTokens>(a, r, T, chunk, stream) : state_inputs<Act, 4, 1>(a, r, T, chunk, stream);
}

int launch_state_inputs(const StateInputs &a, const StackRows &r, int T, bool chunk, cudaStream_t stream) {
  BLOK_REQUIRE(a.heads >= 1 && a.channels % 16 == 0 && a.taps >= 1 && a.ld % 8 == 0 && a.first % 8 == 0 && T >= 1 && T <= a.token_ld, BLOK_ERR_SHAPE,
               "state space: %d heads, %d channels, %d taps", a.heads, a.channels, a.taps);
  return a.f32 ? state_inputs_of<float>(a, r, T, chunk, stream) : state_inputs_of<uint16_t>(a, r, T, chunk, stream);
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
