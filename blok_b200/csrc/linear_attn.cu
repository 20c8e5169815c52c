// Linear attention without a softmax:
//   S_t = decay_t S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t                   (S fp32 [dim, vdim], per head and sequence)
// with a fixed decay per head (retention, lightning attention), or with a decay and a key scale per head and token and a
// skip o_t += D v_t (a selective state space: q = C, k = dt B, v = x, shared by several heads; state_space.cu makes them).
//
// Decode runs the recurrence itself, every thread holding a few elements of S in registers.  A prompt runs in chunks of 64
// tokens: with w_ij = decay^(i-j) for j <= i inside a chunk and S the state in front of it,
//   o_i = sum_j w_ij (q_i . k_j) v_j + decay^(i+1) S^T q_i
//   S'  = decay^L S + sum_j decay^(L-1-j) k_j v_j^T                        (L tokens in the chunk)
// in three launches: every chunk's own contribution to the state in parallel, a scan over the chunks that turns the
// contributions into the states in front of them, every chunk's output in parallel.  With decays per token every power becomes
// the exponential of a difference of the logarithms' running sums, which are kept in two fp32 parts.  The products run on bf16 tensor cores
// with their fp32 factors (scores, decays, states) split into three bf16 parts (bf16_split.cuh).
#include "bf16_split.cuh"
#include "stack_kernels.h"

namespace blok {

template <typename Act>
__device__ __forceinline__ float la_load(const Act *p) {
  if constexpr (sizeof(Act) == 2) return bf16_bits_to_f32(*p);
  else return *p;
}
__device__ __forceinline__ float la_silu(float z) { return z / (1.0f + expf(-z)); }
// A projection after its activation, rounded as the activation's type is.
template <typename Act>
__device__ __forceinline__ float la_proj(const Act *p, bool silu) {
  const float v = la_load(p);
  if (!silu) return v;
  return sizeof(Act) == 2 ? round_bf16(la_silu(v)) : la_silu(v);
}

struct LaArgs {
  const void *q, *k, *v;  // a token's rows: heads / share heads of q and k, heads of v; `ld` values between tokens
  int share;
  const float *decay_pow;
  const float4 *token;    // decays per token: [heads, token_ld] of (key scale, log decay, running sum of the log decays in two parts)
  int token_ld;
  const float *skip;      // with token: [heads]
  float *state, *o, *chunk_state;
  const int *slot_of, *pos;  // step form
  int slot;                  // chunk form
  int fresh;                 // chunk form: the sequence starts here
  int heads, dim, vdim, ld, silu, T, chunks;
  float k_scale;
};

// ---- the recurrence: T tokens of each of gridDim.z sequences, one after the other.  CTA = 32 columns of a head's state,
// thread = 4 columns x every 32nd row. ----
template <typename Act, int R, bool TOKEN>
__global__ void __launch_bounds__(256) linear_recurrent_kernel(const LaArgs a) {
  __shared__ float sq[32 * R], sk[32 * R];
  __shared__ float4 s_red[8][8];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, c4 = tid & 7, rg = tid >> 3;
  const int h = blockIdx.y, b = blockIdx.z, col = blockIdx.x * 32 + c4 * 4;
  const bool in_col = col < a.vdim;
  const int slot = a.slot_of ? a.slot_of[b] : a.slot;
  const bool fresh = a.slot_of ? a.pos[b] == 0 : a.fresh != 0;
  float decay = TOKEN ? 0.f : a.decay_pow[h * (kLinChunk + 1) + 1], k_scale = a.k_scale;
  const float skip = TOKEN ? a.skip[h] : 0.f;
  float *st = a.state + ((size_t)slot * a.heads + h) * a.dim * a.vdim + col;
  float4 s[R];
#pragma unroll
  for (int r = 0; r < R; ++r) {
    const int i = rg + 32 * r;
    s[r] = !fresh && in_col && i < a.dim ? *reinterpret_cast<const float4 *>(st + (size_t)i * a.vdim) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  for (int t = 0; t < a.T; ++t) {
    const size_t row = (size_t)b * a.T + t;
    const size_t qk = row * a.ld + (size_t)(h / a.share) * a.dim + tid;
    if (TOKEN) {
      const float4 w = a.token[(size_t)h * a.token_ld + row];
      k_scale = w.x;
      decay = expf(w.y);
    }
    if (tid < 32 * R) {
      const bool in = tid < a.dim;
      sq[tid] = in ? la_proj(static_cast<const Act *>(a.q) + qk, a.silu) : 0.f;
      sk[tid] = in ? la_proj(static_cast<const Act *>(a.k) + qk, a.silu) * k_scale : 0.f;
    }
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (in_col) {
      const Act *pv = static_cast<const Act *>(a.v) + row * a.ld + (size_t)h * a.vdim + col;
      v = make_float4(la_proj(pv, a.silu), la_proj(pv + 1, a.silu), la_proj(pv + 2, a.silu), la_proj(pv + 3, a.silu));
    }
    __syncthreads();
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int r = 0; r < R; ++r) {
      const float k = sk[rg + 32 * r], q = sq[rg + 32 * r];
      s[r] = make_float4(fmaf(decay, s[r].x, k * v.x), fmaf(decay, s[r].y, k * v.y), fmaf(decay, s[r].z, k * v.z), fmaf(decay, s[r].w, k * v.w));
      o = make_float4(fmaf(q, s[r].x, o.x), fmaf(q, s[r].y, o.y), fmaf(q, s[r].z, o.z), fmaf(q, s[r].w, o.w));
    }
#pragma unroll
    for (int d = 8; d < 32; d <<= 1) {
      o.x += __shfl_xor_sync(0xffffffffu, o.x, d);
      o.y += __shfl_xor_sync(0xffffffffu, o.y, d);
      o.z += __shfl_xor_sync(0xffffffffu, o.z, d);
      o.w += __shfl_xor_sync(0xffffffffu, o.w, d);
    }
    if (lane < 8) s_red[warp][lane] = o;
    __syncthreads();
    if (tid < 8 && in_col) {
      float4 u = s_red[0][tid];
#pragma unroll
      for (int w = 1; w < 8; ++w) u = make_float4(u.x + s_red[w][tid].x, u.y + s_red[w][tid].y, u.z + s_red[w][tid].z, u.w + s_red[w][tid].w);
      if (TOKEN) u = make_float4(fmaf(skip, v.x, u.x), fmaf(skip, v.y, u.y), fmaf(skip, v.z, u.z), fmaf(skip, v.w, u.w));
      *reinterpret_cast<float4 *>(a.o + row * a.heads * a.vdim + (size_t)h * a.vdim + col) = u;
    }
  }
  if (in_col) {
#pragma unroll
    for (int r = 0; r < R; ++r)
      if (rg + 32 * r < a.dim) *reinterpret_cast<float4 *>(st + (size_t)(rg + 32 * r) * a.vdim) = s[r];
  }
}

// ---- chunked form ----
constexpr int kLcThreads = 256;
constexpr int kLcAhead = 4;  // loads in flight per thread while a tile is staged
constexpr int kLcCols = 64;  // columns of v per CTA
constexpr int kLcVPitch = kLcCols * 2 + 16;

__device__ __forceinline__ void lc_wait() {
  asm volatile("cp.async.wait_all;" ::: "memory");
  __syncthreads();
}
__device__ __forceinline__ uint4 lc_silu8(uint4 v) {
  uint32_t w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
  for (int j = 0; j < 4; ++j) w[j] = pack_bf16x2(la_silu(bf16lo(w[j])), la_silu(bf16hi(w[j])));
  return make_uint4(w[0], w[1], w[2], w[3]);
}

// `n` rows of `cols` bf16 (a multiple of 8) from p (row pitch ld elements) into a tile; rows past n are zero.  Without SiLU the
// copies are asynchronous: the caller waits for them.
__device__ __forceinline__ void lc_stage(unsigned char *dst, int pitch, const uint16_t *p, int ld, int n, int cols, bool silu) {
  const int per = cols / 8, total = kLinChunk * per;
  if (!silu) {
    const uint32_t d = (uint32_t)__cvta_generic_to_shared(dst);
    for (int u = threadIdx.x; u < total; u += kLcThreads) {
      const int r = u / per, c = u - r * per;
      asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(d + (uint32_t)(r * pitch + c * 16)), "l"(r < n ? p + (size_t)r * ld + c * 8 : p),
                   "r"(r < n ? 16u : 0u)
                   : "memory");
    }
    return;
  }
  for (int u0 = threadIdx.x; u0 < total; u0 += kLcAhead * kLcThreads) {
    uint4 v[kLcAhead];
#pragma unroll
    for (int q = 0; q < kLcAhead; ++q) {
      const int u = u0 + q * kLcThreads, r = u / per, c = u - r * per;
      v[q] = u < total && r < n ? *reinterpret_cast<const uint4 *>(p + (size_t)r * ld + c * 8) : make_uint4(0, 0, 0, 0);
    }
#pragma unroll
    for (int q = 0; q < kLcAhead; ++q) {
      const int u = u0 + q * kLcThreads, r = u / per, c = u - r * per;
      if (u < total) *reinterpret_cast<uint4 *>(dst + (size_t)r * pitch + c * 16) = silu ? lc_silu8(v[q]) : v[q];
    }
  }
}

// exp(a - b) of running sums in two parts
__device__ __forceinline__ float lc_between(float4 a, float4 b) { return expf((a.z - b.z) + (a.w - b.w)); }

// chunk_state[c][h] = sum_j k_scale decay^(L-1-j) k_j v_j^T.  grid = (chunks, heads, columns / 64)
template <bool TOKEN>
__global__ void __launch_bounds__(kLcThreads) linear_chunk_state_kernel(const LaArgs a) {
  extern __shared__ __align__(16) unsigned char smem[];
  __shared__ float s_wt[kLinChunk];
  const int c = blockIdx.x, h = blockIdx.y, v0 = blockIdx.z * kLcCols;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int n = min(kLinChunk, a.T - c * kLinChunk), vc = min(kLcCols, a.vdim - v0);
  const int kp = a.dim * 2 + 16;  // pitch of the key tiles
  unsigned char *Vs = smem + (size_t)kSplitParts * kLinChunk * kp;
  const size_t rows = (size_t)c * kLinChunk * a.ld;
  const uint16_t *k = static_cast<const uint16_t *>(a.k) + rows + (size_t)(h / a.share) * a.dim;
  lc_stage(Vs, kLcVPitch, static_cast<const uint16_t *>(a.v) + rows + (size_t)h * a.vdim + v0, a.ld, n, vc, a.silu);
  if (threadIdx.x < kLinChunk) {
    const int r = threadIdx.x;
    float wt = 0.f;
    if (r < n) {
      if (TOKEN) {
        const float4 *tok = a.token + (size_t)h * a.token_ld + c * kLinChunk;
        wt = tok[r].x * lc_between(tok[n - 1], tok[r]);
      } else {
        wt = a.k_scale * a.decay_pow[h * (kLinChunk + 1) + n - 1 - r];
      }
    }
    s_wt[r] = wt;
  }
  __syncthreads();
  const int per = a.dim / 8, total = kLinChunk * per;
  for (int u0 = threadIdx.x; u0 < total; u0 += kLcAhead * kLcThreads) {  // the decayed keys in three parts
    uint4 x[kLcAhead];
#pragma unroll
    for (int q = 0; q < kLcAhead; ++q) {
      const int u = u0 + q * kLcThreads, r = u / per;
      x[q] = u < total && r < n ? *reinterpret_cast<const uint4 *>(k + (size_t)r * a.ld + (u - r * per) * 8) : make_uint4(0, 0, 0, 0);
    }
#pragma unroll
    for (int q = 0; q < kLcAhead; ++q) {
      const int u = u0 + q * kLcThreads, r = u / per, col = (u - r * per) * 8;
      if (u >= total) break;
      if (a.silu) x[q] = lc_silu8(x[q]);
      const float wt = s_wt[r];
      const uint32_t w[4] = {x[q].x, x[q].y, x[q].z, x[q].w};
      uint32_t part[4][kSplitParts];
#pragma unroll
      for (int j = 0; j < 4; ++j) split_pair(bf16lo(w[j]) * wt, bf16hi(w[j]) * wt, part[j]);
#pragma unroll
      for (int p = 0; p < kSplitParts; ++p)
        *reinterpret_cast<uint4 *>(smem + (size_t)(p * kLinChunk + r) * kp + col * 2) = make_uint4(part[0][p], part[1][p], part[2][p], part[3][p]);
    }
  }
  lc_wait();
  const uint32_t ks = (uint32_t)__cvta_generic_to_shared(smem), vs = (uint32_t)__cvta_generic_to_shared(Vs);
  float *out = a.chunk_state + (((size_t)c * a.heads + h) * a.dim) * a.vdim + v0;
  const int g = lane >> 2, t = lane & 3;
  for (int m0 = warp * 16; m0 < a.dim; m0 += 16 * (kLcThreads / 32)) {
    float acc[kLcCols / 8][4] = {};
#pragma unroll
    for (int k0 = 0; k0 < kLinChunk; k0 += 16) {
      uint32_t fa[kSplitParts][4];
#pragma unroll
      for (int p = 0; p < kSplitParts; ++p) ldsm4_t(frag_a_t(ks + p * kLinChunk * kp, m0, k0, kp, lane), fa[p][0], fa[p][1], fa[p][2], fa[p][3]);
#pragma unroll
      for (int nt = 0; nt < kLcCols / 8; nt += 2) {
        if (nt * 8 < vc) {
          uint32_t b0, b1, b2, b3;
          ldsm4_t(frag_b_t(vs, nt * 8, k0, kLcVPitch, lane), b0, b1, b2, b3);
#pragma unroll
          for (int p = 0; p < kSplitParts; ++p) {
            mma_bf16_16816(acc[nt], fa[p][0], fa[p][1], fa[p][2], fa[p][3], b0, b1);
            mma_bf16_16816(acc[nt + 1], fa[p][0], fa[p][1], fa[p][2], fa[p][3], b2, b3);
          }
        }
      }
    }
#pragma unroll
    for (int nt = 0; nt < kLcCols / 8; ++nt) {
      const int col = nt * 8 + 2 * t;
      if (nt * 8 < vc) {
        *reinterpret_cast<float2 *>(out + (size_t)(m0 + g) * a.vdim + col) = make_float2(acc[nt][0], acc[nt][1]);
        *reinterpret_cast<float2 *>(out + (size_t)(m0 + g + 8) * a.vdim + col) = make_float2(acc[nt][2], acc[nt][3]);
      }
    }
  }
}

// chunk_state[c] <- the state in front of chunk c; state <- the state behind the last chunk.
template <bool TOKEN>
__global__ void __launch_bounds__(128) linear_scan_kernel(const LaArgs a) {
  const int h = blockIdx.y, i = (blockIdx.x * blockDim.x + threadIdx.x) * 4, n = a.dim * a.vdim;
  if (i >= n) return;
  float4 *st = reinterpret_cast<float4 *>(a.state + ((size_t)a.slot * a.heads + h) * n + i);
  float4 s = a.fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : *st;
  constexpr int kAhead = 8;  // chunks' loads in flight
  const size_t stride = (size_t)a.heads * n / 4;
  float4 *p = reinterpret_cast<float4 *>(a.chunk_state + (size_t)h * n + i);
  for (int c0 = 0; c0 < a.chunks; c0 += kAhead) {
    float4 own[kAhead];
    float decay[kAhead];
#pragma unroll
    for (int j = 0; j < kAhead; ++j)
      if (c0 + j < a.chunks) {
        const int n = min(kLinChunk, a.T - (c0 + j) * kLinChunk);
        if (TOKEN) {
          const float4 w = a.token[(size_t)h * a.token_ld + (c0 + j) * kLinChunk + n - 1];
          decay[j] = w.z + w.w;
        } else {
          decay[j] = a.decay_pow[h * (kLinChunk + 1) + n];
        }
        own[j] = p[(size_t)(c0 + j) * stride];
      }
#pragma unroll
    for (int j = 0; j < kAhead; ++j)
      if (c0 + j < a.chunks) {
        const float d = TOKEN ? expf(decay[j]) : decay[j];
        p[(size_t)(c0 + j) * stride] = s;
        s = make_float4(fmaf(d, s.x, own[j].x), fmaf(d, s.y, own[j].y), fmaf(d, s.z, own[j].z), fmaf(d, s.w, own[j].w));
      }
  }
  *st = s;
}

// grid = (chunks, heads, columns / 64); a warp owns 16 tokens of the chunk and half of the columns.
template <bool TOKEN>
__global__ void __launch_bounds__(kLcThreads, 2) linear_chunk_out_kernel(const LaArgs a) {
  extern __shared__ __align__(16) unsigned char smem[];
  __shared__ float s_pw[TOKEN ? 1 : kLinChunk + 1];
  __shared__ float4 s_tok[TOKEN ? kLinChunk : 1];
  const int c = blockIdx.x, h = blockIdx.y, v0 = blockIdx.z * kLcCols;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, t = lane & 3;
  const int n = min(kLinChunk, a.T - c * kLinChunk), vc = min(kLcCols, a.vdim - v0);
  const int kp = a.dim * 2 + 16;
  unsigned char *Ks = smem + (size_t)kLinChunk * kp, *Vs = Ks + (size_t)kLinChunk * kp, *Ss = Vs + (size_t)kLinChunk * kLcVPitch;
  const size_t qk = (size_t)c * kLinChunk * a.ld + (size_t)(h / a.share) * a.dim;
  if (TOKEN) {
    if (threadIdx.x < kLinChunk)
      s_tok[threadIdx.x] = threadIdx.x < n ? a.token[(size_t)h * a.token_ld + c * kLinChunk + threadIdx.x] : make_float4(0.f, 0.f, 0.f, 0.f);
  } else if (threadIdx.x <= kLinChunk) {
    s_pw[threadIdx.x] = a.decay_pow[h * (kLinChunk + 1) + threadIdx.x];
  }
  lc_stage(smem, kp, static_cast<const uint16_t *>(a.q) + qk, a.ld, n, a.dim, a.silu);
  lc_stage(Ks, kp, static_cast<const uint16_t *>(a.k) + qk, a.ld, n, a.dim, a.silu);
  lc_stage(Vs, kLcVPitch, static_cast<const uint16_t *>(a.v) + (size_t)c * kLinChunk * a.ld + (size_t)h * a.vdim + v0, a.ld, n, vc, a.silu);
  const float *S = a.chunk_state + (((size_t)c * a.heads + h) * a.dim) * a.vdim + v0;
  constexpr int kStateAhead = 8;
  const int per = vc / 4, total = a.dim * per;
  for (int u0 = threadIdx.x; u0 < total; u0 += kStateAhead * kLcThreads) {  // the state in three parts
    float4 x[kStateAhead];
#pragma unroll
    for (int q = 0; q < kStateAhead; ++q) {
      const int u = u0 + q * kLcThreads, r = u / per;
      x[q] = u < total ? *reinterpret_cast<const float4 *>(S + (size_t)r * a.vdim + (u - r * per) * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
#pragma unroll
    for (int q = 0; q < kStateAhead; ++q) {
      const int u = u0 + q * kLcThreads, r = u / per, col = (u - r * per) * 4;
      if (u >= total) break;
      uint32_t p0[kSplitParts], p1[kSplitParts];
      split_pair(x[q].x, x[q].y, p0);
      split_pair(x[q].z, x[q].w, p1);
#pragma unroll
      for (int p = 0; p < kSplitParts; ++p)
        *reinterpret_cast<uint2 *>(Ss + (size_t)(p * a.dim + r) * kLcVPitch + col * 2) = make_uint2(p0[p], p1[p]);
    }
  }
  lc_wait();
  const int m0 = (warp & 3) * 16, c0 = (warp >> 2) * (kLcCols / 2);
  if (m0 >= n || c0 >= vc) return;  // no barrier follows
  constexpr int kTiles = kLcCols / 16;  // the warp's column tiles of 8
  const uint32_t qs = (uint32_t)__cvta_generic_to_shared(smem), ks = (uint32_t)__cvta_generic_to_shared(Ks);
  const uint32_t vs = (uint32_t)__cvta_generic_to_shared(Vs), ss = (uint32_t)__cvta_generic_to_shared(Ss);
  float sc[kLinChunk / 8][4] = {}, acc[kTiles][4] = {};
  for (int k0 = 0; k0 < a.dim; k0 += 16) {
    uint32_t q0, q1, q2, q3;
    ldsm4(frag_a(qs, m0, k0, kp, lane), q0, q1, q2, q3);
#pragma unroll
    for (int nt = 0; nt < kLinChunk / 8; nt += 2) {
      if (nt * 8 <= m0 + 15) {  // later keys are invisible to every token of the warp
        uint32_t b0, b1, b2, b3;
        ldsm4(frag_b(ks, nt * 8, k0, kp, lane), b0, b1, b2, b3);
        mma_bf16_16816(sc[nt], q0, q1, q2, q3, b0, b1);
        mma_bf16_16816(sc[nt + 1], q0, q1, q2, q3, b2, b3);
      }
    }
#pragma unroll
    for (int nt = 0; nt < kTiles; nt += 2) {
      if (c0 + nt * 8 < vc) {
#pragma unroll
        for (int p = 0; p < kSplitParts; ++p) {
          uint32_t b0, b1, b2, b3;
          ldsm4_t(frag_b_t(ss + p * a.dim * kLcVPitch, c0 + nt * 8, k0, kLcVPitch, lane), b0, b1, b2, b3);
          mma_bf16_16816(acc[nt], q0, q1, q2, q3, b0, b1);
          mma_bf16_16816(acc[nt + 1], q0, q1, q2, q3, b2, b3);
        }
      }
    }
  }
  // the state's share decays by one step more than the token's place in the chunk
  float d_lo, d_hi;
  float4 k_lo, k_hi;  // the tokens' own entries
  if (TOKEN) {
    k_lo = s_tok[m0 + g], k_hi = s_tok[m0 + g + 8];
    d_lo = expf(k_lo.z + k_lo.w), d_hi = expf(k_hi.z + k_hi.w);
  } else {
    d_lo = s_pw[m0 + g + 1], d_hi = s_pw[m0 + g + 9];
  }
#pragma unroll
  for (int nt = 0; nt < kTiles; ++nt) {
    acc[nt][0] *= d_lo;
    acc[nt][1] *= d_lo;
    acc[nt][2] *= d_hi;
    acc[nt][3] *= d_hi;
  }
  const int i_lo = m0 + g, i_hi = m0 + g + 8;
#pragma unroll
  for (int kk = 0; kk < kLinChunk / 16; ++kk) {
    if (kk * 16 <= m0 + 15) {
      uint32_t fa[4][kSplitParts];
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const float *s = sc[2 * kk + half];
        const int j = kk * 16 + half * 8 + 2 * t;
        float w0, w1, w2, w3;
        if (TOKEN) {
          const float4 a0 = s_tok[j], a1 = s_tok[j + 1];
          w0 = j <= i_lo ? s[0] * a0.x * lc_between(k_lo, a0) : 0.f, w1 = j + 1 <= i_lo ? s[1] * a1.x * lc_between(k_lo, a1) : 0.f;
          w2 = j <= i_hi ? s[2] * a0.x * lc_between(k_hi, a0) : 0.f, w3 = j + 1 <= i_hi ? s[3] * a1.x * lc_between(k_hi, a1) : 0.f;
        } else {
          w0 = j <= i_lo ? s[0] * a.k_scale * s_pw[i_lo - j] : 0.f, w1 = j + 1 <= i_lo ? s[1] * a.k_scale * s_pw[i_lo - j - 1] : 0.f;
          w2 = j <= i_hi ? s[2] * a.k_scale * s_pw[i_hi - j] : 0.f, w3 = j + 1 <= i_hi ? s[3] * a.k_scale * s_pw[i_hi - j - 1] : 0.f;
        }
        split_pair(w0, w1, fa[2 * half]);
        split_pair(w2, w3, fa[2 * half + 1]);
      }
#pragma unroll
      for (int nt = 0; nt < kTiles; nt += 2) {
        if (c0 + nt * 8 < vc) {
          uint32_t b0, b1, b2, b3;
          ldsm4_t(frag_b_t(vs, c0 + nt * 8, kk * 16, kLcVPitch, lane), b0, b1, b2, b3);
#pragma unroll
          for (int p = 0; p < kSplitParts; ++p) {
            mma_bf16_16816(acc[nt], fa[0][p], fa[1][p], fa[2][p], fa[3][p], b0, b1);
            mma_bf16_16816(acc[nt + 1], fa[0][p], fa[1][p], fa[2][p], fa[3][p], b2, b3);
          }
        }
      }
    }
  }
  if (TOKEN) {
    const float skip = a.skip[h];
#pragma unroll
    for (int nt = 0; nt < kTiles; ++nt) {
      if (c0 + nt * 8 < vc) {
        const unsigned char *v = Vs + (size_t)i_lo * kLcVPitch + (c0 + nt * 8 + 2 * t) * 2;
        const uint32_t lo = *reinterpret_cast<const uint32_t *>(v), hi = *reinterpret_cast<const uint32_t *>(v + 8 * kLcVPitch);
        acc[nt][0] = fmaf(skip, bf16lo(lo), acc[nt][0]);
        acc[nt][1] = fmaf(skip, bf16hi(lo), acc[nt][1]);
        acc[nt][2] = fmaf(skip, bf16lo(hi), acc[nt][2]);
        acc[nt][3] = fmaf(skip, bf16hi(hi), acc[nt][3]);
      }
    }
  }
  const int hv = a.heads * a.vdim;
  float *o = a.o + (size_t)c * kLinChunk * hv + (size_t)h * a.vdim + v0;
#pragma unroll
  for (int nt = 0; nt < kTiles; ++nt) {
    if (c0 + nt * 8 < vc) {
      const int col = c0 + nt * 8 + 2 * t;
      if (i_lo < n) *reinterpret_cast<float2 *>(o + (size_t)i_lo * hv + col) = make_float2(acc[nt][0], acc[nt][1]);
      if (i_hi < n) *reinterpret_cast<float2 *>(o + (size_t)i_hi * hv + col) = make_float2(acc[nt][2], acc[nt][3]);
    }
  }
}

// ---- norm over a head (or all heads), weight, gate ----
template <typename Act>
__global__ void __launch_bounds__(256) gated_norm_kernel(const GatedNorm a) {
  __shared__ float s_red[8];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, n = a.heads * a.vdim;
  const float *o = a.o + (size_t)blockIdx.x * n;
  const Act *g = static_cast<const Act *>(a.g) + (size_t)blockIdx.x * a.ldg;
  Act *out = static_cast<Act *>(a.out) + (size_t)blockIdx.x * a.ldo;
  auto gates4 = [&](int i) {  // columns i .. i + 3 of the gate
    if constexpr (sizeof(Act) == 2) {
      const uint2 v = *reinterpret_cast<const uint2 *>(g + i);
      return make_float4(bf16lo(v.x), bf16hi(v.x), bf16lo(v.y), bf16hi(v.y));
    } else {
      return *reinterpret_cast<const float4 *>(g + i);
    }
  };
  auto write4 = [&](int i, float4 v, float4 gate, float scale) {
    const float x[4] = {v.x, v.y, v.z, v.w}, zs[4] = {gate.x, gate.y, gate.z, gate.w};
    float r[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const float z = zs[j], e = 1.0f / (1.0f + expf(-z));
      r[j] = x[j] * scale * (a.w ? a.w[i + j] : 1.f) * (a.gate == GATE_SILU ? z * e : e);
    }
    if constexpr (sizeof(Act) == 2) *reinterpret_cast<uint2 *>(out + i) = make_uint2(pack_bf16x2(r[0], r[1]), pack_bf16x2(r[2], r[3]));
    else *reinterpret_cast<float4 *>(out + i) = make_float4(r[0], r[1], r[2], r[3]);
  };
  auto sq = [](float4 v, float s) { return fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, s)))); };
  constexpr int kKeep = 8;  // a thread's values stay in registers between the sum and the scaling; longer rows are read again
  float4 keep[kKeep];
  if (a.per_head) {
    const int step = 8 * gridDim.y;
    int h = blockIdx.y * 8 + warp;
    if (a.vdim <= 128) {  // a lane holds four columns of a head: four heads in flight per warp
      const int i = lane * 4;
      const bool in = i < a.vdim;
      for (; h < a.heads; h += 4 * step) {
        float4 v[4], z[4];
#pragma unroll
        for (int q = 0; q < 4; ++q) {
          const bool ok = in && h + q * step < a.heads;
          v[q] = ok ? *reinterpret_cast<const float4 *>(o + (h + q * step) * a.vdim + i) : make_float4(0.f, 0.f, 0.f, 0.f);
          z[q] = ok ? gates4((h + q * step) * a.vdim + i) : v[q];
        }
#pragma unroll
        for (int q = 0; q < 4; ++q) {
          const float scale = 1.0f / sqrtf(warp_sum(sq(v[q], 0.f)) / (float)a.true_vdim + a.eps);
          if (in && h + q * step < a.heads) write4((h + q * step) * a.vdim + i, v[q], z[q], scale);
        }
      }
    }
    for (; h < a.heads; h += step) {
      float s = 0.f;
#pragma unroll
      for (int k = 0; k < kKeep; ++k) {
        const int i = (lane + 32 * k) * 4;
        if (i < a.vdim) s = sq(keep[k] = *reinterpret_cast<const float4 *>(o + h * a.vdim + i), s);
      }
      for (int i = (lane + 32 * kKeep) * 4; i < a.vdim; i += 128) s = sq(*reinterpret_cast<const float4 *>(o + h * a.vdim + i), s);
      const float scale = 1.0f / sqrtf(warp_sum(s) / (float)a.true_vdim + a.eps);
#pragma unroll
      for (int k = 0; k < kKeep; ++k) {
        const int i = (lane + 32 * k) * 4;
        if (i < a.vdim) write4(h * a.vdim + i, keep[k], gates4(h * a.vdim + i), scale);
      }
      for (int i = (lane + 32 * kKeep) * 4; i < a.vdim; i += 128) write4(h * a.vdim + i, *reinterpret_cast<const float4 *>(o + h * a.vdim + i), gates4(h * a.vdim + i), scale);
    }
  } else {
    float s = 0.f;
#pragma unroll
    for (int k = 0; k < kKeep; ++k) {
      const int i = (tid + 256 * k) * 4;
      if (i < n) s = sq(keep[k] = *reinterpret_cast<const float4 *>(o + i), s);
    }
    for (int i = (tid + 256 * kKeep) * 4; i < n; i += 1024) s = sq(*reinterpret_cast<const float4 *>(o + i), s);
    s = warp_sum(s);
    if (lane == 0) s_red[warp] = s;
    __syncthreads();
    s = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) s += s_red[w];
    const float scale = 1.0f / sqrtf(s / (float)(a.heads * a.true_vdim) + a.eps);
    // several CTAs of one token: CTA y writes every gridDim.y-th group of 1,024 columns
#pragma unroll
    for (int k = 0; k < kKeep; ++k) {
      const int i = (tid + 256 * k) * 4;
      if (k % gridDim.y == blockIdx.y && i < n) write4(i, keep[k], gates4(i), scale);
    }
    for (int k = kKeep, i = (tid + 256 * kKeep) * 4; i < n; ++k, i += 1024)
      if (k % gridDim.y == blockIdx.y) write4(i, *reinterpret_cast<const float4 *>(o + i), gates4(i), scale);
  }
  if (blockIdx.y == 0)
    for (int i = n + tid; i < a.ldo; i += 256) out[i] = Act(0);
}

int launch_gated_norm(const GatedNorm &a, int T, cudaStream_t stream) {
  // few tokens: several CTAs share a token's heads (or columns; each then takes the whole sum)
  const int parts = T >= sm_count() ? 1 : (a.per_head ? (a.heads + 7) / 8 : (a.heads * a.vdim + 1023) / 1024);
  const dim3 grid(T, parts < 1 ? 1 : parts);
  if (a.f32) gated_norm_kernel<float><<<grid, 256, 0, stream>>>(a);
  else gated_norm_kernel<uint16_t><<<grid, 256, 0, stream>>>(a);
  return launch_status("gated_norm_kernel");
}

static LaArgs la_args(const LinearAttn &a) {
  LaArgs r{};
  const size_t esz = a.f32 ? 4 : 2, hd = (size_t)a.heads / a.share * a.dim;
  const char *p = static_cast<const char *>(a.qkvg);
  r.q = p + (a.v_first ? ((size_t)a.heads * a.vdim + hd) * esz : 0);
  r.k = p + (a.v_first ? (size_t)a.heads * a.vdim : hd) * esz;
  r.v = p + (a.v_first ? 0 : 2 * hd * esz);
  r.share = a.share;
  r.token = a.token;
  r.token_ld = a.token_ld;
  r.skip = a.skip;
  r.decay_pow = a.decay_pow;
  r.state = a.state;
  r.o = a.o;
  r.chunk_state = a.chunk_state;
  r.heads = a.heads;
  r.dim = a.dim;
  r.vdim = a.vdim;
  r.ld = a.ld;
  r.silu = a.silu_qkv;
  r.k_scale = a.k_scale;
  return r;
}

template <typename Act, bool TOKEN>
static int recurrent_of(const LaArgs &r, int seqs, cudaStream_t stream) {
  const dim3 grid((r.vdim + 31) / 32, r.heads, seqs);
  if (r.dim <= 64) linear_recurrent_kernel<Act, 2, TOKEN><<<grid, 256, 0, stream>>>(r);
  else if (r.dim <= 128) linear_recurrent_kernel<Act, 4, TOKEN><<<grid, 256, 0, stream>>>(r);
  else linear_recurrent_kernel<Act, 8, TOKEN><<<grid, 256, 0, stream>>>(r);
  return launch_status("linear_recurrent_kernel");
}
template <typename Act>
static int recurrent(const LaArgs &r, int seqs, cudaStream_t stream) {
  return r.token ? recurrent_of<Act, true>(r, seqs, stream) : recurrent_of<Act, false>(r, seqs, stream);
}

static int check_shape(const LinearAttn &a) {
  BLOK_REQUIRE(a.share >= 1 && a.heads % a.share == 0 && (!a.token || a.skip), BLOK_ERR_SHAPE, "linear attention: %d heads, %d to a key", a.heads, a.share);
  BLOK_REQUIRE(a.heads >= 1 && a.dim >= 16 && a.dim % 16 == 0 && a.dim <= kLinMaxDim && a.vdim >= 16 && a.vdim % 16 == 0 && a.ld % 8 == 0,
               BLOK_ERR_SHAPE, "linear attention: %d heads of %d x %d (a head's key size is at most %d)", a.heads, a.dim, a.vdim, kLinMaxDim);
  return BLOK_OK;
}

int launch_linear_step(const LinearAttn &a, const StackRows &rows, int B, cudaStream_t stream) {
  if (int rc = check_shape(a)) return rc;
  LaArgs r = la_args(a);
  r.slot_of = rows.slot_of;
  r.pos = rows.pos;
  r.T = 1;
  return a.f32 ? recurrent<float>(r, B, stream) : recurrent<uint16_t>(r, B, stream);
}

size_t linear_chunk_scratch_bytes(int heads, int dim, int vdim, int T) {
  return (size_t)((T + kLinChunk - 1) / kLinChunk) * heads * dim * vdim * sizeof(float);
}

template <bool TOKEN>
static int chunked(const LaArgs &r, cudaStream_t stream) {
  const int kp = r.dim * 2 + 16;
  const dim3 grid(r.chunks, r.heads, (r.vdim + kLcCols - 1) / kLcCols);
  const size_t smem1 = (size_t)kSplitParts * kLinChunk * kp + (size_t)kLinChunk * kLcVPitch;
  const size_t smem3 = (size_t)2 * kLinChunk * kp + (size_t)kLinChunk * kLcVPitch + (size_t)kSplitParts * r.dim * kLcVPitch;
  BLOK_CUDA(cudaFuncSetAttribute(linear_chunk_state_kernel<TOKEN>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem1));
  BLOK_CUDA(cudaFuncSetAttribute(linear_chunk_out_kernel<TOKEN>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem3));
  linear_chunk_state_kernel<TOKEN><<<grid, kLcThreads, smem1, stream>>>(r);
  if (int rc = launch_status("linear_chunk_state_kernel")) return rc;
  linear_scan_kernel<TOKEN><<<dim3((r.dim * r.vdim / 4 + 127) / 128, r.heads), 128, 0, stream>>>(r);
  if (int rc = launch_status("linear_scan_kernel")) return rc;
  linear_chunk_out_kernel<TOKEN><<<grid, kLcThreads, smem3, stream>>>(r);
  return launch_status("linear_chunk_out_kernel");
}

int launch_linear_chunk(const LinearAttn &a, int slot, long first_pos, int T, cudaStream_t stream) {
  if (int rc = check_shape(a)) return rc;
  LaArgs r = la_args(a);
  r.slot = slot;
  r.fresh = first_pos == 0;
  r.T = T;
  if (a.f32) return recurrent<float>(r, 1, stream);
  if (T <= 8) return recurrent<uint16_t>(r, 1, stream);
  r.chunks = (T + kLinChunk - 1) / kLinChunk;
  return a.token ? chunked<true>(r, stream) : chunked<false>(r, stream);
}

}  // namespace blok
