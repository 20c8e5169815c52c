// Softmax attention with grouped heads over a paged cache whose row is [keys of every key head | values of every key head]:
//   score_h(i, j) = (q_h(i) . k_g(j)) * scale + bias_h(i - j),   out_h(i) = gate_h(i) * sum_j softmax_j v_g(j),   g = h / (heads / kv_heads)
// causal, with an optional bias per head and distance and an optional sigmoid gate per head and token.
//
// Decode and short portions: a CTA takes the query heads of one key head of one entry (16 or 32 rows of a tensor-core
// tile) and a range of the context in tiles of 64 rows; the parts are merged afterwards (mla_merge.cuh), where the gate is
// applied.  Long portions: prompt_attn_tc.cu (tcgen05).  fp32 models, and heads too wide for either, use CUDA cores.
//
// Scores, bias, softmax and its weights are fp32; the weights enter the second product in three bf16 parts (bf16_split.cuh).
#include <algorithm>

#include "bf16_split.cuh"
#include "mla_merge.cuh"
#include "stack_kernels.h"

namespace blok {

constexpr float kGaLog2e = 1.4426950408889634f;

template <typename Act>
__device__ __forceinline__ float ga_load(const Act *p) {
  if constexpr (sizeof(Act) == 2) return bf16_bits_to_f32(*p);
  else return *p;
}
template <typename Act>
__device__ __forceinline__ void ga_store(Act *p, float v) {
  if constexpr (sizeof(Act) == 2) *p = f32_to_bf16_bits(v);
  else *p = v;
}
__device__ __forceinline__ size_t ga_row(const StackRows &r, int slot, int pos) {
  return (size_t)r.table[(size_t)slot * r.table_stride + pos / r.page_rows] * r.page_rows + pos % r.page_rows;
}

// ---- norms over all of q and all of k, cache append; one CTA per token ----
template <typename Act>
__global__ void __launch_bounds__(256) grouped_append_kernel(const GroupedShape s, Act *__restrict__ qkv, int ld, const float *__restrict__ q_norm,
                                                             const float *__restrict__ k_norm, const StackRows r, Act *__restrict__ pool) {
  __shared__ float s_red[2][8];
  const int t = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int nq = s.heads * s.dim, nk = pool ? s.kv_heads * s.dim : 0, nv = s.kv_heads * s.vdim;
  Act *q = qkv + (size_t)t * ld;
  const Act *k = q + nq;
  auto four = [](const Act *p) {
    if constexpr (sizeof(Act) == 2) {
      const uint2 v = *reinterpret_cast<const uint2 *>(p);
      return make_float4(bf16lo(v.x), bf16hi(v.x), bf16lo(v.y), bf16hi(v.y));
    } else {
      return *reinterpret_cast<const float4 *>(p);
    }
  };
  auto scaled = [&](Act *dst, const Act *src, const float *w, float f, int i) {
    const float4 v = four(src + i), n = *reinterpret_cast<const float4 *>(w + i);
    if constexpr (sizeof(Act) == 2)
      *reinterpret_cast<uint2 *>(dst + i) = make_uint2(pack_bf16x2(v.x * f * n.x, v.y * f * n.y), pack_bf16x2(v.z * f * n.z, v.w * f * n.w));
    else *reinterpret_cast<float4 *>(dst + i) = make_float4(v.x * f * n.x, v.y * f * n.y, v.z * f * n.z, v.w * f * n.w);
  };
  auto copy = [&](Act *dst, const Act *src, int i) {
    if constexpr (sizeof(Act) == 2) *reinterpret_cast<uint2 *>(dst + i) = *reinterpret_cast<const uint2 *>(src + i);
    else *reinterpret_cast<float4 *>(dst + i) = *reinterpret_cast<const float4 *>(src + i);
  };
  float rq = 0.f, rk = 0.f;
  if (q_norm) {
    float sq = 0.f, sk = 0.f;
    auto add = [&](const Act *p, int i, float a) {
      const float4 v = four(p + i);
      return fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, a))));
    };
    for (int i = tid * 4; i < nq; i += 1024) sq = add(q, i, sq);
    for (int i = tid * 4; i < nk; i += 1024) sk = add(k, i, sk);
    sq = warp_sum(sq);
    sk = warp_sum(sk);
    if (lane == 0) s_red[0][warp] = sq, s_red[1][warp] = sk;
    __syncthreads();
    sq = sk = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) sq += s_red[0][w], sk += s_red[1][w];
    // the padding holds zeros: the means are over the true columns
    rq = 1.0f / sqrtf(sq / (float)(s.heads * s.true_dim) + s.eps);
    rk = 1.0f / sqrtf(sk / (float)(s.kv_heads * s.true_dim) + s.eps);
    for (int i = tid * 4; i < nq; i += 1024) scaled(q, q, q_norm, rq, i);
  }
  if (!pool) return;  // another layer's keys and values
  const int pos = r.pos[t];
  if (pos < 0 || pos >= r.table_stride * r.page_rows) return;  // the host keeps positions inside the table
  Act *row = pool + ga_row(r, r.slot_of[t], pos) * s.row();
  for (int i = tid * 4; i < nk; i += 1024) {
    if (q_norm) scaled(row, k, k_norm, rk, i);
    else copy(row, k, i);
  }
  for (int i = tid * 4; i < nv; i += 1024) copy(row + nk, k + nk, i);
}

int launch_grouped_append(const GroupedShape &s, void *qkv, int ld, const float *q_norm, const float *k_norm, const StackRows &r, int T, void *pool,
                          bool f32, cudaStream_t stream) {
  BLOK_REQUIRE(s.dim % 4 == 0 && s.vdim % 4 == 0 && ld % 4 == 0, BLOK_ERR_SHAPE, "grouped attention: rows of %d values", ld);
  if (f32) grouped_append_kernel<float><<<T, 256, 0, stream>>>(s, static_cast<float *>(qkv), ld, q_norm, k_norm, r, static_cast<float *>(pool));
  else grouped_append_kernel<uint16_t><<<T, 256, 0, stream>>>(s, static_cast<uint16_t *>(qkv), ld, q_norm, k_norm, r, static_cast<uint16_t *>(pool));
  return launch_status("grouped_append_kernel");
}

__device__ __forceinline__ float ga_gate(float z) { return 1.0f / (1.0f + expf(-z)); }

// ---- CUDA cores, any sizes: one CTA per (head, entry) ----
constexpr int kGsKeys = 128;

template <typename Act>
__global__ void __launch_bounds__(kGsKeys) grouped_attend_simple_kernel(const GroupedShape s, const GroupedQuery<Act> a, const Act *__restrict__ pool,
                                                                        const StackRows r) {
  extern __shared__ float sm[];  // q [dim], o [vdim]
  __shared__ float s_p[kGsKeys], s_red[kGsKeys / 32];
  __shared__ size_t s_row[kGsKeys];
  const int h = blockIdx.x, t = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, row = s.row(), kvh = h / (s.heads / s.kv_heads);
  const int pos = r.pos[t], n = min(pos + 1, r.table_stride * r.page_rows), slot = r.slot_of[t];
  const float *bias = s.bias ? s.bias + (size_t)h * s.bias_len : nullptr;
  float *sq = sm, *so = sm + s.dim;
  for (int i = tid; i < s.dim; i += kGsKeys) sq[i] = ga_load(a.q + (size_t)t * a.ldq + (size_t)h * s.dim + i);
  for (int i = tid; i < s.vdim; i += kGsKeys) so[i] = 0.f;
  float m = -INFINITY, l = 0.f;
  __syncthreads();
  for (int j0 = 0; j0 < n; j0 += kGsKeys) {
    const int cnt = min(kGsKeys, n - j0);
    float sc = -INFINITY;
    if (tid < cnt) {
      const size_t at = ga_row(r, slot, j0 + tid) * row;
      s_row[tid] = at + (size_t)s.kv_heads * s.dim + (size_t)kvh * s.vdim;
      const Act *k = pool + at + (size_t)kvh * s.dim;
      float d = 0.f;
      for (int i = 0; i < s.dim; ++i) d = fmaf(sq[i], ga_load(k + i), d);
      sc = d * s.scale;
      if (bias) sc += bias[min(pos - j0 - tid, s.bias_len - 1)];
    }
    float mx = warp_max(sc);
    if (lane == 0) s_red[warp] = mx;
    __syncthreads();
    mx = fmaxf(fmaxf(s_red[0], s_red[1]), fmaxf(s_red[2], s_red[3]));
    const float mn = fmaxf(m, mx), al = expf(m - mn), p = expf(sc - mn);
    s_p[tid] = p;
    const float sum = warp_sum(p);
    __syncthreads();
    if (lane == 0) s_red[warp] = sum;
    __syncthreads();
    l = l * al + ((s_red[0] + s_red[1]) + (s_red[2] + s_red[3]));
    m = mn;
    for (int i = tid; i < s.vdim; i += kGsKeys) {
      float o = so[i] * al;
      for (int j = 0; j < cnt; ++j) o = fmaf(s_p[j], ga_load(pool + s_row[j] + i), o);
      so[i] = o;
    }
    __syncthreads();
  }
  const float f = (a.gate ? ga_gate(ga_load(a.gate + (size_t)t * a.ld_gate + h)) : 1.f) / l;
  for (int i = tid; i < s.vdim; i += kGsKeys) ga_store(a.out + (size_t)t * a.ldo + (size_t)h * s.vdim + i, so[i] * f);
}

// ---- tensor cores (bf16): CTA = up to MT x 16 query heads of a key head of one entry, a range of the context ----
constexpr int kGaTile = 64, kGaWarps = 8, kGaThreads = kGaWarps * 32;
constexpr int kGaSPitch = kGaTile + 4;       // floats per score row
constexpr int kGaPPitch = kGaTile * 2 + 16;  // bytes per row of a weight part
constexpr int kGaMaxV = 256;

static size_t ga_smem_bytes(const GroupedShape &s, int mt) {
  const size_t kp = (size_t)s.dim * 2 + 16, vp = (size_t)s.vdim * 2 + 16;
  return mt * 16 * kp + 2 * kGaTile * (kp + vp) + (size_t)mt * 16 * kGaSPitch * 4 + (size_t)kSplitParts * mt * 16 * kGaPPitch;
}

// NT: column tiles of 8 values per warp (vdim <= 64 NT).
template <int MT, int NT>
__global__ void __launch_bounds__(kGaThreads, MT * NT <= 2 ? 2 : 1)
    grouped_attend_kernel(const GroupedShape s, const GroupedQuery<uint16_t> a, const uint16_t *__restrict__ pool, const StackRows r,
                          float *__restrict__ part_o, float *__restrict__ part_ml) {
  extern __shared__ __align__(16) unsigned char smem[];
  __shared__ float s_alpha[MT * 16];
  constexpr int M = MT * 16;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
  const int split = blockIdx.x, splits = gridDim.x, per_kv = s.heads / s.kv_heads, blocks = (per_kv + M - 1) / M;
  const int kvh = blockIdx.y / blocks, first = blockIdx.y % blocks * M, nh = min(M, per_kv - first), h0 = kvh * per_kv + first, b = blockIdx.z;
  const int kp = s.dim * 2 + 16, vp = s.vdim * 2 + 16;
  const int pos = r.pos[b], n = min(pos + 1, r.table_stride * r.page_rows);
  const int ntiles = (n + kGaTile - 1) / kGaTile, per = (ntiles + splits - 1) / splits;
  const int ts = split * per, te = min(ntiles, ts + per);
  float *ml = part_ml + (((size_t)b * splits + split) * s.heads + h0) * 2;
  if (ts >= te) {
    if (tid < nh) ml[tid * 2] = -INFINITY, ml[tid * 2 + 1] = 0.f;
    return;
  }
  const uint32_t qs = (uint32_t)__cvta_generic_to_shared(smem), ks = qs + M * kp, vs = ks + 2 * kGaTile * kp;
  float *Ss = reinterpret_cast<float *>(smem + (size_t)M * kp + (size_t)2 * kGaTile * (kp + vp));
  unsigned char *Ps = reinterpret_cast<unsigned char *>(Ss + M * kGaSPitch);
  const uint32_t ps = (uint32_t)__cvta_generic_to_shared(Ps);
  const int *table = r.table + (size_t)r.slot_of[b] * r.table_stride;
  const int qu = s.dim / 8, vu = s.vdim / 8;
  for (int u = tid; u < M * qu; u += kGaThreads) {
    const int h = u / qu, c = u - h * qu;  // heads past the last repeat it; their results are not stored
    cp_async16(qs + h * kp + c * 16, a.q + (size_t)b * a.ldq + (size_t)(h0 + min(h, nh - 1)) * s.dim + c * 8);
  }
  // a row of the tile belongs to four neighbouring threads: one look into the page table per thread and tile
  constexpr int kRowThreads = kGaThreads / kGaTile;
  const int lk = tid / kRowThreads, lc = tid % kRowThreads, row = s.row();
  auto load_tile = [&](int tile, int buf) {
    const int j = min(tile * kGaTile + lk, n - 1);  // rows past the end repeat the last; they take no weight
    const uint16_t *src = pool + ((size_t)table[j / r.page_rows] * r.page_rows + j % r.page_rows) * row;
    const uint16_t *sk = src + kvh * s.dim, *sv = src + s.kv_heads * s.dim + kvh * s.vdim;
    const uint32_t dk = ks + (uint32_t)(buf * kGaTile + lk) * kp, dv = vs + (uint32_t)(buf * kGaTile + lk) * vp;
#pragma unroll 4
    for (int c = lc; c < qu; c += kRowThreads) cp_async16(dk + c * 16, sk + c * 8);
#pragma unroll 4
    for (int c = lc; c < vu; c += kRowThreads) cp_async16(dv + c * 16, sv + c * 8);
  };
  load_tile(ts, 0);
  asm volatile("cp.async.commit_group;" ::: "memory");
  float o[MT][NT][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int i = 0; i < NT; ++i) o[m][i][0] = o[m][i][1] = o[m][i][2] = o[m][i][3] = 0.f;
  // the softmax of a head row belongs to kGaThreads / M consecutive lanes
  constexpr int kPer = kGaThreads / M, kCols = kGaTile / kPer;
  const int sh = tid / kPer, sl = tid % kPer;
  float m_run = -INFINITY, l_run = 0.f;
  const float sl2 = s.scale * kGaLog2e;
  const float *bias = s.bias ? s.bias + (size_t)(h0 + min(sh, nh - 1)) * s.bias_len : nullptr;
  for (int tile = ts; tile < te; ++tile) {
    const int buf = (tile - ts) & 1;
    // this row's biases, on their way while the tile is
    float bv[kCols];
#pragma unroll
    for (int i = 0; i < kCols; ++i) bv[i] = bias ? bias[min(max(pos - (tile * kGaTile + sl * kCols + i), 0), s.bias_len - 1)] : 0.f;
    if (tile + 1 < te) load_tile(tile + 1, buf ^ 1);
    asm volatile("cp.async.commit_group;" ::: "memory");
    asm volatile("cp.async.wait_group 1;" ::: "memory");
    __syncthreads();
    const uint32_t kb = ks + (uint32_t)(buf * kGaTile) * kp, vb = vs + (uint32_t)(buf * kGaTile) * vp;
    {  // scores of 8 rows per warp
      float sc[MT][4] = {};
      const uint32_t baddr = kb + (uint32_t)(8 * warp + (lane & 7)) * kp + (lane >> 3) * 16;
#pragma unroll 2
      for (int k0 = 0; k0 < s.dim; k0 += 32) {
        uint32_t b0, b1, b2, b3;
        ldsm4(baddr + k0 * 2, b0, b1, b2, b3);
#pragma unroll
        for (int m = 0; m < MT; ++m) {
          uint32_t a0, a1, a2, a3;
          ldsm4(frag_a(qs, 16 * m, k0, kp, lane), a0, a1, a2, a3);
          mma_bf16_16816(sc[m], a0, a1, a2, a3, b0, b1);
          ldsm4(frag_a(qs, 16 * m, k0 + 16, kp, lane), a0, a1, a2, a3);
          mma_bf16_16816(sc[m], a0, a1, a2, a3, b2, b3);
        }
      }
#pragma unroll
      for (int m = 0; m < MT; ++m) {
        float *d = Ss + (16 * m + g) * kGaSPitch + 8 * warp + 2 * t;
        *reinterpret_cast<float2 *>(d) = make_float2(sc[m][0], sc[m][1]);
        *reinterpret_cast<float2 *>(d + 8 * kGaSPitch) = make_float2(sc[m][2], sc[m][3]);
      }
    }
    __syncthreads();
    {  // online softmax in the log2 domain
      float v[kCols], mx = -INFINITY, sum = 0.f;
      const int j = tile * kGaTile + sl * kCols;
#pragma unroll
      for (int i = 0; i < kCols; i += 2) {
        const float2 x = *reinterpret_cast<const float2 *>(Ss + sh * kGaSPitch + sl * kCols + i);
        v[i] = j + i < n ? fmaf(x.x, sl2, bv[i] * kGaLog2e) : -INFINITY;
        v[i + 1] = j + i + 1 < n ? fmaf(x.y, sl2, bv[i + 1] * kGaLog2e) : -INFINITY;
        mx = fmaxf(mx, fmaxf(v[i], v[i + 1]));
      }
#pragma unroll
      for (int d = 1; d < kPer; d <<= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, d));
      const float mn = fmaxf(m_run, mx), al = exp2f(m_run - mn);  // a tile of the range holds at least one key: mn is finite
      m_run = mn;
#pragma unroll
      for (int i = 0; i < kCols; i += 2) {
        const float p0 = exp2f(v[i] - mn), p1 = exp2f(v[i + 1] - mn);
        sum += p0 + p1;
        uint32_t part[kSplitParts];
        split_pair(p0, p1, part);
#pragma unroll
        for (int p = 0; p < kSplitParts; ++p) *reinterpret_cast<uint32_t *>(Ps + (size_t)(p * M + sh) * kGaPPitch + (sl * kCols + i) * 2) = part[p];
      }
#pragma unroll
      for (int d = 1; d < kPer; d <<= 1) sum += __shfl_xor_sync(0xffffffffu, sum, d);
      l_run = l_run * al + sum;
      if (sl == 0) s_alpha[sh] = al;
    }
    __syncthreads();
    // O += P V, columns of 8 values: warp, warp + 8, ... (pairs of tiles share a load)
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      const float al = s_alpha[16 * m + g], ah = s_alpha[16 * m + g + 8];
#pragma unroll
      for (int i = 0; i < NT; ++i) {
        o[m][i][0] *= al;
        o[m][i][1] *= al;
        o[m][i][2] *= ah;
        o[m][i][3] *= ah;
      }
    }
#pragma unroll
    for (int k0 = 0; k0 < kGaTile; k0 += 16) {
      uint32_t fa[MT][kSplitParts][4];
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int p = 0; p < kSplitParts; ++p)
          ldsm4(frag_a(ps + (uint32_t)(p * M) * kGaPPitch, 16 * m, k0, kGaPPitch, lane), fa[m][p][0], fa[m][p][1], fa[m][p][2], fa[m][p][3]);
#pragma unroll
      for (int i = 0; i < NT; i += 2) {
        const int col = (warp + kGaWarps * (i / 2)) * 16;
        if (col < s.vdim) {
          uint32_t b0, b1, b2, b3;
          ldsm4_t(frag_b_t(vb, col, k0, vp, lane), b0, b1, b2, b3);
#pragma unroll
          for (int m = 0; m < MT; ++m)
#pragma unroll
            for (int p = 0; p < kSplitParts; ++p) {
              mma_bf16_16816(o[m][i], fa[m][p][0], fa[m][p][1], fa[m][p][2], fa[m][p][3], b0, b1);
              mma_bf16_16816(o[m][i + 1], fa[m][p][0], fa[m][p][1], fa[m][p][2], fa[m][p][3], b2, b3);
            }
        }
      }
    }
    __syncthreads();  // the tile buffer, the weights and their scales are free again
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  float *po = part_o + (((size_t)b * splits + split) * s.heads + h0) * s.vdim;
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int i = 0; i < NT; ++i) {
      const int col = (warp + kGaWarps * (i / 2)) * 16 + (i & 1) * 8 + 2 * t, h = 16 * m + g;
      if (col < s.vdim) {
        if (h < nh) *reinterpret_cast<float2 *>(po + (size_t)h * s.vdim + col) = make_float2(o[m][i][0], o[m][i][1]);
        if (h + 8 < nh) *reinterpret_cast<float2 *>(po + (size_t)(h + 8) * s.vdim + col) = make_float2(o[m][i][2], o[m][i][3]);
      }
    }
  if (sl == 0 && sh < nh) {
    ml[sh * 2] = m_run * 0.6931471805599453f;  // natural units, as the merge takes them
    ml[sh * 2 + 1] = l_run;
  }
}

static int ga_mt(const GroupedShape &s) { return s.heads / s.kv_heads > 16 ? 2 : 1; }
static bool ga_tensor(const GroupedShape &s) { return s.vdim <= kGaMaxV && ga_smem_bytes(s, ga_mt(s)) <= 227 * 1024; }
static int ga_blocks(const GroupedShape &s) {
  const int per_kv = s.heads / s.kv_heads, m = 16 * ga_mt(s);
  return s.kv_heads * ((per_kv + m - 1) / m);
}
static int ga_splits(const GroupedShape &s, int T, long max_ctx) {
  const long cap = (max_ctx + 2 * kGaTile - 1) / (2 * kGaTile);  // at least two tiles each
  return (int)std::max(1l, std::min(cap, (long)(2 * sm_count()) / ((long)ga_blocks(s) * T)));
}

size_t grouped_attend_max_parts(const GroupedShape &s, int T, long max_ctx) {
  if (!ga_tensor(s)) return 0;
  size_t worst = 0;
  for (int t = 1; t <= T; ++t) worst = std::max(worst, (size_t)t * ga_splits(s, t, max_ctx));
  return worst;
}

template <typename Act>
static int ga_simple(const GroupedShape &s, const GroupedQuery<Act> &a, const void *pool, const StackRows &r, int T, cudaStream_t stream) {
  const size_t smem = (size_t)(s.dim + s.vdim) * sizeof(float);
  BLOK_REQUIRE(smem <= 200 * 1024, BLOK_ERR_SHAPE, "grouped attention: heads of %d / %d are too wide", s.dim, s.vdim);
  if (smem > 40 * 1024) BLOK_CUDA(cudaFuncSetAttribute(grouped_attend_simple_kernel<Act>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  grouped_attend_simple_kernel<Act><<<dim3(s.heads, T), kGsKeys, smem, stream>>>(s, a, static_cast<const Act *>(pool), r);
  return launch_status("grouped_attend_simple_kernel");
}

template <int MT, int NT>
static int ga_launch(const GroupedShape &s, const GroupedQuery<uint16_t> &a, const uint16_t *pool, const StackRows &r, int T, int splits, float *po,
                     float *pml, cudaStream_t stream) {
  const size_t smem = ga_smem_bytes(s, MT);
  BLOK_CUDA(cudaFuncSetAttribute(grouped_attend_kernel<MT, NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  grouped_attend_kernel<MT, NT><<<dim3(splits, ga_blocks(s), T), kGaThreads, smem, stream>>>(s, a, pool, r, po, pml);
  return launch_status("grouped_attend_kernel");
}

int launch_grouped_attend_f32(const GroupedShape &s, const GroupedQuery<float> &a, const void *pool, const StackRows &r, int T, cudaStream_t stream) {
  return ga_simple<float>(s, a, pool, r, T, stream);
}

int launch_grouped_attend(const GroupedShape &s, const GroupedQuery<uint16_t> &a, const void *pool, const StackRows &r, int T, long max_ctx,
                          float *part_o, float *part_ml, cudaStream_t stream) {
  if (!ga_tensor(s)) return ga_simple<uint16_t>(s, a, pool, r, T, stream);
  const int splits = ga_splits(s, T, max_ctx);
  const uint16_t *p = static_cast<const uint16_t *>(pool);
  int rc;
#define BLOK_GA(MT) \
  rc = s.vdim <= 128 ? ga_launch<MT, 2>(s, a, p, r, T, splits, part_o, part_ml, stream) : ga_launch<MT, 4>(s, a, p, r, T, splits, part_o, part_ml, stream)
  if (ga_mt(s) == 2) BLOK_GA(2);
  else BLOK_GA(1);
#undef BLOK_GA
  if (rc) return rc;
  mla_merge_kernel<<<dim3(s.heads, T), 128, (size_t)splits * sizeof(float), stream>>>(part_o, part_ml, splits, s.heads, s.vdim, a.out, a.ldo, a.gate,
                                                                                      a.ld_gate);
  return launch_status("mla_merge_kernel");
}

}  // namespace blok
