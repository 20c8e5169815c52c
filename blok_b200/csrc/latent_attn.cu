// Latent attention of any size over a paged cache whose row is [latent c | rotated key part]:
//   score_h(i, j) = (q_h . W_UK_h c_j + qr_h . kr_j) * scale,   out_h(i) = sum_j softmax_j W_UV_h c_j
//
// Two forms, both causal.  Absorbed (decode, short portions): queries multiplied by W_UK^T score against the cached rows
// themselves and the latents are averaged, one pass over the cache, the context split over CTAs (mla_merge.cuh adds the
// parts).  Prompt form (long portions): per-head keys and values are made from the cached latents by one product and a
// tile kernel walks them, which needs 3 to 4 times fewer multiply-adds per query and key (prompt_attn_tc.cu on tcgen05 for
// sizes in multiples of 64, the mma.sync kernel here for the others).
//
// Scores, softmax and its weights are fp32; the weights enter the second product in three bf16 parts (bf16_split.cuh).
// Positions become angles in double precision.  (The cores of mla_attend.cu and mla_attend_tc.cu are built for 64 heads of
// one size and round the weights to bf16.)
#include <algorithm>
#include <cstdlib>
#include <cstring>

#include "bf16_split.cuh"
#include "mla_merge.cuh"
#include "stack_kernels.h"

namespace blok {

template <typename Act>
__device__ __forceinline__ float lt_load(const Act *p) {
  if constexpr (sizeof(Act) == 2) return bf16_bits_to_f32(*p);
  else return *p;
}
template <typename Act>
__device__ __forceinline__ void lt_store(Act *p, float v) {
  if constexpr (sizeof(Act) == 2) *p = f32_to_bf16_bits(v);
  else *p = v;
}
__device__ __forceinline__ size_t lt_row(const StackRows &r, int slot, int pos) {
  return (size_t)r.table[(size_t)slot * r.table_stride + pos / r.page_rows] * r.page_rows + pos % r.page_rows;
}
// Sine and cosine at position pos of a pair that makes `rate` turns per position, reduced to one turn in double.
__device__ __forceinline__ void lt_angle(int pos, double rate, float *s, float *c) {
  const double turns = (double)pos * rate;
  sincosf((float)((turns - rint(turns)) * 6.28318530717958647693), s, c);
}

// ---- norms of the latents, rotation of the shared key part, cache append; one CTA per token ----
template <typename Act>
__global__ void __launch_bounds__(256) latent_append_kernel(const LatentShape s, const float *__restrict__ ckr, const float *__restrict__ q_norm,
                                                            const float *__restrict__ kv_norm, const StackRows r, Act *__restrict__ cq,
                                                            Act *__restrict__ pool) {
  __shared__ float s_red[2][8];
  const int t = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const float *q = ckr + (size_t)t * (s.q_rank + s.rank + s.rot), *c = q + s.q_rank, *k = c + s.rank;
  float sq = 0.f, sc = 0.f;
  for (int i = tid; i < s.true_q_rank; i += 256) sq = fmaf(q[i], q[i], sq);
  for (int i = tid; i < s.true_rank; i += 256) sc = fmaf(c[i], c[i], sc);
  sq = warp_sum(sq);
  sc = warp_sum(sc);
  if (lane == 0) s_red[0][warp] = sq, s_red[1][warp] = sc;
  __syncthreads();
  sq = sc = 0.f;
#pragma unroll
  for (int w = 0; w < 8; ++w) sq += s_red[0][w], sc += s_red[1][w];
  const float rq = 1.0f / sqrtf(sq / (float)s.true_q_rank + s.eps), rc = 1.0f / sqrtf(sc / (float)s.true_rank + s.eps);
  for (int i = tid; i < s.q_rank; i += 256) lt_store(cq + (size_t)t * s.q_rank + i, q[i] * rq * q_norm[i]);
  const int pos = r.pos[t];
  if (pos < 0 || pos >= r.table_stride * r.page_rows) return;  // the host keeps positions inside the table
  Act *row = pool + lt_row(r, r.slot_of[t], pos) * (s.rank + s.rot);
  for (int i = tid; i < s.rank; i += 256) lt_store(row + i, c[i] * rc * kv_norm[i]);
  row += s.rank;
  for (int i = tid; i < s.rot / 2; i += 256) {
    float u = k[2 * i], v = k[2 * i + 1];
    if (2 * i < s.rot_dims) {
      float sn, cs;
      lt_angle(pos, s.turns[i], &sn, &cs);
      const float a = u * cs - v * sn;
      v = v * cs + u * sn;
      u = a;
    }
    lt_store(row + 2 * i, u);
    lt_store(row + 2 * i + 1, v);
  }
}

int launch_latent_append(const LatentShape &s, const float *ckr, const float *q_norm, const float *kv_norm, const StackRows &r, int T, void *cq,
                         void *pool, bool f32, cudaStream_t stream) {
  if (f32) latent_append_kernel<float><<<T, 256, 0, stream>>>(s, ckr, q_norm, kv_norm, r, static_cast<float *>(cq), static_cast<float *>(pool));
  else latent_append_kernel<uint16_t><<<T, 256, 0, stream>>>(s, ckr, q_norm, kv_norm, r, static_cast<uint16_t *>(cq), static_cast<uint16_t *>(pool));
  return launch_status("latent_append_kernel");
}

template <typename Act>
__global__ void __launch_bounds__(256) latent_rotate_kernel(const LatentShape s, const Act *q, const StackRows r, int T, Act *dst,
                                                            int dst_head, int dst_off) {
  extern __shared__ float2 s_sc[];  // sine and cosine of every pair at this token's position
  const int t = blockIdx.x, pos = r.pos[t], half = s.rot / 2;
  for (int i = threadIdx.x; i < half; i += blockDim.x) {
    float sn = 0.f, cs = 1.f;
    if (2 * i < s.rot_dims) lt_angle(pos, s.turns[i], &sn, &cs);
    s_sc[i] = make_float2(sn, cs);
  }
  __syncthreads();
  for (int u = threadIdx.x + blockIdx.y * blockDim.x; u < s.heads * half; u += blockDim.x * gridDim.y) {
    const int h = u / half, i = u - h * half;
    const Act *p = q + ((size_t)t * s.heads + h) * s.head() + s.dim + 2 * i;
    const float a = lt_load(p), b = lt_load(p + 1);
    const float2 sc = s_sc[i];
    Act *o = dst + ((size_t)t * s.heads + h) * dst_head + dst_off + 2 * i;
    lt_store(o, a * sc.y - b * sc.x);
    lt_store(o + 1, b * sc.y + a * sc.x);
  }
}

int launch_latent_rotate(const LatentShape &s, const void *q, const StackRows &r, int T, void *dst, int dst_head, int dst_off, bool f32,
                         cudaStream_t stream) {
  const dim3 grid(T, T >= 64 ? 1 : std::max(1, s.heads * (s.rot / 2) / 512));
  const size_t smem = (size_t)(s.rot / 2) * sizeof(float2);
  if (f32) latent_rotate_kernel<float><<<grid, 256, smem, stream>>>(s, static_cast<const float *>(q), r, T, static_cast<float *>(dst), dst_head, dst_off);
  else latent_rotate_kernel<uint16_t><<<grid, 256, smem, stream>>>(s, static_cast<const uint16_t *>(q), r, T, static_cast<uint16_t *>(dst), dst_head, dst_off);
  return launch_status("latent_rotate_kernel");
}

// ---- absorbed form, any sizes, CUDA cores: one CTA per (head, entry).  fp32 models, and latents too wide for the tensor-
// core kernel below. ----
constexpr int kLsKeys = 128;

template <typename Act>
__global__ void __launch_bounds__(kLsKeys) latent_attend_simple_kernel(const LatentShape s, const Act *__restrict__ q_abs, const Act *__restrict__ pool,
                                                                       const StackRows r, Act *__restrict__ o) {
  extern __shared__ float sm[];  // q [row], o [rank]
  __shared__ float s_p[kLsKeys], s_red[kLsKeys / 32];
  __shared__ size_t s_row[kLsKeys];
  const int h = blockIdx.x, t = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, row = s.rank + s.rot;
  const int n = min(r.pos[t] + 1, r.table_stride * r.page_rows), slot = r.slot_of[t];
  float *sq = sm, *so = sm + row;
  for (int i = tid; i < row; i += kLsKeys) sq[i] = lt_load(q_abs + ((size_t)t * s.heads + h) * row + i);
  for (int i = tid; i < s.rank; i += kLsKeys) so[i] = 0.f;
  float m = -INFINITY, l = 0.f;
  __syncthreads();
  for (int j0 = 0; j0 < n; j0 += kLsKeys) {
    const int cnt = min(kLsKeys, n - j0);
    float sc = -INFINITY;
    if (tid < cnt) {
      const size_t at = lt_row(r, slot, j0 + tid);
      s_row[tid] = at;
      const Act *k = pool + at * row;
      float a = 0.f;
      for (int i = 0; i < row; ++i) a = fmaf(sq[i], lt_load(k + i), a);
      sc = a * s.scale;
    }
    float mx = warp_max(sc);
    if (lane == 0) s_red[warp] = mx;
    __syncthreads();
    mx = fmaxf(fmaxf(s_red[0], s_red[1]), fmaxf(s_red[2], s_red[3]));
    const float mn = fmaxf(m, mx), al = expf(m - mn);
    const float p = expf(sc - mn);
    s_p[tid] = p;
    float sum = warp_sum(p);
    __syncthreads();
    if (lane == 0) s_red[warp] = sum;
    __syncthreads();
    l = l * al + ((s_red[0] + s_red[1]) + (s_red[2] + s_red[3]));
    m = mn;
    for (int i = tid; i < s.rank; i += kLsKeys) {
      float a = so[i] * al;
      for (int j = 0; j < cnt; ++j) a = fmaf(s_p[j], lt_load(pool + s_row[j] * row + i), a);
      so[i] = a;
    }
    __syncthreads();
  }
  for (int i = tid; i < s.rank; i += kLsKeys) lt_store(o + ((size_t)t * s.heads + h) * s.rank + i, so[i] / l);
}

// ---- absorbed form on tensor cores (bf16): CTA = MT x 16 heads of one entry, a range of the context in tiles of 64 rows ----
constexpr int kLaTile = 64, kLaWarps = 8, kLaThreads = kLaWarps * 32;
constexpr int kLaMaxRank = 512;
constexpr int kLaSPitch = kLaTile + 4;             // floats per score row
constexpr int kLaPPitch = kLaTile * 2 + 16;        // bytes per row of a weight part

static size_t la_smem_bytes(const LatentShape &s, int mt) {
  const size_t pitch = (size_t)s.row() * 2 + 16;
  return (mt * 16 + 2 * kLaTile) * pitch + (size_t)mt * 16 * kLaSPitch * 4 + (size_t)kSplitParts * mt * 16 * kLaPPitch;
}

// NT: column tiles of 8 latents per warp (rank <= 64 NT).
template <int MT, int NT>
__global__ void __launch_bounds__(kLaThreads, 1)
    latent_attend_kernel(const LatentShape s, const uint16_t *__restrict__ q_abs, const uint16_t *__restrict__ pool, const StackRows r,
                         float *__restrict__ part_o, float *__restrict__ part_ml) {
  extern __shared__ __align__(16) unsigned char smem[];
  __shared__ float s_alpha[MT * 16];
  constexpr int M = MT * 16;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
  const int split = blockIdx.x, splits = gridDim.x, h0 = blockIdx.y * M, b = blockIdx.z;
  const int row = s.row(), pitch = row * 2 + 16, nh = min(M, s.heads - h0);
  const int n = min(r.pos[b] + 1, r.table_stride * r.page_rows);
  const int ntiles = (n + kLaTile - 1) / kLaTile, per = (ntiles + splits - 1) / splits;
  const int ts = split * per, te = min(ntiles, ts + per);
  float *ml = part_ml + (((size_t)b * splits + split) * s.heads + h0) * 2;
  if (ts >= te) {
    if (tid < nh) ml[tid * 2] = -INFINITY, ml[tid * 2 + 1] = 0.f;
    return;
  }
  unsigned char *Ks = smem + (size_t)M * pitch;
  float *Ss = reinterpret_cast<float *>(Ks + (size_t)2 * kLaTile * pitch);
  unsigned char *Ps = reinterpret_cast<unsigned char *>(Ss + M * kLaSPitch);
  const uint32_t qs = (uint32_t)__cvta_generic_to_shared(smem), ks = (uint32_t)__cvta_generic_to_shared(Ks),
                 ps = (uint32_t)__cvta_generic_to_shared(Ps);
  const int *table = r.table + (size_t)r.slot_of[b] * r.table_stride;
  const int units = row / 8;
  for (int u = tid; u < M * units; u += kLaThreads) {
    const int h = u / units, c = u - h * units;  // heads past the last repeat it; their results are not stored
    cp_async16(qs + h * pitch + c * 16, q_abs + ((size_t)b * s.heads + h0 + min(h, nh - 1)) * row + c * 8);
  }
  // a row of the tile belongs to four neighbouring threads: one look into the page table per thread and tile
  constexpr int kRowThreads = kLaThreads / kLaTile;
  const int lk = tid / kRowThreads, lc = tid % kRowThreads;
  auto load_tile = [&](int tile, int buf) {
    const int j = min(tile * kLaTile + lk, n - 1);  // rows past the end repeat the last; they take no weight
    const uint16_t *src = pool + ((size_t)table[j / r.page_rows] * r.page_rows + j % r.page_rows) * row;
    const uint32_t dst = ks + (uint32_t)(buf * kLaTile + lk) * pitch;
#pragma unroll 6
    for (int c = lc; c < units; c += kRowThreads) cp_async16(dst + c * 16, src + c * 8);
  };
  load_tile(ts, 0);
  asm volatile("cp.async.commit_group;" ::: "memory");
  float o[MT][NT][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int i = 0; i < NT; ++i) o[m][i][0] = o[m][i][1] = o[m][i][2] = o[m][i][3] = 0.f;
  // the softmax of a head row belongs to kLaThreads / M consecutive lanes
  constexpr int kPer = kLaThreads / M, kCols = kLaTile / kPer;
  const int sh = tid / kPer, sl = tid % kPer;
  float m_run = -INFINITY, l_run = 0.f;
  const float sl2 = s.scale * 1.4426950408889634f;
  for (int tile = ts; tile < te; ++tile) {
    const int buf = (tile - ts) & 1;
    if (tile + 1 < te) load_tile(tile + 1, buf ^ 1);
    asm volatile("cp.async.commit_group;" ::: "memory");
    asm volatile("cp.async.wait_group 1;" ::: "memory");
    __syncthreads();
    const uint32_t kb = ks + (uint32_t)(buf * kLaTile) * pitch;
    {  // scores of 8 rows per warp
      float sc[MT][4] = {};
      const uint32_t baddr = kb + (uint32_t)(8 * warp + (lane & 7)) * pitch + (lane >> 3) * 16;
#pragma unroll 2
      for (int k0 = 0; k0 < row; k0 += 32) {
        uint32_t b0, b1, b2, b3;
        ldsm4(baddr + k0 * 2, b0, b1, b2, b3);
#pragma unroll
        for (int m = 0; m < MT; ++m) {
          uint32_t a0, a1, a2, a3;
          ldsm4(frag_a(qs, 16 * m, k0, pitch, lane), a0, a1, a2, a3);
          mma_bf16_16816(sc[m], a0, a1, a2, a3, b0, b1);
          ldsm4(frag_a(qs, 16 * m, k0 + 16, pitch, lane), a0, a1, a2, a3);
          mma_bf16_16816(sc[m], a0, a1, a2, a3, b2, b3);
        }
      }
      const int j = tile * kLaTile + 8 * warp + 2 * t;
#pragma unroll
      for (int m = 0; m < MT; ++m) {
        float *d = Ss + (16 * m + g) * kLaSPitch + 8 * warp + 2 * t;
        *reinterpret_cast<float2 *>(d) = make_float2(j < n ? sc[m][0] * sl2 : -INFINITY, j + 1 < n ? sc[m][1] * sl2 : -INFINITY);
        *reinterpret_cast<float2 *>(d + 8 * kLaSPitch) = make_float2(j < n ? sc[m][2] * sl2 : -INFINITY, j + 1 < n ? sc[m][3] * sl2 : -INFINITY);
      }
    }
    __syncthreads();
    {  // online softmax in the log2 domain
      float v[kCols], mx = -INFINITY, sum = 0.f;
#pragma unroll
      for (int i = 0; i < kCols; i += 2) {
        const float2 x = *reinterpret_cast<const float2 *>(Ss + sh * kLaSPitch + sl * kCols + i);
        v[i] = x.x;
        v[i + 1] = x.y;
        mx = fmaxf(mx, fmaxf(x.x, x.y));
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
        for (int p = 0; p < kSplitParts; ++p) *reinterpret_cast<uint32_t *>(Ps + (size_t)(p * M + sh) * kLaPPitch + (sl * kCols + i) * 2) = part[p];
      }
#pragma unroll
      for (int d = 1; d < kPer; d <<= 1) sum += __shfl_xor_sync(0xffffffffu, sum, d);
      l_run = l_run * al + sum;
      if (sl == 0) s_alpha[sh] = al;
    }
    __syncthreads();
    // O += P . C, columns of 8 latents: warp, warp + 8, ... (pairs of tiles share a load)
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
    for (int k0 = 0; k0 < kLaTile; k0 += 16) {
      uint32_t fa[MT][kSplitParts][4];
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int p = 0; p < kSplitParts; ++p)
          ldsm4(frag_a(ps + (uint32_t)(p * M) * kLaPPitch, 16 * m, k0, kLaPPitch, lane), fa[m][p][0], fa[m][p][1], fa[m][p][2], fa[m][p][3]);
#pragma unroll
      for (int i = 0; i < NT; i += 2) {
        const int col = (warp + kLaWarps * (i / 2)) * 16;
        if (col < s.rank) {
          uint32_t b0, b1, b2, b3;
          ldsm4_t(frag_b_t(kb, col, k0, pitch, lane), b0, b1, b2, b3);
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
  float *po = part_o + (((size_t)b * splits + split) * s.heads + h0) * s.rank;
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int i = 0; i < NT; ++i) {
      const int col = (warp + kLaWarps * (i / 2)) * 16 + (i & 1) * 8 + 2 * t, h = 16 * m + g;
      if (col < s.rank) {
        if (h < nh) *reinterpret_cast<float2 *>(po + (size_t)h * s.rank + col) = make_float2(o[m][i][0], o[m][i][1]);
        if (h + 8 < nh) *reinterpret_cast<float2 *>(po + (size_t)(h + 8) * s.rank + col) = make_float2(o[m][i][2], o[m][i][3]);
      }
    }
  if (sl == 0 && sh < nh) {
    ml[sh * 2] = m_run * 0.6931471805599453f;  // natural units, as the merge takes them
    ml[sh * 2 + 1] = l_run;
  }
}

int launch_mla_attend_tc_fine(const uint16_t *q, const uint16_t *pool, long pool_rows, const int *block_table, const int *slot_of, int table_stride,
                              int page_rows, const int *pos, int B, int heads, int splits, float scale, float *part_o, float *part_ml,
                              cudaStream_t stream);

// The tcgen05 core (mla_attend_tc.cu) is built for rows of 512 + 64 values and takes heads 64 at a time; fewer than 24 are
// better off with the kernel above.  BLOK_MLA_ATTEND_IMPL=mma (read at every call) switches it off.
static bool la_fine(const LatentShape &s, int page_rows) {
  const char *impl = getenv("BLOK_MLA_ATTEND_IMPL");
  return s.scale > 0.f && s.rank == 512 && s.rot == 64 && s.heads >= 24 && page_rows % 64 == 0 && !(impl && strcmp(impl, "mma") == 0);
}
static int la_fine_splits(const LatentShape &s, int T, long max_ctx) {
  const int groups = (s.heads + 63) / 64;
  return (int)std::max(1l, std::min((max_ctx + 63) / 64, (long)(sm_count() / (groups * T))));
}
static bool la_tensor(const LatentShape &s) { return s.rank <= kLaMaxRank && la_smem_bytes(s, s.heads > 16 ? 2 : 1) <= 227 * 1024; }
static int la_splits(const LatentShape &s, int T, long max_ctx) {
  const int groups = (s.heads + (s.heads > 16 ? 31 : 15)) / (s.heads > 16 ? 32 : 16);
  const long cap = (max_ctx + 2 * kLaTile - 1) / (2 * kLaTile);  // at least two tiles each
  return (int)std::max(1l, std::min(cap, (long)(sm_count() / (groups * T))));
}

size_t latent_attend_max_parts(const LatentShape &s, int T, long max_ctx) {
  size_t worst = 0;
  for (int t = 1; t <= T; ++t) worst = std::max(worst, (size_t)t * std::max(la_splits(s, t, max_ctx), la_fine_splits(s, t, max_ctx)));
  return worst;
}

template <int MT, int NT>
static int la_launch(const LatentShape &s, const uint16_t *q, const uint16_t *pool, const StackRows &r, int T, int splits, float *po, float *pml,
                     cudaStream_t stream) {
  const size_t smem = la_smem_bytes(s, MT);
  BLOK_CUDA(cudaFuncSetAttribute(latent_attend_kernel<MT, NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  latent_attend_kernel<MT, NT><<<dim3(splits, (s.heads + 16 * MT - 1) / (16 * MT), T), kLaThreads, smem, stream>>>(s, q, pool, r, po, pml);
  return launch_status("latent_attend_kernel");
}

int launch_latent_attend(const LatentShape &s, const void *q_abs, const void *pool, const StackRows &r, int T, long max_ctx, void *o, bool f32,
                         float *part_o, float *part_ml, cudaStream_t stream) {
  if (f32 || !la_tensor(s)) {
    const dim3 grid(s.heads, T);
    const size_t smem = (size_t)(s.row() + s.rank) * sizeof(float);
    BLOK_REQUIRE(smem <= 200 * 1024, BLOK_ERR_SHAPE, "latent attention: a latent of %d values is too wide", s.rank);
    if (f32) {
      if (smem > 40 * 1024) BLOK_CUDA(cudaFuncSetAttribute(latent_attend_simple_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
      latent_attend_simple_kernel<float><<<grid, kLsKeys, smem, stream>>>(s, static_cast<const float *>(q_abs), static_cast<const float *>(pool), r,
                                                                          static_cast<float *>(o));
    } else {
      if (smem > 40 * 1024) BLOK_CUDA(cudaFuncSetAttribute(latent_attend_simple_kernel<uint16_t>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
      latent_attend_simple_kernel<uint16_t><<<grid, kLsKeys, smem, stream>>>(s, static_cast<const uint16_t *>(q_abs), static_cast<const uint16_t *>(pool), r,
                                                                             static_cast<uint16_t *>(o));
    }
    return launch_status("latent_attend_simple_kernel");
  }
  const bool fine = la_fine(s, r.page_rows);
  const int splits = fine ? la_fine_splits(s, T, max_ctx) : la_splits(s, T, max_ctx);
  const uint16_t *q = static_cast<const uint16_t *>(q_abs), *p = static_cast<const uint16_t *>(pool);
  int rc;
#define BLOK_LA(MT)                                                                        \
  rc = s.rank <= 128   ? la_launch<MT, 2>(s, q, p, r, T, splits, part_o, part_ml, stream)  \
       : s.rank <= 256 ? la_launch<MT, 4>(s, q, p, r, T, splits, part_o, part_ml, stream)  \
                       : la_launch<MT, 8>(s, q, p, r, T, splits, part_o, part_ml, stream)
  if (fine)  // a tile never leaves its page: the pool needs no tighter bound than the coordinate range
    rc = launch_mla_attend_tc_fine(q, p, (1l << 31) - 64, r.table, r.slot_of, r.table_stride, r.page_rows, r.pos, T, s.heads, splits, s.scale, part_o,
                                   part_ml, stream);
  else if (s.heads > 16) BLOK_LA(2);
  else BLOK_LA(1);
#undef BLOK_LA
  if (rc) return rc;
  mla_merge_kernel<<<dim3(s.heads, T), 128, (size_t)splits * sizeof(float), stream>>>(part_o, part_ml, splits, s.heads, s.rank, static_cast<uint16_t *>(o));
  return launch_status("mla_merge_kernel");
}

// ---- prompt form ----
__global__ void __launch_bounds__(256) latent_gather_kernel(const LatentShape s, const uint16_t *__restrict__ pool, const StackRows r, int slot, int n,
                                                            uint16_t *__restrict__ c_all, uint16_t *__restrict__ kr_all) {
  const int units = s.row() / 8, cu = s.rank / 8;
  const long total = (long)n * units;
  for (long u = (long)blockIdx.x * blockDim.x + threadIdx.x; u < total; u += (long)gridDim.x * blockDim.x) {
    const int j = (int)(u / units), c = (int)(u - (long)j * units);
    const uint4 v = *reinterpret_cast<const uint4 *>(pool + lt_row(r, slot, j) * s.row() + c * 8);
    uint16_t *d = c < cu ? c_all + (size_t)j * s.rank + c * 8 : kr_all + (size_t)j * s.rot + (c - cu) * 8;
    *reinterpret_cast<uint4 *>(d) = v;
  }
}

int launch_latent_gather(const LatentShape &s, const uint16_t *pool, const StackRows &r, int slot, int n, uint16_t *c_all, uint16_t *kr_all,
                         cudaStream_t stream) {
  const long blocks = ((long)n * (s.row() / 8) + 255) / 256;
  latent_gather_kernel<<<(unsigned)std::min(blocks, 4096l), 256, 0, stream>>>(s, pool, r, slot, n, c_all, kr_all);
  return launch_status("latent_gather_kernel");
}

constexpr int kLpRows = 128, kLpKeys = 64, kLpThreads = 256;

// Zero-filling copy: nothing is read when `ok` is false.
__device__ __forceinline__ void lp_cp(uint32_t dst, const void *src, bool ok) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(ok ? 16u : 0u) : "memory");
}

// grid = (query tiles of 128, heads); a warp owns 16 queries.  DQ >= head(), DV >= vdim: multiples of 32.
template <int DQ, int DV>
__global__ void __launch_bounds__(kLpThreads, 1)
    latent_prompt_kernel(const LatentShape s, const uint16_t *__restrict__ q, const uint16_t *__restrict__ kv, const uint16_t *__restrict__ kr_all,
                         int T, int n, uint16_t *__restrict__ out, int ldo) {
  extern __shared__ __align__(16) unsigned char smem[];
  constexpr int QP = DQ * 2 + 16, VP = DV * 2 + 16;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
  const int h = blockIdx.y, q0 = (gridDim.x - 1 - blockIdx.x) * kLpRows;  // the longest tiles start first
  const int first = n - T, nq = min(kLpRows, T - q0);
  const uint32_t qs = (uint32_t)__cvta_generic_to_shared(smem), ks = qs + kLpRows * QP, vs = ks + 2 * kLpKeys * QP;
  const int ldkv = s.heads * (s.dim + s.vdim);
  for (int u = tid; u < kLpRows * (DQ / 8); u += kLpThreads) {
    const int r = u / (DQ / 8), c = u % (DQ / 8);
    const bool ok = r < nq && c * 8 < s.dim + s.rot;
    lp_cp(qs + r * QP + c * 16, ok ? q + ((size_t)(q0 + r) * s.heads + h) * s.head() + c * 8 : q, ok);
  }
  auto load_tile = [&](int tile, int buf) {
    for (int u = tid; u < kLpKeys * (DQ / 8); u += kLpThreads) {
      const int r = u / (DQ / 8), c = u % (DQ / 8), j = tile * kLpKeys + r;
      const bool ok = j < n && c * 8 < s.dim + s.rot;
      const uint16_t *src = !ok ? kv : c * 8 < s.dim ? kv + (size_t)j * ldkv + h * s.dim + c * 8 : kr_all + (size_t)j * s.rot + (c * 8 - s.dim);
      lp_cp(ks + (buf * kLpKeys + r) * QP + c * 16, src, ok);
    }
    for (int u = tid; u < kLpKeys * (DV / 8); u += kLpThreads) {
      const int r = u / (DV / 8), c = u % (DV / 8), j = tile * kLpKeys + r;
      const bool ok = j < n && c * 8 < s.vdim;
      lp_cp(vs + (buf * kLpKeys + r) * VP + c * 16, ok ? kv + (size_t)j * ldkv + s.heads * s.dim + h * s.vdim + c * 8 : kv, ok);
    }
  };
  const int tiles = (first + q0 + nq + kLpKeys - 1) / kLpKeys;
  load_tile(0, 0);
  asm volatile("cp.async.commit_group;" ::: "memory");
  float o[DV / 8][4];
#pragma unroll
  for (int i = 0; i < DV / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  float m_lo = -INFINITY, m_hi = -INFINITY, l_lo = 0.f, l_hi = 0.f;
  const float sl2 = s.scale * 1.4426950408889634f;
  const int i_lo = first + q0 + 16 * warp + g, i_hi = i_lo + 8;  // positions of the lane's two queries
  const int last_of_warp = first + q0 + 16 * warp + 15;
  for (int tile = 0; tile < tiles; ++tile) {
    const int buf = tile & 1;
    if (tile + 1 < tiles) load_tile(tile + 1, buf ^ 1);
    asm volatile("cp.async.commit_group;" ::: "memory");
    asm volatile("cp.async.wait_group 1;" ::: "memory");
    __syncthreads();
    if (tile * kLpKeys <= last_of_warp) {
      const uint32_t kb = ks + buf * kLpKeys * QP, vb = vs + buf * kLpKeys * VP;
      float sc[kLpKeys / 8][4];
#pragma unroll
      for (int i = 0; i < kLpKeys / 8; ++i) sc[i][0] = sc[i][1] = sc[i][2] = sc[i][3] = 0.f;
#pragma unroll
      for (int k0 = 0; k0 < DQ; k0 += 16) {
        uint32_t a0, a1, a2, a3;
        ldsm4(frag_a(qs, 16 * warp, k0, QP, lane), a0, a1, a2, a3);
#pragma unroll
        for (int i = 0; i < kLpKeys / 8; i += 2) {
          uint32_t b0, b1, b2, b3;
          ldsm4(frag_b(kb, i * 8, k0, QP, lane), b0, b1, b2, b3);
          mma_bf16_16816(sc[i], a0, a1, a2, a3, b0, b1);
          mma_bf16_16816(sc[i + 1], a0, a1, a2, a3, b2, b3);
        }
      }
      float x_lo = -INFINITY, x_hi = -INFINITY;
      const bool edge = tile * kLpKeys + kLpKeys - 1 > first + q0 + 16 * warp;
#pragma unroll
      for (int i = 0; i < kLpKeys / 8; ++i) {
        const int j = tile * kLpKeys + 8 * i + 2 * t;
        sc[i][0] = edge && j > i_lo ? -INFINITY : sc[i][0] * sl2;
        sc[i][1] = edge && j + 1 > i_lo ? -INFINITY : sc[i][1] * sl2;
        sc[i][2] = edge && j > i_hi ? -INFINITY : sc[i][2] * sl2;
        sc[i][3] = edge && j + 1 > i_hi ? -INFINITY : sc[i][3] * sl2;
        x_lo = fmaxf(x_lo, fmaxf(sc[i][0], sc[i][1]));
        x_hi = fmaxf(x_hi, fmaxf(sc[i][2], sc[i][3]));
      }
#pragma unroll
      for (int d = 1; d < 4; d <<= 1) {
        x_lo = fmaxf(x_lo, __shfl_xor_sync(0xffffffffu, x_lo, d));
        x_hi = fmaxf(x_hi, __shfl_xor_sync(0xffffffffu, x_hi, d));
      }
      // tile 0 holds position 0, which every query sees: the maxima are finite from the start
      const float n_lo = fmaxf(m_lo, x_lo), n_hi = fmaxf(m_hi, x_hi);
      const float al = exp2f(m_lo - n_lo), ah = exp2f(m_hi - n_hi);
      m_lo = n_lo;
      m_hi = n_hi;
      l_lo *= al;
      l_hi *= ah;
#pragma unroll
      for (int i = 0; i < DV / 8; ++i) {
        o[i][0] *= al;
        o[i][1] *= al;
        o[i][2] *= ah;
        o[i][3] *= ah;
      }
#pragma unroll
      for (int kk = 0; kk < kLpKeys / 16; ++kk) {
        uint32_t fa[4][kSplitParts];
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const float *v = sc[2 * kk + half];
          const float p0 = exp2f(v[0] - m_lo), p1 = exp2f(v[1] - m_lo), p2 = exp2f(v[2] - m_hi), p3 = exp2f(v[3] - m_hi);
          l_lo += p0 + p1;
          l_hi += p2 + p3;
          split_pair(p0, p1, fa[2 * half]);
          split_pair(p2, p3, fa[2 * half + 1]);
        }
#pragma unroll
        for (int i = 0; i < DV / 8; i += 2) {
          uint32_t b0, b1, b2, b3;
          ldsm4_t(frag_b_t(vb, i * 8, kk * 16, VP, lane), b0, b1, b2, b3);
#pragma unroll
          for (int p = 0; p < kSplitParts; ++p) {
            mma_bf16_16816(o[i], fa[0][p], fa[1][p], fa[2][p], fa[3][p], b0, b1);
            mma_bf16_16816(o[i + 1], fa[0][p], fa[1][p], fa[2][p], fa[3][p], b2, b3);
          }
        }
      }
    }
    __syncthreads();
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
#pragma unroll
  for (int d = 1; d < 4; d <<= 1) {
    l_lo += __shfl_xor_sync(0xffffffffu, l_lo, d);
    l_hi += __shfl_xor_sync(0xffffffffu, l_hi, d);
  }
  const float r_lo = 1.0f / l_lo, r_hi = 1.0f / l_hi;
  const int row_lo = 16 * warp + g;
  uint16_t *po = out + (size_t)(q0 + row_lo) * ldo + h * s.vdim;
#pragma unroll
  for (int i = 0; i < DV / 8; ++i) {
    const int col = 8 * i + 2 * t;
    if (col < s.vdim) {
      if (row_lo < nq) *reinterpret_cast<uint32_t *>(po + col) = pack_bf16x2(o[i][0] * r_lo, o[i][1] * r_lo);
      if (row_lo + 8 < nq) *reinterpret_cast<uint32_t *>(po + (size_t)8 * ldo + col) = pack_bf16x2(o[i][2] * r_hi, o[i][3] * r_hi);
    }
  }
}

bool latent_prompt_tc_supports(const LatentShape &s);
int launch_latent_prompt_tc(const LatentShape &s, const uint16_t *q, const uint16_t *kv, const uint16_t *kr_all, int T, int n, uint16_t *o, int ldo,
                            cudaStream_t stream);

bool latent_prompt_supports(const LatentShape &s) { return s.head() <= 256 && s.vdim <= 256; }

template <int DQ, int DV>
static int lp_launch(const LatentShape &s, const uint16_t *q, const uint16_t *kv, const uint16_t *kr_all, int T, int n, uint16_t *o, int ldo,
                     cudaStream_t stream) {
  constexpr int smem = (kLpRows + 2 * kLpKeys) * (DQ * 2 + 16) + 2 * kLpKeys * (DV * 2 + 16);
  BLOK_CUDA(cudaFuncSetAttribute(latent_prompt_kernel<DQ, DV>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
  latent_prompt_kernel<DQ, DV><<<dim3((T + kLpRows - 1) / kLpRows, s.heads), kLpThreads, smem, stream>>>(s, q, kv, kr_all, T, n, o, ldo);
  return launch_status("latent_prompt_kernel");
}

int launch_latent_prompt(const LatentShape &s, const uint16_t *q, const uint16_t *kv, const uint16_t *kr_all, int T, int n, uint16_t *o, int ldo,
                         cudaStream_t stream) {
  BLOK_REQUIRE(latent_prompt_supports(s) && n >= T && T >= 1, BLOK_ERR_SHAPE, "latent attention: heads of %d / %d", s.head(), s.vdim);
  const char *impl = getenv("BLOK_MLA_ATTEND_IMPL");
  if (latent_prompt_tc_supports(s) && !(impl && strcmp(impl, "mma") == 0)) return launch_latent_prompt_tc(s, q, kv, kr_all, T, n, o, ldo, stream);
  if (s.head() <= 96 && s.vdim <= 64) return lp_launch<96, 64>(s, q, kv, kr_all, T, n, o, ldo, stream);
  if (s.head() <= 128 && s.vdim <= 128) return lp_launch<128, 128>(s, q, kv, kr_all, T, n, o, ldo, stream);
  if (s.head() <= 192 && s.vdim <= 128) return lp_launch<192, 128>(s, q, kv, kr_all, T, n, o, ldo, stream);
  return lp_launch<256, 256>(s, q, kv, kr_all, T, n, o, ldo, stream);
}

}  // namespace blok
