// Softmax attention of a prompt on tcgen05: causal attention of T queries over n keys and values, for the prompt form of latent
// attention (per-head keys and values, latent_attn.cu) and for grouped attention over cached pages (grouped_attn.cu).  Query-key
// sizes up to 256 and value sizes up to 128.
//
// A CTA owns 128 queries of one head and walks the keys in tiles of 64:
//   S [queries x 64]   = Q K^T    both operands in shared memory (TMA, 128-byte swizzle), accumulator in tensor memory, two
//                                 buffers
//   P = exp2(S * scale * log2 e + bias - m)   two threads per query, 32 keys each; they exchange their maxima.  A bias depends on
//                                 the distance alone: a warp's 32 queries meet 32 keys at 63 distances, which the warp puts
//                                 into shared memory with the causal mask in them
//   O [queries x vdim] += P V     P in tensor memory as the A operand, in three bf16 parts (bf16_split.cuh); V is read from
//                                 its rows as they are (MN-major B operand)
// The scores of tile n + 1 are computed under the softmax of tile n.  The running maximum is kept lazily: a row's reference
// moves, and its 64 or 128 accumulators are rescaled, only when a tile's maximum exceeds it by more than 40 natural units.
//
// Warps: 0..7 softmax (a warp reaches the 32 lanes of tensor memory of its index mod 4: warps w and w + 4 share 32 queries; two
// warps per scheduler hide each other's latencies), 8: copies, 9: MMA.  Every wait is bounded; a CTA that
// gives up records it, waits for its copies in flight, releases its tensor memory and returns.  No copy is multicast.
#include <algorithm>

#include "bf16_split.cuh"
#include "gemm_tma.h"
#include "prompt_attn_tc.h"
#include "stack_kernels.h"
#include "tc_pipe.cuh"

namespace blok {

constexpr int kPtRows = 128, kPtKeys = 64, kPtMaxStages = 6, kPtThreads = 320;
constexpr int kPtQChunk = kPtRows * 128, kPtKChunk = kPtKeys * 128;  // bytes of a 64-column chunk
constexpr int kPtMaxQ = 4;                                           // chunks of a query
constexpr int kPtMaxSmem = 220 * 1024;
constexpr int kPtColS = 0, kPtColP = 128, kPtColO = 384;             // tensor memory: S 2 x 64, P 2 x 3 x 32 (of 4 x 64), O
constexpr int kPtTmemCols = 512;
constexpr float kPtLog2e = 1.4426950408889634f;
constexpr float kPtLazy = 57.7f;  // 40 natural units in the log2 domain

__device__ unsigned g_prompt_attn_error = 0;

__device__ __forceinline__ float pt_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// BIAS: scores take a bias by distance.
template <bool BIAS>
__global__ void __launch_bounds__(kPtThreads, 1)
    prompt_attn_tc_kernel(const __grid_constant__ CUtensorMap mq, const __grid_constant__ CUtensorMap mkv, const __grid_constant__ CUtensorMap mkr,
                          const PromptAttn a) {
  extern __shared__ unsigned char smem_raw[];
  __shared__ __align__(8) unsigned long long s_bar[2 * kPtMaxStages + 13];
  __shared__ uint32_t s_tmem;
  __shared__ float s_window[BIAS ? 8 : 1][BIAS ? 64 : 1];
  __shared__ float s_pair[2][2][kPtRows];  // maxima (at the end: sums) of the two halves of a tile
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int h = blockIdx.y, q0 = (gridDim.x - 1 - blockIdx.x) * kPtRows;  // the longest rows of tiles start first
  const int first = a.n - a.T, nq = min(kPtRows, a.T - q0);
  const int nt = (first + q0 + nq + kPtKeys - 1) / kPtKeys;
  const int qc = (a.dim + 63) / 64, vc = (a.vdim + 63) / 64, kh = h / a.share;
  const uint32_t sQ = ((uint32_t)__cvta_generic_to_shared(smem_raw) + 1023u) & ~1023u;
  const uint32_t stage_bytes = (uint32_t)(qc + vc) * kPtKChunk, sT = sQ + (uint32_t)qc * kPtQChunk;
  const uint32_t bar = (uint32_t)__cvta_generic_to_shared(&s_bar[0]);
  const uint32_t full = bar, empty = bar + 8 * kPtMaxStages, qfull = bar + 16 * kPtMaxStages, sfull = qfull + 8, sfree = qfull + 24, pfull = qfull + 40,
                 pdone = qfull + 56, paired = qfull + 72;
  if (tid == 0) {
    for (int s = 0; s < a.stages; ++s) {
      tp_mbar_init(full + 8 * s, 1);
      tp_mbar_init(empty + 8 * s, 1);
    }
    tp_mbar_init(qfull, 1);
    for (int b = 0; b < 2; ++b) {
      tp_mbar_init(sfull + 8 * b, 1);
      tp_mbar_init(sfree + 8 * b, 8);
      tp_mbar_init(pfull + 8 * b, 8);
      tp_mbar_init(pdone + 8 * b, 1);
    }
    for (int w = 0; w < 4; ++w) tp_mbar_init(paired + 8 * w, 2);
    tp_mbar_init_fence();
  }
  if (warp == 0) tp_tmem_alloc((uint32_t)__cvta_generic_to_shared(&s_tmem), kPtTmemCols);
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = s_tmem;
  bool failed = false;

  if (warp == 8) {
    if (lane == 0) {
      tp_expect_tx(qfull, (uint32_t)qc * kPtQChunk);
      for (int c = 0; c < qc; ++c) tp_load_2d(sQ + c * kPtQChunk, &mq, h * a.q_head + 64 * c, q0, qfull);
      // the row of key j: its page's, or j itself.  A box past the last key repeats the tile's first; its keys take no weight.
      auto row_of = [&](int j) { return a.table ? a.table[j / a.page_rows] * a.page_rows + j % a.page_rows : j; };
      int next[2] = {row_of(0), a.box < kPtKeys ? row_of(a.box < a.n ? a.box : 0) : 0};
      int issued = 0, s = 0;
      uint32_t turn = 1;  // of the stage's last release; the first turn needs none
      for (int n = 0; n < nt; ++n) {
        const int row[2] = {next[0], next[1]};
        if (n + 1 < nt) {
          const int j = (n + 1) * kPtKeys;
          next[0] = row_of(j);
          if (a.box < kPtKeys) next[1] = row_of(j + a.box < a.n ? j + a.box : j);
        }
        if (n >= a.stages && !tp_wait(empty + 8 * s, turn)) {
          failed = true;
          break;
        }
        const uint32_t dst = sT + (uint32_t)s * stage_bytes, f = full + 8 * s;
        tp_expect_tx(f, stage_bytes);
        for (int p = 0; p * a.box < kPtKeys; ++p) {
          const uint32_t to = dst + p * a.box * 128;
          for (int c = 0; c < a.key_chunks; ++c) tp_load_2d(to + c * kPtKChunk, &mkv, kh * a.k_head + 64 * c, row[p], f);
          for (int c = a.key_chunks; c < qc; ++c) tp_load_2d(to + c * kPtKChunk, &mkr, 64 * (c - a.key_chunks), row[p], f);
          for (int c = 0; c < vc; ++c) tp_load_2d(to + (qc + c) * kPtKChunk, &mkv, a.v_first + kh * a.vdim + 64 * c, row[p], f);
        }
        issued = n + 1;
        if (++s == a.stages) s = 0, turn ^= 1;
      }
      // no copy may be in flight when the CTA leaves
      tp_wait(qfull, 0);
      for (int n = max(0, issued - a.stages); n < issued; ++n) tp_wait(full + 8 * (n % a.stages), (uint32_t)((n / a.stages) & 1));
    }
  } else if (warp == 9) {
    // The whole warp walks the tiles, so that addresses and descriptors stay warp-uniform; one lane issues.
    const bool issues = tp_elect();
    auto ready = [](uint32_t mbar, uint32_t parity) { return __all_sync(0xffffffffu, tp_wait(mbar, parity)) != 0; };
    // V: MN-major B operand; columns past the value size hold whatever the copy brought and are not stored
    const uint32_t idesc_s = tp_idesc_bf16(kPtKeys), idesc_pv = tp_idesc_bf16(64 * vc) | (1u << 16);
    const uint64_t qd = tp_desc_k_sw128(sQ);
    auto issue_s = [&](int n, int stage) {
      const uint64_t kd = tp_desc_k_sw128(sT + (uint32_t)stage * stage_bytes);
      const uint32_t to = tmem + kPtColS + 64 * (n & 1);
      if (issues) {
#pragma unroll
        for (int c = 0; c < kPtMaxQ; ++c) {
          if (c < qc) {
#pragma unroll
            for (int j = 0; j < 4; ++j)
              if (64 * c + 16 * j < a.dim)
                tp_mma(to, qd + (uint64_t)(c * (kPtQChunk >> 4) + 2 * j), kd + (uint64_t)(c * (kPtKChunk >> 4) + 2 * j), idesc_s, (c | j) ? 1u : 0u);
          }
        }
        tp_commit(sfull + 8 * (n & 1));
      }
    };
    failed = !ready(qfull, 0) || !ready(full, 0);
    if (!failed) {
      tc_fence_after();
      issue_s(0, 0);
    }
    int stage = 0;  // of tile n
    uint32_t turn = 0;
    for (int n = 0; n < nt && !failed; ++n) {
      const int b = n & 1, ahead = stage + 1 == a.stages ? 0 : stage + 1;
      const uint32_t ahead_turn = turn ^ (ahead == 0 ? 1u : 0u);
      if (n + 1 < nt) {
        const int m = n + 1;
        if (!ready(full + 8 * ahead, ahead_turn) || (m >= 2 && !ready(sfree + 8 * (m & 1), (uint32_t)(((m >> 1) - 1) & 1)))) {
          failed = true;
          break;
        }
        tc_fence_after();
        issue_s(m, ahead);
      }
      if (!ready(pfull + 8 * b, (uint32_t)((n >> 1) & 1))) {
        failed = true;
        break;
      }
      tc_fence_after();
      const uint64_t vd = tp_desc_mn_sw128(sT + (uint32_t)stage * stage_bytes + qc * kPtKChunk, kPtKChunk);
      if (issues) {
#pragma unroll
        for (int p = 0; p < kSplitParts; ++p)
#pragma unroll
          for (int j = 0; j < kPtKeys / 16; ++j)
            tp_mma_ts(tmem + kPtColO, tmem + kPtColP + 128 * b + 32 * p + 8 * j, vd + (uint64_t)(j * (2048 >> 4)), idesc_pv, (n | p | j) ? 1u : 0u);
        tp_commit(empty + 8 * stage);
        tp_commit(pdone + 8 * b);
      }
      stage = ahead;
      turn = ahead_turn;
    }
  } else {
    const int quad = warp & 3, half = warp >> 2, row = 32 * quad + lane;
    const uint32_t lanes = (uint32_t)(32 * quad) << 16;
    const int pos = first + q0 + row;        // this thread's query
    const int warp_first = first + q0 + 32 * quad;
    // the values both threads of a query have put into s_pair[parity]; false when the other did not come
    auto exchange = [&](int parity, float v, float *other) {
      s_pair[parity][half][row] = v;
      __syncwarp();
      if (lane == 0) tp_arrive(paired + 8 * quad);
      const bool ok = tp_wait(paired + 8 * quad, (uint32_t)parity);
      *other = s_pair[parity][half ^ 1][row];
      return ok;
    };
    float m_ref = 0.f, l = 0.f;
    const float *bias = BIAS ? a.bias + (size_t)h * a.bias_len : nullptr;
    for (int n = 0; n < nt; ++n) {
      const int b = n & 1, key0 = n * kPtKeys + 32 * half;  // the thread's first key
      // entry i: distance near + i, lane l's key j at i = l + 31 - j
      const int near = warp_first - key0 - 31;
      if (BIAS) {
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          const int d = near + lane + 32 * i;
          s_window[warp][lane + 32 * i] = d < 0 ? -INFINITY : bias[min(d, a.bias_len - 1)] * kPtLog2e;
        }
        __syncwarp();
      }
      failed = !tp_wait(sfull + 8 * b, (uint32_t)((n >> 1) & 1));
      if (__any_sync(0xffffffffu, failed)) {
        failed = true;
        break;
      }
      tc_fence_after();
      uint32_t r[32];
      tmem_ld32(tmem + lanes + kPtColS + 64 * b + 32 * half, r);
      tmem_wait_ld();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) tp_arrive(sfree + 8 * b);
      if (BIAS) {
        const float *w = s_window[warp] + lane + 31;
#pragma unroll
        for (int j = 0; j < 32; ++j) r[j] = __float_as_uint(fmaf(__uint_as_float(r[j]), a.scale_log2, w[-j]));
      } else if (key0 + 31 > warp_first) {  // keys behind a query take no weight
#pragma unroll
        for (int j = 0; j < 32; ++j)
          if (key0 + j > pos) r[j] = 0xff800000u;
      }
      float x0 = -INFINITY, x1 = -INFINITY, x2 = -INFINITY, x3 = -INFINITY;
#pragma unroll
      for (int j = 0; j < 32; j += 4) {
        x0 = fmaxf(x0, __uint_as_float(r[j]));
        x1 = fmaxf(x1, __uint_as_float(r[j + 1]));
        x2 = fmaxf(x2, __uint_as_float(r[j + 2]));
        x3 = fmaxf(x3, __uint_as_float(r[j + 3]));
      }
      float mx = fmaxf(fmaxf(x0, x1), fmaxf(x2, x3)) * (BIAS ? 1.f : a.scale_log2), other;  // without a bias the scale is positive
      failed = !exchange(b, mx, &other);
      mx = fmaxf(mx, other);
      float alpha = 1.f;
      bool need = false;
      if (n == 0) {
        m_ref = mx;  // position 0 is in this tile and every query sees it
      } else if (mx > m_ref + kPtLazy) {
        alpha = pt_ex2(m_ref - mx);
        m_ref = mx;
        need = true;
      }
      const float nm = -m_ref;
      float s0 = 0.f, s1 = 0.f;
#pragma unroll
      for (int j = 0; j < 32; j += 2) {
        const float u = __uint_as_float(r[j]), v = __uint_as_float(r[j + 1]);
        const float p0 = pt_ex2(BIAS ? u + nm : fmaf(u, a.scale_log2, nm)), p1 = pt_ex2(BIAS ? v + nm : fmaf(v, a.scale_log2, nm));
        s0 += p0;
        s1 += p1;
        r[j] = __float_as_uint(p0);
        r[j + 1] = __float_as_uint(p1);
      }
      l = l * alpha + (s0 + s1);
      if (n >= 2) failed = failed || !tp_wait(pdone + 8 * b, (uint32_t)(((n >> 1) - 1) & 1));  // the products of tile n - 2 have read this buffer
      if (__any_sync(0xffffffffu, need) && n >= 1) failed = failed || !tp_wait(pdone + 8 * (b ^ 1), (uint32_t)(((n - 1) >> 1) & 1));
      if (__any_sync(0xffffffffu, failed)) {
        failed = true;
        break;
      }
      tc_fence_after();
      if (__any_sync(0xffffffffu, need)) {  // the two threads of a query take turns with its columns, 32 at a time
#pragma unroll 1
        for (int c = half; c < 2 * vc; c += 2) {
          uint32_t o[32];
          tmem_ld32(tmem + lanes + kPtColO + 32 * c, o);
          tmem_wait_ld();
#pragma unroll
          for (int j = 0; j < 32; ++j) o[j] = __float_as_uint(__uint_as_float(o[j]) * alpha);
          tmem_st32(tmem + lanes + kPtColO + 32 * c, o);
        }
      }
#pragma unroll
      for (int p = 0; p < kSplitParts; ++p) {
        uint32_t w[16];
#pragma unroll
        for (int j = 0; j < 16; ++j) {
          const float u = __uint_as_float(r[2 * j]), v = __uint_as_float(r[2 * j + 1]);
          w[j] = pack_pair(u, v);
          r[2 * j] = __float_as_uint(u - bf16lo(w[j]));
          r[2 * j + 1] = __float_as_uint(v - bf16hi(w[j]));
        }
        tmem_st16(tmem + lanes + kPtColP + 128 * b + 32 * p + 16 * half, w);
      }
      tmem_wait_st();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) tp_arrive(pfull + 8 * b);
    }
    if (!failed) {
      float other;
      failed = !exchange(nt & 1, l, &other);
      l += other;
    }
    if (!failed) failed = !tp_wait(pdone + 8 * ((nt - 1) & 1), (uint32_t)(((nt - 1) >> 1) & 1));
    failed = __any_sync(0xffffffffu, failed);
    if (!failed) {
      tc_fence_after();
      const bool in = row < nq;
      float inv = 1.0f / l;
      if (a.gate && in) inv /= 1.0f + expf(-bf16_bits_to_f32(a.gate[(size_t)(q0 + row) * a.ld_gate + h]));
      uint16_t *o = a.out + (size_t)(q0 + row) * a.ldo + (size_t)h * a.vdim;
#pragma unroll 1
      for (int c = half; c < 2 * vc; c += 2) {
        uint32_t v[32];
        tmem_ld32(tmem + lanes + kPtColO + 32 * c, v);
        tmem_wait_ld();
        if (in) {
#pragma unroll
          for (int j = 0; j < 32; j += 8) {
            if (32 * c + j >= a.vdim) break;
            uint32_t w[4];
#pragma unroll
            for (int k = 0; k < 4; ++k) w[k] = pack_bf16x2(__uint_as_float(v[j + 2 * k]) * inv, __uint_as_float(v[j + 2 * k + 1]) * inv);
            *reinterpret_cast<uint4 *>(o + 32 * c + j) = make_uint4(w[0], w[1], w[2], w[3]);
          }
        }
      }
    }
  }
  if (failed) atomicExch(&g_prompt_attn_error, 1u);
  tc_fence_before();
  __syncthreads();
  if (warp == 0) tp_tmem_free(tmem, kPtTmemCols);
}

bool prompt_attn_supports(int dim, int vdim) { return dim % 16 == 0 && dim <= 64 * kPtMaxQ && vdim % 16 == 0 && vdim <= 128; }

int launch_prompt_attn(const CUtensorMap &mq, const CUtensorMap &mkv, const CUtensorMap &mkr, PromptAttn a, cudaStream_t stream) {
  BLOK_REQUIRE(prompt_attn_supports(a.dim, a.vdim) && a.ldo % 8 == 0 && a.T >= 1 && a.n >= a.T && a.heads % a.share == 0, BLOK_ERR_SHAPE,
               "prompt attention: heads of %d / %d, rows of %d outputs", a.dim, a.vdim, a.ldo);
  const int qc = (a.dim + 63) / 64, vc = (a.vdim + 63) / 64, stage_bytes = (qc + vc) * kPtKChunk;
  a.stages = std::min(kPtMaxStages, (kPtMaxSmem - 1024 - qc * kPtQChunk) / stage_bytes);
  const int smem = qc * kPtQChunk + a.stages * stage_bytes + 1024;
  const dim3 grid((a.T + kPtRows - 1) / kPtRows, a.heads);
  if (a.bias) {
    BLOK_CUDA(cudaFuncSetAttribute(prompt_attn_tc_kernel<true>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
    prompt_attn_tc_kernel<true><<<grid, kPtThreads, smem, stream>>>(mq, mkv, mkr, a);
  } else {
    BLOK_CUDA(cudaFuncSetAttribute(prompt_attn_tc_kernel<false>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
    prompt_attn_tc_kernel<false><<<grid, kPtThreads, smem, stream>>>(mq, mkv, mkr, a);
  }
  return launch_status("prompt_attn_tc_kernel");
}

bool latent_prompt_tc_supports(const LatentShape &s) {
  return s.scale > 0.f && s.dim % 64 == 0 && s.rot % 64 == 0 && s.head() <= 64 * kPtMaxQ && (s.vdim == 64 || s.vdim == 128);
}

int launch_latent_prompt_tc(const LatentShape &s, const uint16_t *q, const uint16_t *kv, const uint16_t *kr_all, int T, int n, uint16_t *o, int ldo,
                            cudaStream_t stream) {
  CUtensorMap mq, mkv, mkr;
  const int qw = s.heads * s.head(), kw = s.heads * (s.dim + s.vdim);
  int rc;
  // rows past the last query and key read as zeros
  if ((rc = gemm_operand_map(q, T, qw, qw, kPtRows, &mq)) || (rc = gemm_operand_map(kv, n, kw, kw, kPtKeys, &mkv)) ||
      (rc = gemm_operand_map(kr_all, n, s.rot, s.rot, kPtKeys, &mkr)))
    return rc;
  PromptAttn a;
  a.out = o;
  a.ldo = ldo;
  a.T = T;
  a.n = n;
  a.heads = s.heads;
  a.q_head = a.dim = s.head();
  a.k_head = s.dim;
  a.key_chunks = s.dim / 64;
  a.v_first = s.heads * s.dim;
  a.vdim = s.vdim;
  a.scale_log2 = s.scale * kPtLog2e;
  return launch_prompt_attn(mq, mkv, mkr, a, stream);
}

bool grouped_prompt_supports(const GroupedShape &s) { return (s.bias || s.scale > 0.f) && prompt_attn_supports(s.dim, s.vdim); }

int launch_grouped_prompt(const GroupedShape &s, const GroupedQuery<uint16_t> &g, const void *pool, long pool_rows, const StackRows &r, int slot, int T,
                          int n, cudaStream_t stream) {
  BLOK_REQUIRE(g.ldq % 8 == 0 && r.page_rows % 32 == 0, BLOK_ERR_SHAPE, "prompt attention: rows of %d values, pages of %d", g.ldq, r.page_rows);
  CUtensorMap mq, mkv;
  const int box = r.page_rows % kPtKeys ? 32 : kPtKeys;  // a box stays inside a page
  int rc;
  if ((rc = gemm_operand_map(g.q, T, s.heads * s.dim, g.ldq, kPtRows, &mq)) || (rc = gemm_operand_map(pool, pool_rows, s.row(), s.row(), box, &mkv))) return rc;
  PromptAttn a;
  a.out = g.out;
  a.ldo = g.ldo;
  a.gate = g.gate;
  a.ld_gate = g.ld_gate;
  a.T = T;
  a.n = n;
  a.heads = s.heads;
  a.share = s.heads / s.kv_heads;
  a.q_head = a.k_head = a.dim = s.dim;
  a.key_chunks = (s.dim + 63) / 64;
  a.v_first = s.kv_heads * s.dim;
  a.vdim = s.vdim;
  a.scale_log2 = s.scale * kPtLog2e;
  a.bias = s.bias;
  a.bias_len = s.bias_len;
  a.table = r.table + (size_t)slot * r.table_stride;
  a.page_rows = r.page_rows;
  a.box = box;
  return launch_prompt_attn(mq, mkv, mkv, a, stream);
}

// *out becomes non-zero if a CTA has given up on a barrier since the last call (the flag is cleared).
int prompt_attn_take_error(unsigned *out) {
  unsigned zero = 0;
  BLOK_CUDA(cudaMemcpyFromSymbol(out, g_prompt_attn_error, sizeof(unsigned)));
  if (*out) BLOK_CUDA(cudaMemcpyToSymbol(g_prompt_attn_error, &zero, sizeof(unsigned)));
  return BLOK_OK;
}

}  // namespace blok
