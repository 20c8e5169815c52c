// bf16 GEMM of a prompt chunk (or of a step of many sequences) on the 5th-generation tensor cores, plain or grouped by
// expert: out[t, r] = act(sum_k x[t, k] W[r, k]).
//
// One CTA = 128 rows of x times BN weight rows.  A producer warp brings 64-column slices of both operands into shared
// memory by TMA (128-byte swizzle, no multicast), kStages of them in flight; one lane of the MMA warp issues four
// tcgen05.mma M128 N(BN) K16 per slice with the accumulator in tensor memory; four epilogue warps read it back (a thread
// owns one row of x), apply the activation and store.  Rows and columns past the matrices' ends are filled with zeros by
// the copies and masked at the store, so any T, R and K work.  The grouped form takes its tiles from a device table whose
// length the host does not know: the grid covers the worst case and surplus CTAs leave at once.
//
// Every mbarrier wait is bounded.  A CTA that gives up records it, waits for its own copies in flight, releases its
// tensor memory and returns.
#include <mutex>

#include "gemm_tma.h"
#include "tc_pipe.cuh"

namespace blok {

constexpr int kGtThreads = 192;  // warps 0..3: epilogue, 4: copies, 5: MMA
constexpr int kGtKStep = 64;

template <int BN>
struct GtCfg {
  static constexpr int kStages = BN == 128 ? 3 : 2;  // 96 KB: two CTAs per SM, one computes while the other stores
  static constexpr int kABytes = kGtTileRows * 128, kBBytes = BN * 128;
  static constexpr int kStageBytes = kABytes + kBBytes;
  static constexpr int kSmem = kStages * kStageBytes + 1024;  // + 1,024: the slices start on a 1,024-byte boundary
};

__device__ unsigned g_gemm_tma_error = 0;

struct GtArgs {
  void *out;
  const int *tile_expert, *tile_start, *tile_count, *num_tiles;
  int T, R, K, ldo, act_cols, up_row;
};

template <int ACT>
__device__ __forceinline__ float gt_act(float v) {
  if (ACT == GEMM_ACT_RELU2) {
    v = fmaxf(v, 0.f);
    return v * v;
  }
  if (ACT == GEMM_ACT_SILU) return __fdividef(v, 1.0f + __expf(-v));  // the result is rounded to bf16
  return v;
}

template <int BN, int ACT, bool F32>
__global__ void __launch_bounds__(kGtThreads)
    gemm_tma_kernel(const __grid_constant__ CUtensorMap mx, const __grid_constant__ CUtensorMap mw, const GtArgs a) {
  using Cfg = GtCfg<BN>;
  constexpr int S = Cfg::kStages;
  // a pair of 128-row boxes, gate and up, makes 128 output columns
  constexpr int kCols = ACT == GEMM_ACT_SWIGLU ? BN / 2 : BN;
  extern __shared__ unsigned char smem_raw[];
  __shared__ __align__(8) unsigned long long s_bar[2 * S + 1];
  __shared__ uint32_t s_tmem;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  int row0, count, wrow = blockIdx.x * kCols;
  if (a.tile_start) {
    if ((int)blockIdx.y >= *a.num_tiles) return;
    row0 = a.tile_start[blockIdx.y];
    count = a.tile_count[blockIdx.y];
    wrow += a.tile_expert[blockIdx.y] * a.R;
  } else {
    row0 = blockIdx.y * kGtTileRows;
    count = min(kGtTileRows, a.T - row0);
  }
  const uint32_t sbase = ((uint32_t)__cvta_generic_to_shared(smem_raw) + 1023u) & ~1023u;
  const uint32_t bar = (uint32_t)__cvta_generic_to_shared(&s_bar[0]);
  const uint32_t full = bar, empty = bar + 8 * S, done = bar + 16 * S;
  if (tid == 0) {
#pragma unroll
    for (int s = 0; s < S; ++s) {
      tp_mbar_init(full + 8 * s, 1);
      tp_mbar_init(empty + 8 * s, 1);
    }
    tp_mbar_init(done, 1);
    tp_mbar_init_fence();
  }
  if (warp == 0) tp_tmem_alloc((uint32_t)__cvta_generic_to_shared(&s_tmem), BN);
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = s_tmem;
  const int nsteps = (a.K + kGtKStep - 1) / kGtKStep;
  bool failed = false;

  if (warp == 4) {
    if (lane == 0) {
      int issued = 0;
      for (int c = 0; c < nsteps; ++c) {
        const int s = c % S;
        if (c >= S && !tp_wait(empty + 8 * s, (uint32_t)((c / S - 1) & 1))) {
          failed = true;
          break;
        }
        const uint32_t dst = sbase + (uint32_t)s * Cfg::kStageBytes;
        tp_expect_tx(full + 8 * s, Cfg::kStageBytes);
        tp_load_2d(dst, &mx, c * kGtKStep, row0, full + 8 * s);
        tp_load_2d(dst + Cfg::kABytes, &mw, c * kGtKStep, wrow, full + 8 * s);
        if (ACT == GEMM_ACT_SWIGLU) tp_load_2d(dst + Cfg::kABytes + kCols * 128, &mw, c * kGtKStep, a.up_row + wrow, full + 8 * s);
        issued = c + 1;
      }
      // no copy may be in flight when the CTA leaves; the MMA lane has seen all of them unless a wait gave up
      for (int c = max(0, issued - S); c < issued; ++c) tp_wait(full + 8 * (c % S), (uint32_t)((c / S) & 1));
    }
  } else if (warp == 5) {
    // the whole warp walks the slices, so that addresses and descriptors stay warp-uniform; one lane issues
    const bool issues = tp_elect();
    int s = 0;
    uint32_t turn = 0;
    for (int c = 0; c < nsteps; ++c) {
      if (!__all_sync(0xffffffffu, tp_wait(full + 8 * s, turn))) {
        failed = true;
        break;
      }
      tc_fence_after();
      const uint64_t ad = tp_desc_k_sw128(sbase + (uint32_t)s * Cfg::kStageBytes);
      const uint64_t bd = tp_desc_k_sw128(sbase + (uint32_t)s * Cfg::kStageBytes + Cfg::kABytes);
      if (issues) {
#pragma unroll
        for (int k = 0; k < kGtKStep / 16; ++k)
          tp_mma(tmem, ad + (uint64_t)(2 * k), bd + (uint64_t)(2 * k), tp_idesc_bf16(BN), (c | k) ? 1u : 0u);
        tp_commit(empty + 8 * s);
        if (c == nsteps - 1) tp_commit(done);
      }
      if (++s == S) s = 0, turn ^= 1;
    }
  } else {
    failed = !tp_wait(done, 0);
    failed = __any_sync(0xffffffffu, failed);
    if (!failed) {
      tc_fence_after();
      const int r = 32 * warp + lane;
      const size_t o = (size_t)(row0 + r) * a.ldo;
      const int n0 = blockIdx.x * kCols;
      if constexpr (ACT == GEMM_ACT_SWIGLU) {
#pragma unroll 1
        for (int c0 = 0; c0 < kCols; c0 += 16) {
          if (n0 + c0 >= a.R) break;
          uint32_t gate[16], up[16];
          const uint32_t at = tmem + ((uint32_t)(32 * warp) << 16) + c0;
          tmem_ld16(at, gate);
          tmem_ld16(at + kCols, up);
          tmem_wait_ld();
          if (r < count) {
#pragma unroll
            for (int j = 0; j < 16; j += 4) {
              const int col = n0 + c0 + j;
              if (col < a.R) {
                float f[4];
#pragma unroll
                for (int i = 0; i < 4; ++i) f[i] = gt_act<GEMM_ACT_SILU>(__uint_as_float(gate[j + i])) * __uint_as_float(up[j + i]);
                *reinterpret_cast<uint2 *>(static_cast<uint16_t *>(a.out) + o + col) = make_uint2(pack_bf16x2(f[0], f[1]), pack_bf16x2(f[2], f[3]));
              }
            }
          }
        }
      } else {
#pragma unroll 1
        for (int c0 = 0; c0 < BN; c0 += 32) {
          if (n0 + c0 >= a.R) break;
          uint32_t v[32];
          tmem_ld32(tmem + ((uint32_t)(32 * warp) << 16) + c0, v);
          tmem_wait_ld();
          if (r < count) {
#pragma unroll
            for (int j = 0; j < 32; j += 4) {
              const int col = n0 + c0 + j;
              if (col < a.R) {  // R is a multiple of 4
                float f0 = __uint_as_float(v[j]), f1 = __uint_as_float(v[j + 1]), f2 = __uint_as_float(v[j + 2]), f3 = __uint_as_float(v[j + 3]);
                if (ACT != GEMM_ACT_SILU || col < a.act_cols) f0 = gt_act<ACT>(f0), f1 = gt_act<ACT>(f1), f2 = gt_act<ACT>(f2), f3 = gt_act<ACT>(f3);
                if (F32) *reinterpret_cast<float4 *>(static_cast<float *>(a.out) + o + col) = make_float4(f0, f1, f2, f3);
                else *reinterpret_cast<uint2 *>(static_cast<uint16_t *>(a.out) + o + col) = make_uint2(pack_bf16x2(f0, f1), pack_bf16x2(f2, f3));
              }
            }
          }
        }
      }
    }
  }
  if (failed) atomicExch(&g_gemm_tma_error, 1u);
  tc_fence_before();
  __syncthreads();
  if (warp == 0) tp_tmem_free(tmem, BN);
}

int gemm_operand_map(const void *base, long rows, int cols, long pitch, int box, CUtensorMap *out) {
  typedef CUresult (*encode_fn)(CUtensorMap *, CUtensorMapDataType, cuuint32_t, void *, const cuuint64_t *, const cuuint64_t *,
                                const cuuint32_t *, const cuuint32_t *, CUtensorMapInterleave, CUtensorMapSwizzle, CUtensorMapL2promotion,
                                CUtensorMapFloatOOBfill);
  static std::mutex mu;
  static encode_fn encode = nullptr;
  {
    std::lock_guard<std::mutex> lock(mu);
    if (!encode) {
      void *fn = nullptr;
      cudaDriverEntryPointQueryResult qres;
      BLOK_CUDA(cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &fn, cudaEnableDefault, &qres));
      BLOK_REQUIRE(fn && qres == cudaDriverEntryPointSuccess, BLOK_ERR_CUDA, "gemm: the driver has no cuTensorMapEncodeTiled");
      encode = reinterpret_cast<encode_fn>(fn);
    }
  }
  const cuuint64_t dims[2] = {(cuuint64_t)cols, (cuuint64_t)rows};
  const cuuint64_t strides[1] = {(cuuint64_t)pitch * 2};
  const cuuint32_t boxes[2] = {kGtKStep, (cuuint32_t)box};
  const cuuint32_t estr[2] = {1, 1};
  const CUresult r = encode(out, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void *>(base), dims, strides, boxes, estr,
                            CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                            CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  BLOK_REQUIRE(r == CUDA_SUCCESS, BLOK_ERR_CUDA, "gemm: no tensor map (%d) for a matrix of %ld x %d, pitch %ld", (int)r, rows, cols, pitch);
  return BLOK_OK;
}

template <int BN, int ACT, bool F32>
static int gt_launch(const GemmTma &g, dim3 grid, cudaStream_t stream) {
  const GtArgs a = {g.out, g.tile_expert, g.tile_start, g.tile_count, g.num_tiles, g.T, g.R, g.K, g.ldo, g.act_cols, g.up_row};
  BLOK_CUDA(cudaFuncSetAttribute(gemm_tma_kernel<BN, ACT, F32>, cudaFuncAttributeMaxDynamicSharedMemorySize, GtCfg<BN>::kSmem));
  gemm_tma_kernel<BN, ACT, F32><<<grid, kGtThreads, GtCfg<BN>::kSmem, stream>>>(*g.x, BN == 128 || ACT == GEMM_ACT_SWIGLU ? *g.w128 : *g.w256, a);
  return launch_status("gemm_tma_kernel");
}

int launch_gemm_tma(const GemmTma &g, cudaStream_t stream) {
  BLOK_REQUIRE(g.x && g.w128 && g.out && g.R % 4 == 0 && g.K % 8 == 0 && g.T >= 1, BLOK_ERR_SHAPE, "gemm: T %d, R %d, K %d", g.T, g.R, g.K);
  if (g.act == GEMM_ACT_SWIGLU) {
    BLOK_REQUIRE(!g.out_f32 && !g.tile_start, BLOK_ERR_SHAPE, "gemm: a gated product is bf16 and not grouped");
    return gt_launch<256, GEMM_ACT_SWIGLU, false>(g, dim3((g.R + 127) / 128, (g.T + kGtTileRows - 1) / kGtTileRows), stream);
  }
  const int tiles = g.tile_start ? g.max_tiles : (g.T + kGtTileRows - 1) / kGtTileRows;
  // the wide tile reads fewer bytes from shared memory per product; it needs enough tiles to fill the GPU
  const long wide = (long)((g.R + 255) / 256) * (g.tile_start ? (g.T + kGtTileRows - 1) / kGtTileRows : tiles);
  const bool use256 = g.w256 && wide >= sm_count();
  const dim3 grid((g.R + (use256 ? 255 : 127)) / (use256 ? 256 : 128), tiles);
  if (g.act == GEMM_ACT_SILU) {
    BLOK_REQUIRE(!g.out_f32 && g.act_cols % 4 == 0, BLOK_ERR_SHAPE, "gemm: SiLU on %d columns of an fp32 output", g.act_cols);
    return use256 ? gt_launch<256, GEMM_ACT_SILU, false>(g, grid, stream) : gt_launch<128, GEMM_ACT_SILU, false>(g, grid, stream);
  }
#define BLOK_GT(BN)                                                                                   \
  return g.act == GEMM_ACT_RELU2 ? (g.out_f32 ? gt_launch<BN, GEMM_ACT_RELU2, true>(g, grid, stream)   \
                                              : gt_launch<BN, GEMM_ACT_RELU2, false>(g, grid, stream)) \
                                 : (g.out_f32 ? gt_launch<BN, GEMM_ACT_NONE, true>(g, grid, stream)    \
                                              : gt_launch<BN, GEMM_ACT_NONE, false>(g, grid, stream));
  if (use256) {
    BLOK_GT(256)
  }
  BLOK_GT(128)
#undef BLOK_GT
}

int gemm_tma_take_error(unsigned *out) {
  unsigned zero = 0;
  BLOK_CUDA(cudaMemcpyFromSymbol(out, g_gemm_tma_error, sizeof(unsigned)));
  if (*out) BLOK_CUDA(cudaMemcpyToSymbol(g_gemm_tma_error, &zero, sizeof(unsigned)));
  return BLOK_OK;
}

}  // namespace blok
