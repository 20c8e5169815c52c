// bf16 GEMM on tcgen05 with TMA-fed operands (gemm_tma.cu): out[t, r] = act(sum_k x[t, k] W[r, k]), fp32 accumulation.
#pragma once
#include <cuda.h>
#include <cuda_runtime.h>

#include <cstdint>

namespace blok {

enum { GEMM_ACT_NONE = 0, GEMM_ACT_RELU2 = 1, GEMM_ACT_SILU = 2, GEMM_ACT_SWIGLU = 3 };
constexpr int kGtTileRows = 128;  // rows of x per tile

// A matrix operand: bf16 [rows, cols], rows `pitch` elements apart (pitch a multiple of 8, base 16-byte aligned).
// `box`: rows per copied box (128 for x, 128 or 256 for weights).
int gemm_operand_map(const void *base, long rows, int cols, long pitch, int box, CUtensorMap *out);

struct GemmTma {
  const CUtensorMap *x = nullptr;              // boxes of kGtTileRows rows
  const CUtensorMap *w128 = nullptr, *w256 = nullptr;  // the weights in boxes of 128 and of 256 rows
  int T = 0;                                   // rows of x
  int R = 0, K = 0;                            // weight rows (a multiple of 4) and columns (a multiple of 8)
  void *out = nullptr;                         // bf16 or fp32 [T, ldo]
  bool out_f32 = false;
  int ldo = 0;
  int act = GEMM_ACT_NONE;
  int act_cols = 0;                            // GEMM_ACT_SILU: the first so many columns (a multiple of 4) only; bf16 output
  // GEMM_ACT_SWIGLU: out[t, r] = silu(row r) * (row up_row + r), bf16 (R counts the outputs; the weights hold both halves)
  int up_row = 0;
  // Grouped form: tile i covers rows [tile_start[i], + tile_count[i]) of x (at most kGtTileRows) and weight rows
  // [tile_expert[i] * R, + R); at most max_tiles tiles, *num_tiles of them valid.  NULL: consecutive tiles of one matrix.
  const int *tile_expert = nullptr, *tile_start = nullptr, *tile_count = nullptr, *num_tiles = nullptr;
  int max_tiles = 0;
};
int launch_gemm_tma(const GemmTma &g, cudaStream_t stream);
// *out becomes non-zero if a CTA has given up on a barrier since the last call (the flag is cleared).
int gemm_tma_take_error(unsigned *out);

}  // namespace blok
