// The tcgen05 attention core of prompts (prompt_attn_tc.cu).
#pragma once
#include <cuda.h>
#include <cuda_runtime.h>

#include <cstdint>

namespace blok {

struct PromptAttn {
  uint16_t *out = nullptr;  // bf16 [T, ldo]: head by head
  int ldo = 0;
  const uint16_t *gate = nullptr;  // bf16 [T, ld_gate]: head h's output times sigmoid(gate[t][h]); or NULL
  int ld_gate = 0;
  int T = 0, n = 0;  // queries at positions n - T .. n - 1
  int heads = 0, share = 1;  // so many query heads share a key head
  int q_head = 0;            // columns between query heads
  int dim = 0, vdim = 0;     // query-key and value size, multiples of 16
  // a key: key_chunks chunks of 64 columns from column (key head) * k_head of the key map, then chunks 0, 1, .. of the map of
  // the part that the heads share; its value from column v_first + (key head) * vdim of the key map
  int k_head = 0, key_chunks = 0, v_first = 0;
  float scale_log2 = 0.f;    // scale * log2 e; positive unless there is a bias
  const float *bias = nullptr;  // [heads, bias_len] by distance, the last entry from there on; or NULL
  int bias_len = 0;
  const int *table = nullptr;   // pages of the sequence, `page_rows` rows each (a multiple of `box`); NULL: key j is row j
  int page_rows = 1, box = 64;  // box: rows per copied box of the key maps, 64 or 32
  int stages = 0;               // tiles of 64 keys in shared memory at a time (set by the launch)
};
bool prompt_attn_supports(int dim, int vdim);
// Maps of 64 columns, bf16, 128-byte swizzle (gemm_operand_map): boxes of 128 queries, of `box` keys.
int launch_prompt_attn(const CUtensorMap &mq, const CUtensorMap &mkv, const CUtensorMap &mkr, PromptAttn a, cudaStream_t stream);
int prompt_attn_take_error(unsigned *out);

}  // namespace blok
