// C entry points of the layer-stack kernels, one mechanism each, for parity checks and measurement.
#include <cmath>
#include <vector>

#include "gemm_tma.h"
#include "stack_kernels.h"
#include "common.cuh"

using namespace blok;

extern "C" size_t blok_linear_attention_scratch_bytes(int heads, int dim, int vdim, int T) {
  return heads > 0 && dim > 0 && vdim > 0 && T > 0 ? linear_chunk_scratch_bytes(heads, dim, vdim, T) : 0;
}

extern "C" void blok_linear_attention_decay(const double *decay, int heads, float *table) {
  if (!decay || !table) return;
  for (int h = 0; h < heads; ++h)
    for (int i = 0; i <= kLinChunk; ++i) table[(size_t)h * (kLinChunk + 1) + i] = (float)std::pow(decay[h], i);
}

extern "C" int blok_linear_attention(const void *qkvg, int f32, int ld, int heads, int dim, int vdim, const float *decay_table, float k_scale,
                                     int silu_qkv, float *state, int slot, int first_pos, int T, const int *slot_of, const int *pos, float *o,
                                     void *scratch, blok_stream_t stream) {
  BLOK_REQUIRE(qkvg && decay_table && state && o && T >= 1 && slot >= 0 && first_pos >= 0, BLOK_ERR_ARG, "blok_linear_attention: null pointer or bad place");
  BLOK_REQUIRE(ld >= 2 * heads * dim + heads * vdim, BLOK_ERR_SHAPE, "blok_linear_attention: rows of %d values are too short", ld);
  BLOK_REQUIRE((slot_of != nullptr) == (pos != nullptr), BLOK_ERR_ARG, "blok_linear_attention: a step needs slot_of and pos");
  BLOK_REQUIRE(slot_of || f32 || T <= 8 || scratch, BLOK_ERR_WORKSPACE, "blok_linear_attention: a portion needs scratch");
  LinearAttn a;
  a.heads = heads;
  a.dim = dim;
  a.vdim = vdim;
  a.qkvg = qkvg;
  a.ld = ld;
  a.f32 = f32 != 0;
  a.silu_qkv = silu_qkv != 0;
  a.k_scale = k_scale;
  a.decay_pow = decay_table;
  a.state = state;
  a.o = o;
  a.chunk_state = static_cast<float *>(scratch);
  if (!slot_of) return launch_linear_chunk(a, slot, first_pos, T, (cudaStream_t)stream);
  StackRows r;
  r.slot_of = slot_of;
  r.pos = pos;
  return launch_linear_step(a, r, T, (cudaStream_t)stream);
}

extern "C" int blok_gated_norm(const float *o, const void *gate, int ld_gate, const float *w, int heads, int vdim, int true_vdim, int per_head, float eps,
                               int sigmoid, int T, void *out, int ld_out, int f32, blok_stream_t stream) {
  BLOK_REQUIRE(o && gate && out && T >= 1 && heads >= 1 && vdim % 4 == 0 && true_vdim >= 1 && true_vdim <= vdim && ld_gate % 4 == 0 && ld_out % 4 == 0 && ld_out >= heads * vdim,
               BLOK_ERR_ARG, "blok_gated_norm: null pointer or bad size");
  GatedNorm g;
  g.heads = heads;
  g.vdim = vdim;
  g.true_vdim = true_vdim;
  g.per_head = per_head != 0;
  g.w = w;
  g.eps = eps;
  g.gate = sigmoid ? GATE_SIGMOID : GATE_SILU;
  g.o = o;
  g.g = gate;
  g.ldg = ld_gate;
  g.out = out;
  g.ldo = ld_out;
  g.f32 = f32 != 0;
  return launch_gated_norm(g, T, (cudaStream_t)stream);
}

static LatentShape latent_shape(int heads, int dim, int rot, int vdim, int rank, float scale) {
  LatentShape s;
  s.heads = heads;
  s.dim = dim;
  s.rot = s.true_rot = s.rot_dims = rot;
  s.vdim = vdim;
  s.rank = s.true_rank = rank;
  s.q_rank = s.true_q_rank = 32;
  s.scale = scale;
  return s;
}
static int latent_sizes_ok(const LatentShape &s, const char *who) {
  BLOK_REQUIRE(s.heads >= 1 && s.dim % 32 == 0 && s.rot % 32 == 0 && s.vdim % 16 == 0 && s.rank % 32 == 0 && s.rank > 0 && s.rot > 0, BLOK_ERR_SHAPE,
               "%s: dim, rot and rank must be multiples of 32 and vdim of 16", who);
  return BLOK_OK;
}

extern "C" size_t blok_latent_attend_workspace_bytes(int heads, int rot, int rank, int T, long max_ctx) {
  const LatentShape s = latent_shape(heads, 32, rot, 16, rank, 1.f);
  return latent_attend_max_parts(s, T, max_ctx) * heads * (size_t)(rank + 2) * sizeof(float);
}

extern "C" int blok_latent_attend(const void *q, const void *pool, const int *table, int table_stride, int page_rows, const int *slot_of, const int *pos,
                                  int heads, int rot, int rank, float scale, int T, long max_ctx, void *o, int f32, void *workspace,
                                  blok_stream_t stream) {
  BLOK_REQUIRE(q && pool && table && slot_of && pos && o && workspace && T >= 1 && table_stride >= 1 && page_rows >= 1, BLOK_ERR_ARG,
               "blok_latent_attend: null pointer or no entries");
  const LatentShape s = latent_shape(heads, 32, rot, 16, rank, scale);
  if (int rc = latent_sizes_ok(s, "blok_latent_attend")) return rc;
  StackRows r;
  r.slot_of = slot_of;
  r.pos = pos;
  r.table = table;
  r.table_stride = table_stride;
  r.page_rows = page_rows;
  float *part_o = static_cast<float *>(workspace);
  return launch_latent_attend(s, q, pool, r, T, max_ctx, o, f32 != 0, part_o, part_o + latent_attend_max_parts(s, T, max_ctx) * heads * (size_t)rank,
                              (cudaStream_t)stream);
}

extern "C" int blok_latent_prompt(const blok_bf16_t *q, const blok_bf16_t *kv, const blok_bf16_t *k_rot, int heads, int dim, int rot, int vdim, float scale,
                                  int T, int n, blok_bf16_t *o, int ld_out, blok_stream_t stream) {
  BLOK_REQUIRE(q && kv && k_rot && o && ld_out >= heads * vdim, BLOK_ERR_ARG, "blok_latent_prompt: null pointer or short rows");
  const LatentShape s = latent_shape(heads, dim, rot, vdim, 32, scale);
  if (int rc = latent_sizes_ok(s, "blok_latent_prompt")) return rc;
  return launch_latent_prompt(s, q, kv, k_rot, T, n, o, ld_out, (cudaStream_t)stream);
}

extern "C" int blok_gemm_bf16(const blok_bf16_t *x, const blok_bf16_t *w, int T, int R, int K, int relu2, blok_bf16_t *out_bf16, float *out_f32,
                              blok_stream_t stream) {
  BLOK_REQUIRE(x && w && (out_bf16 != nullptr) != (out_f32 != nullptr), BLOK_ERR_ARG, "blok_gemm_bf16: need x, w and exactly one output");
  BLOK_REQUIRE(T >= 1 && R >= 4 && R % 4 == 0 && K >= 8 && K % 8 == 0, BLOK_ERR_SHAPE, "blok_gemm_bf16: T %d, R %d (a multiple of 4), K %d (of 8)", T, R, K);
  CUtensorMap mx, m128, m256;
  int rc;
  if ((rc = gemm_operand_map(x, T, K, K, kGtTileRows, &mx)) || (rc = gemm_operand_map(w, R, K, K, 128, &m128)) ||
      (rc = gemm_operand_map(w, R, K, K, 256, &m256)))
    return rc;
  GemmTma g;
  g.x = &mx;
  g.w128 = &m128;
  g.w256 = &m256;
  g.T = T;
  g.R = g.ldo = R;
  g.K = K;
  g.out = out_bf16 ? static_cast<void *>(out_bf16) : out_f32;
  g.out_f32 = out_f32 != nullptr;
  g.act = relu2 ? GEMM_ACT_RELU2 : GEMM_ACT_NONE;
  return launch_gemm_tma(g, (cudaStream_t)stream);
}
