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

extern "C" int blok_residual_norm(float *x, const float *y, const float *post_w, float mult, const float *norm_w, float eps, int T, int width,
                                  int true_width, void *h, int f32, blok_stream_t stream) {
  BLOK_REQUIRE(x && norm_w && h, BLOK_ERR_ARG, "blok_residual_norm: null pointer");
  ResidualNorm a;
  a.T = T;
  a.width = width;
  a.true_width = true_width;
  a.x = x;
  a.y = y;
  a.post_w = post_w;
  a.mult = mult;
  a.eps = eps;
  a.norm_w = norm_w;
  a.h = h;
  a.h_f32 = f32 != 0;
  return launch_residual_norm(a, (cudaStream_t)stream);
}

extern "C" int blok_token_embedding(const uint32_t *ids, uint32_t *last_ids, const int *slot_of, const int *pos, int chunk, int keep,
                                    const blok_bf16_t *embed, int vocab, const blok_bf16_t *bigram, int buckets, long mul_prev, long mul_cur,
                                    float scale, const double *turns, int T, int width, int true_width, float *x, blok_stream_t stream) {
  BLOK_REQUIRE(ids && embed && x && pos && slot_of && vocab >= 1 && (!bigram || (last_ids && buckets >= 1 && mul_prev >= 0 && mul_cur >= 0)) && (!keep || last_ids),
               BLOK_ERR_ARG, "blok_token_embedding: null pointer or bad size");
  ResidualNorm a;
  a.T = T;
  a.width = width;
  a.true_width = true_width;
  a.x = x;
  a.ids = ids;
  a.embed = embed;
  a.vocab = vocab;
  a.embed_scale = scale;
  a.bigram = bigram;
  a.buckets = buckets;
  a.mul_prev = mul_prev;
  a.mul_cur = mul_cur;
  a.turns = turns;
  a.pos = pos;
  a.slot_of = slot_of;
  a.chunk = chunk != 0;
  a.last_ids = last_ids;
  if (int rc = launch_residual_norm(a, (cudaStream_t)stream)) return rc;
  if (!keep) return BLOK_OK;
  a.ids = nullptr;
  a.keep_ids = ids;
  return launch_residual_norm(a, (cudaStream_t)stream);
}

extern "C" int blok_state_inputs(const void *proj, int f32, int ld, int first, int dt_at, int heads, int channels, int taps, const float *conv_w,
                                 const float *conv_b, const float *dt_bias, const float *rate, void *ring, const int *slot_of, const int *pos, int T,
                                 int chunk, void *out, float *token, int token_ld, blok_stream_t stream) {
  BLOK_REQUIRE(proj && conv_w && conv_b && dt_bias && rate && ring && slot_of && pos && out && token, BLOK_ERR_ARG, "blok_state_inputs: null pointer");
  BLOK_REQUIRE(first >= 0 && first + channels <= ld && dt_at >= 0 && dt_at + heads <= ld, BLOK_ERR_SHAPE, "blok_state_inputs: rows of %d values are too short", ld);
  StateInputs a;
  a.heads = heads;
  a.channels = channels;
  a.taps = taps;
  a.proj = proj;
  a.ld = ld;
  a.first = first;
  a.dt_at = dt_at;
  a.f32 = f32 != 0;
  a.conv_w = conv_w;
  a.conv_b = conv_b;
  a.dt_bias = dt_bias;
  a.rate = rate;
  a.ring = ring;
  a.out = out;
  a.token = reinterpret_cast<float4 *>(token);
  a.token_ld = token_ld;
  StackRows r;
  r.slot_of = slot_of;
  r.pos = pos;
  return launch_state_inputs(a, r, T, chunk != 0, (cudaStream_t)stream);
}

extern "C" int blok_selective_state(const void *xbc, int f32, int ld, int heads, int groups, int state_dim, int vdim, const float *token, int token_ld,
                                    const float *skip, float *state, int slot, int first_pos, int T, const int *slot_of, const int *pos, float *o,
                                    void *scratch, blok_stream_t stream) {
  BLOK_REQUIRE(xbc && token && skip && state && o && T >= 1 && T <= token_ld && slot >= 0 && first_pos >= 0, BLOK_ERR_ARG,
               "blok_selective_state: null pointer or bad place");
  BLOK_REQUIRE(groups >= 1 && heads % groups == 0 && ld >= heads * vdim + 2 * groups * state_dim, BLOK_ERR_SHAPE,
               "blok_selective_state: %d heads in %d groups, rows of %d values", heads, groups, ld);
  BLOK_REQUIRE((slot_of != nullptr) == (pos != nullptr), BLOK_ERR_ARG, "blok_selective_state: a step needs slot_of and pos");
  BLOK_REQUIRE(slot_of || f32 || T <= 8 || scratch, BLOK_ERR_WORKSPACE, "blok_selective_state: a portion needs scratch");
  LinearAttn a;
  a.heads = heads;
  a.dim = state_dim;
  a.vdim = vdim;
  a.qkvg = xbc;
  a.share = heads / groups;
  a.v_first = true;
  a.ld = ld;
  a.f32 = f32 != 0;
  a.token = reinterpret_cast<const float4 *>(token);
  a.token_ld = token_ld;
  a.skip = skip;
  a.state = state;
  a.o = o;
  a.chunk_state = static_cast<float *>(scratch);
  if (!slot_of) return launch_linear_chunk(a, slot, first_pos, T, (cudaStream_t)stream);
  StackRows r;
  r.slot_of = slot_of;
  r.pos = pos;
  return launch_linear_step(a, r, T, (cudaStream_t)stream);
}

extern "C" int blok_gate_then_norm(const float *o, const void *gate, int ld_gate, const float *w, int heads, int vdim, int true_vdim, int parts, float eps,
                                   int T, void *out, int ld_out, int f32, blok_stream_t stream) {
  BLOK_REQUIRE(o && gate && out && T >= 1 && heads >= 1 && vdim >= 1 && true_vdim >= 1 && true_vdim <= vdim && ld_gate >= heads * vdim && ld_out >= heads * vdim,
               BLOK_ERR_ARG, "blok_gate_then_norm: null pointer or bad size");
  GatedNorm g;
  g.heads = heads;
  g.vdim = vdim;
  g.true_vdim = true_vdim;
  g.w = w;
  g.eps = eps;
  g.o = o;
  g.g = gate;
  g.ldg = ld_gate;
  g.out = out;
  g.ldo = ld_out;
  g.f32 = f32 != 0;
  return launch_gate_then_norm(g, parts, T, (cudaStream_t)stream);
}

static int grouped_shape(const char *who, int heads, int kv_heads, int dim, int vdim, float scale, const float *bias, int bias_len, GroupedShape *s) {
  BLOK_REQUIRE(heads >= 1 && kv_heads >= 1 && heads % kv_heads == 0 && dim >= 32 && dim % 32 == 0 && vdim >= 16 && vdim % 16 == 0 &&
                   (!bias || bias_len >= 1),
               BLOK_ERR_SHAPE, "%s: %d heads over %d of %d / %d (multiples of 32 and 16)", who, heads, kv_heads, dim, vdim);
  s->heads = heads;
  s->kv_heads = kv_heads;
  s->dim = s->true_dim = dim;
  s->vdim = vdim;
  s->scale = scale;
  s->bias = bias;
  s->bias_len = bias_len;
  return BLOK_OK;
}
static StackRows paged_rows(const int *table, int table_stride, int page_rows, const int *slot_of, const int *pos) {
  StackRows r;
  r.slot_of = slot_of;
  r.pos = pos;
  r.table = table;
  r.table_stride = table_stride;
  r.page_rows = page_rows;
  return r;
}

extern "C" int blok_grouped_append(void *qkv, int f32, int ld, int heads, int kv_heads, int dim, int true_dim, int vdim, const float *q_norm,
                                   const float *k_norm, float eps, const int *table, int table_stride, int page_rows, const int *slot_of,
                                   const int *pos, int T, void *pool, blok_stream_t stream) {
  BLOK_REQUIRE(qkv && T >= 1 && (!pool || (table && slot_of && pos && table_stride >= 1 && page_rows >= 1 && (!q_norm || k_norm))), BLOK_ERR_ARG,
               "blok_grouped_append: null pointer or no rows");
  GroupedShape s;
  if (int rc = grouped_shape("blok_grouped_append", heads, kv_heads, dim, vdim, 1.f, nullptr, 0, &s)) return rc;
  BLOK_REQUIRE(true_dim >= 1 && true_dim <= dim && ld >= heads * dim + (pool ? kv_heads * (dim + vdim) : 0), BLOK_ERR_SHAPE,
               "blok_grouped_append: rows of %d values are too short", ld);
  s.true_dim = true_dim;
  s.eps = eps;
  return launch_grouped_append(s, qkv, ld, q_norm, k_norm, paged_rows(table, table_stride, page_rows, slot_of, pos), T, pool, f32 != 0,
                               (cudaStream_t)stream);
}

extern "C" size_t blok_grouped_attend_workspace_bytes(int heads, int kv_heads, int dim, int vdim, int T, long max_ctx) {
  GroupedShape s;
  if (grouped_shape("blok_grouped_attend", heads, kv_heads, dim, vdim, 1.f, nullptr, 0, &s) || T < 1 || max_ctx < 1) return 0;
  return grouped_attend_max_parts(s, T, max_ctx) * heads * (size_t)(vdim + 2) * sizeof(float);
}

template <typename Act>
static GroupedQuery<Act> grouped_query(const void *q, int ldq, const void *gate, int ld_gate, void *out, int ldo) {
  GroupedQuery<Act> a;
  a.q = static_cast<const Act *>(q);
  a.ldq = ldq;
  a.gate = static_cast<const Act *>(gate);
  a.ld_gate = ld_gate;
  a.out = static_cast<Act *>(out);
  a.ldo = ldo;
  return a;
}

extern "C" int blok_grouped_attend(const void *q, int f32, int ldq, const void *gate, int ld_gate, const void *pool, const int *table, int table_stride,
                                   int page_rows, const int *slot_of, const int *pos, int heads, int kv_heads, int dim, int vdim, float scale,
                                   const float *bias, int bias_len, int T, long max_ctx, void *out, int ldo, void *workspace, blok_stream_t stream) {
  BLOK_REQUIRE(q && pool && table && slot_of && pos && out && (f32 || workspace) && T >= 1 && table_stride >= 1 && page_rows >= 1, BLOK_ERR_ARG,
               "blok_grouped_attend: null pointer or no entries");
  GroupedShape s;
  if (int rc = grouped_shape("blok_grouped_attend", heads, kv_heads, dim, vdim, scale, bias, bias_len, &s)) return rc;
  BLOK_REQUIRE(ldq >= heads * dim && ldq % 8 == 0 && ldo >= heads * vdim && ldo % 4 == 0, BLOK_ERR_SHAPE, "blok_grouped_attend: rows of %d and %d values",
               ldq, ldo);
  const StackRows r = paged_rows(table, table_stride, page_rows, slot_of, pos);
  if (f32) return launch_grouped_attend_f32(s, grouped_query<float>(q, ldq, gate, ld_gate, out, ldo), pool, r, T, (cudaStream_t)stream);
  float *part_o = static_cast<float *>(workspace);
  return launch_grouped_attend(s, grouped_query<uint16_t>(q, ldq, gate, ld_gate, out, ldo), pool, r, T, max_ctx, part_o,
                               part_o + grouped_attend_max_parts(s, T, max_ctx) * heads * (size_t)vdim, (cudaStream_t)stream);
}

extern "C" int blok_grouped_prompt(const blok_bf16_t *q, int ldq, const blok_bf16_t *gate, int ld_gate, const blok_bf16_t *pool, long pool_rows,
                                   const int *table, int table_stride, int page_rows, int slot, int heads, int kv_heads, int dim, int vdim, float scale,
                                   const float *bias, int bias_len, int T, int n, blok_bf16_t *out, int ldo, blok_stream_t stream) {
  BLOK_REQUIRE(q && pool && table && out && T >= 1 && n >= T && slot >= 0 && page_rows >= 1 && n <= (long)table_stride * page_rows && pool_rows >= page_rows,
               BLOK_ERR_ARG, "blok_grouped_prompt: null pointer or bad place");
  GroupedShape s;
  if (int rc = grouped_shape("blok_grouped_prompt", heads, kv_heads, dim, vdim, scale, bias, bias_len, &s)) return rc;
  BLOK_REQUIRE(grouped_prompt_supports(s) && ldq >= heads * dim && ldo >= heads * vdim, BLOK_ERR_SHAPE, "blok_grouped_prompt: heads of %d / %d, scale %g", dim, vdim,
               scale);
  return launch_grouped_prompt(s, grouped_query<uint16_t>(q, ldq, gate, ld_gate, out, ldo), pool, pool_rows,
                               paged_rows(table, table_stride, page_rows, nullptr, nullptr), slot, T, n, (cudaStream_t)stream);
}

extern "C" int blok_gemm_swiglu(const blok_bf16_t *x, const blok_bf16_t *w, int T, int R, int K, blok_bf16_t *out, blok_stream_t stream) {
  BLOK_REQUIRE(x && w && out, BLOK_ERR_ARG, "blok_gemm_swiglu: null pointer");
  BLOK_REQUIRE(T >= 1 && R >= 4 && R % 4 == 0 && K >= 8 && K % 8 == 0, BLOK_ERR_SHAPE, "blok_gemm_swiglu: T %d, R %d (a multiple of 4), K %d (of 8)", T, R, K);
  CUtensorMap mx, m128;
  int rc;
  if ((rc = gemm_operand_map(x, T, K, K, kGtTileRows, &mx)) || (rc = gemm_operand_map(w, 2 * R, K, K, 128, &m128))) return rc;
  GemmTma g;
  g.x = &mx;
  g.w128 = &m128;
  g.T = T;
  g.R = g.ldo = g.up_row = R;
  g.K = K;
  g.act = GEMM_ACT_SWIGLU;
  g.out = out;
  return launch_gemm_tma(g, (cudaStream_t)stream);
}
