// Kernels of the layer-stack models (model_stack.cu).  Sizes here are the padded ones the loader makes (zero rows and
// columns), so that no kernel needs a bound on a head's dimensions; the true sizes enter only where a mean is taken.
//
// Activations are bf16, or fp32 for a BLOK_DTYPE_F32 model: `Act` pointers are void* with the flag `f32`.
#pragma once
#include <cuda_runtime.h>

#include <cstdint>

namespace blok {

// Where a batch entry's cached rows and state live: entry i is the token at position pos[i] of the sequence in slot
// slot_of[i].
struct StackRows {
  const int *slot_of = nullptr, *pos = nullptr;
  const int *table = nullptr;  // [slots, table_stride] pages
  int table_stride = 0, page_rows = 0;
};

// ---- residual streams (residual_streams.cu) ----
constexpr int kMaxStreams = 16;
struct StreamsStep {
  int T = 0, width = 0, streams = 0;  // width: padded
  float *x = nullptr;                 // [T, streams, width], updated in place
  // x from the embedding (all streams alike) when ids is set
  const uint32_t *ids = nullptr;
  const uint16_t *embed = nullptr;  // bf16 [vocab, width]
  int vocab = 0;
  // else the update by a sublayer's output y: x'_t = sum_s mix[s, t] x_s + out[t] y with y = part_scale * the sum of
  // `parts` rows: y_rows[part_at ? part_at[t * parts + k] : t * parts + k].  fp32 [., width]
  const float *y_rows = nullptr;
  int parts = 1;
  const int *part_at = nullptr;
  float part_scale = 1.f;
  const float *mix = nullptr, *out = nullptr;
  bool store_x = true;  // false: x stays as it was (the update feeds the norm only)
  // what the next sublayer reads: u = sum_s in[s] x'_s (in NULL: the plain sum), h = tanh(alpha u) * w + b
  const float *in = nullptr;
  const float *norm_w = nullptr, *norm_b = nullptr;  // [width], zero in the padding; NULL: no norm wanted
  float alpha = 0.f;
  void *h = nullptr;  // Act [rows, width]
  bool h_f32 = false;
  int copies = 1;               // h of token t goes to rows copy_at[t * copies + k] (copy_at NULL: row t)
  const int *copy_at = nullptr;
  const int *rows = nullptr;    // only these tokens (T of them), row i of h is token rows[i]
  float *sum = nullptr;         // fp32 [T, true_width]: the sum of the streams (for parity checks)
  int true_width = 0;
};
int launch_streams_step(const StreamsStep &a, cudaStream_t stream);

// ---- one residual between sandwiched sublayers (residual_norm.cu) ----
constexpr int kMaxNormWidth = 32768;
struct ResidualNorm {
  int T = 0, width = 0, true_width = 0;  // width: padded, zero in the padding
  float *x = nullptr;                    // [T, width]
  // x from the embeddings when ids is set: embed_scale * embed[id] + the pair's row + the position's sinusoid
  const uint32_t *ids = nullptr;
  const uint16_t *embed = nullptr, *bigram = nullptr;  // bf16 [vocab, width], [buckets + 1, width] or NULL
  int vocab = 0, buckets = 0;
  long mul_prev = 0, mul_cur = 0;
  float embed_scale = 1.f;
  const double *turns = nullptr;         // [width / 2] turns per position of every pair of columns, or NULL
  const int *pos = nullptr, *slot_of = nullptr;
  bool chunk = false;                    // rows are consecutive tokens of one sequence
  uint32_t *last_ids = nullptr;          // [slots] the newest token of every sequence
  const uint32_t *keep_ids = nullptr;    // set: last_ids takes in this call's newest tokens (in a later launch than ids)
  // else x += mult * layer_norm(y) * post_w (post_w NULL: += mult * y) when y is set
  const float *y = nullptr;              // [T, width]
  const float *post_w = nullptr;
  float mult = 1.f, eps = 0.f;
  float *copy = nullptr;                 // [T, true_width]: x (for parity checks)
  // h = layer_norm(x) * norm_w, Act [T, width]
  const float *norm_w = nullptr;
  void *h = nullptr;
  bool h_f32 = false;
};
int launch_residual_norm(const ResidualNorm &a, cudaStream_t stream);

// ---- linear attention with a decay per head, fixed or per token (linear_attn.cu) ----
enum { GATE_SILU = 0, GATE_SIGMOID = 1 };
struct LinearAttn {
  int heads = 0, dim = 0, vdim = 0;  // padded: multiples of 16
  const void *qkvg = nullptr;        // Act [T, ld]: q | k | v | g, head by head
  int share = 1;                     // so many heads share one head of q and k
  bool v_first = false;              // Act [T, ld]: v | k | q
  int ld = 0;
  bool f32 = false;
  bool silu_qkv = false;             // q, k and v go through SiLU (rounded to Act) when they are read
  float k_scale = 1.f;
  const float *decay_pow = nullptr;  // [heads, kLinChunk + 1]: decay^i
  // decays per token instead: [heads, token_ld] of (key scale, log decay, the log decays' running sum inside the token's chunk
  // of kLinChunk in two parts), and o += skip[head] v
  const float4 *token = nullptr;
  int token_ld = 0;
  const float *skip = nullptr;       // [heads]
  float *state = nullptr;            // fp32 [slots, heads, dim, vdim]
  float *o = nullptr;                // fp32 [T, heads * vdim]
  float *chunk_state = nullptr;      // scratch [chunks, heads, dim, vdim] of the chunked form
};
constexpr int kLinChunk = 64;
constexpr int kLinMaxDim = 256;
// One token of each of B sequences, or (chunk) T tokens of one sequence whose first position is first_pos.
int launch_linear_step(const LinearAttn &a, const StackRows &r, int B, cudaStream_t stream);
int launch_linear_chunk(const LinearAttn &a, int slot, long first_pos, int T, cudaStream_t stream);
size_t linear_chunk_scratch_bytes(int heads, int dim, int vdim, int T);
// out = rmsnorm(o) * w * gate(g): per head over true_vdim values (per_head), or over all heads together.
struct GatedNorm {
  int heads = 0, vdim = 0, true_vdim = 0;
  bool per_head = false;
  const float *w = nullptr;  // [heads * vdim] or NULL
  float eps = 0.f;
  int gate = GATE_SILU;
  const float *o = nullptr;  // fp32 [T, heads * vdim]
  const void *g = nullptr;   // Act [T, ldg]
  int ldg = 0;
  void *out = nullptr;       // Act [T, ldo], columns past heads * vdim zeroed
  int ldo = 0;
  bool f32 = false;
};
int launch_gated_norm(const GatedNorm &a, int T, cudaStream_t stream);
// out = rmsnorm(o * silu(g)) * w over `parts` equal parts of the heads * true_vdim true columns (per_head, gate: unused).
int launch_gate_then_norm(const GatedNorm &a, int parts, int T, cudaStream_t stream);

// ---- inputs of a selective state space (state_space.cu) ----
struct StateInputs {
  int heads = 0, channels = 0, taps = 0;  // channels: padded, a multiple of 16
  const void *proj = nullptr;             // Act [T, ld]: anything | channels at `first` | anything | steps at dt_at
  int ld = 0, first = 0, dt_at = 0;
  bool f32 = false;
  const float *conv_w = nullptr, *conv_b = nullptr;   // [taps, channels] (current token last), [channels]
  const float *dt_bias = nullptr, *rate = nullptr;    // [heads]; rate = -exp(log rate)
  void *ring = nullptr;                   // Act [slots, taps, channels]: the input at position p lies at p % taps
  void *out = nullptr;                    // Act [T, channels]: silu(conv + b)
  float4 *token = nullptr;                // [heads, token_ld], see LinearAttn
  int token_ld = 0;
};
// Rows are the next token of T sequences, or (chunk) T consecutive tokens of one.
int launch_state_inputs(const StateInputs &a, const StackRows &r, int T, bool chunk, cudaStream_t stream);

// ---- latent attention over a paged cache of rows [latent | rotated key] (latent_attn.cu) ----
struct LatentShape {
  int heads = 0, dim = 0, rot = 0, vdim = 0, rank = 0, q_rank = 0;          // padded
  int true_rot = 0, true_rank = 0, true_q_rank = 0, rot_dims = 0;
  const double *turns = nullptr;  // device, [rot_dims / 2]: turns per position of every pair, base^(-2i / dims) / 2 pi
  float scale = 1.f, eps = 0.f;
  __host__ __device__ int row() const { return rank + rot; }  // a cached row
  __host__ __device__ int head() const { return dim + rot; }  // a query head
};
// ckr fp32 [T, q_rank + row]: the query latent is normed into cq (Act [T, q_rank]); the key latent is normed, the shared
// key part rotated, and the row appended to the pool (Act [pages, page_rows, row]).
int launch_latent_append(const LatentShape &s, const float *ckr, const float *q_norm, const float *kv_norm, const StackRows &r, int T, void *cq,
                         void *pool, bool f32, cudaStream_t stream);
// Rotates the last `rot` columns of every query head of q (Act [T, heads, head()]) into dst, whose heads are dst_head
// columns apart starting at dst_off (dst == q, dst_head == head(), dst_off == dim: in place).
int launch_latent_rotate(const LatentShape &s, const void *q, const StackRows &r, int T, void *dst, int dst_head, int dst_off, bool f32,
                         cudaStream_t stream);
// Absorbed form: q_abs Act [T, heads, row()], o Act [T, heads, rank].  Entry i attends to positions 0..pos[i].
// Scratch for calls of up to T entries: part_o fp32 [max_parts, heads, rank] and part_ml fp32 [max_parts, heads, 2].  Each
// buffer must hold finite values (part_o) at the first call and serve this purpose only: an empty part leaves its rows as
// they were and the merge multiplies them by zero.
size_t latent_attend_max_parts(const LatentShape &s, int T, long max_ctx);
int launch_latent_attend(const LatentShape &s, const void *q_abs, const void *pool, const StackRows &r, int T, long max_ctx, void *o, bool f32,
                         float *part_o, float *part_ml, cudaStream_t stream);
// Prompt form (bf16): the first n cached rows of the sequence in `slot` copied to c_all [n, rank] and kr_all [n, rot] ...
int launch_latent_gather(const LatentShape &s, const uint16_t *pool, const StackRows &r, int slot, int n, uint16_t *c_all, uint16_t *kr_all,
                         cudaStream_t stream);
// ... and, with kv = the per-head keys and values made from them (bf16 [n, heads * (dim + vdim)]: all keys, then all
// values), causal attention of T queries at positions n - T .. n - 1: q bf16 [T, heads, head()], o bf16 [T, ldo].
bool latent_prompt_supports(const LatentShape &s);
int launch_latent_prompt(const LatentShape &s, const uint16_t *q, const uint16_t *kv, const uint16_t *kr_all, int T, int n, uint16_t *o, int ldo,
                         cudaStream_t stream);

// ---- grouped softmax attention over a paged cache of rows [keys | values] (grouped_attn.cu, prompt_attn_tc.cu) ----
struct GroupedShape {
  int heads = 0, kv_heads = 0, dim = 0, vdim = 0;  // padded: dim a multiple of 32, vdim of 16
  int true_dim = 0;
  float scale = 1.f, eps = 0.f;
  const float *bias = nullptr;  // [heads, bias_len] by distance, the last entry for every distance from there on; or NULL
  int bias_len = 0;
  __host__ __device__ int row() const { return kv_heads * (dim + vdim); }  // a cached row
};
template <typename Act>
struct GroupedQuery {
  const Act *q = nullptr;     // [T, ldq]: head by head
  int ldq = 0;
  const Act *gate = nullptr;  // [T, ld_gate], one value per head, before the sigmoid; or NULL
  int ld_gate = 0;
  Act *out = nullptr;         // [T, ldo]: head by head
  int ldo = 0;
};
// qkv Act [T, ld]: q | k | v.  q is normed in place over all heads (q_norm NULL: left alone), k likewise, and the row appended to
// the pool (Act [pages, page_rows, row]; NULL: q only).
int launch_grouped_append(const GroupedShape &s, void *qkv, int ld, const float *q_norm, const float *k_norm, const StackRows &r, int T, void *pool,
                          bool f32, cudaStream_t stream);
// Entry i attends to positions 0..pos[i].  part_o fp32 [max_parts, heads, vdim], part_ml fp32 [max_parts, heads, 2], finite at the
// first call (see launch_latent_attend).
size_t grouped_attend_max_parts(const GroupedShape &s, int T, long max_ctx);
int launch_grouped_attend(const GroupedShape &s, const GroupedQuery<uint16_t> &a, const void *pool, const StackRows &r, int T, long max_ctx,
                          float *part_o, float *part_ml, cudaStream_t stream);
int launch_grouped_attend_f32(const GroupedShape &s, const GroupedQuery<float> &a, const void *pool, const StackRows &r, int T, cudaStream_t stream);
// T tokens of the sequence in `slot` at positions n - T .. n - 1; every row of the pool must hold finite values.
bool grouped_prompt_supports(const GroupedShape &s);
int launch_grouped_prompt(const GroupedShape &s, const GroupedQuery<uint16_t> &a, const void *pool, long pool_rows, const StackRows &r, int slot, int T,
                          int n, cudaStream_t stream);

// ---- experts chosen by a table of token ids (table_experts.cu) ----
struct ExpertPlan {          // of one layer and call
  int *at = nullptr;         // [T * top] row of assignment (t, k) in expert order
  int *tile_expert = nullptr, *tile_start = nullptr, *tile_count = nullptr, *num_tiles = nullptr;  // tiles of up to 128 rows
};
struct ExpertPlanArgs {
  const int *table = nullptr;  // [vocab, top]
  int experts = 0, top = 0;
  ExpertPlan plan;
};
constexpr int kMaxTableExperts = 4096;
int expert_plan_max_tiles(int assignments, int experts);
// One block per layer of `layers` (device array of n_layers).
int launch_expert_plan(const ExpertPlanArgs *layers, int n_layers, const uint32_t *ids, int vocab, int T, cudaStream_t stream);
// y[a, :] = act(W[e(a)] x[row(a), :]) assignment by assignment, e(a) = table[ids[a / top]][a % top] and row(a) = a / top
// (shared_x) or a.  W bf16 [experts, R, K]; x Act [., K]; y Act or fp32 [T * top, R].
int launch_expert_gemv(const uint16_t *w, int R, int K, const int *table, const uint32_t *ids, int vocab, int top, int T, const void *x, bool x_f32,
                       bool shared_x, bool relu2, void *y, bool y_f32, cudaStream_t stream);

// ---- fp32 products (gemm_f32.cu): y[z][t, r] = sum_k x[z][t, k] W[z][r, k], W bf16, x and y fp32 ----
struct GemmF32 {
  const uint16_t *w = nullptr;
  const float *x = nullptr;
  float *y = nullptr;
  int R = 0, K = 0, T = 0, ldw = 0, ldx = 0, ldy = 0, batch = 1;
  long w_stride = 0, x_stride = 0, y_stride = 0;  // between batches
};
int launch_gemm_f32(const GemmF32 &g, cudaStream_t stream);
// out[t, r] = silu(x[t, r]) * x[t, cols + r], x fp32 [T, 2 cols]
int launch_swiglu_f32(const float *x, float *out, int cols, int T, cudaStream_t stream);

}  // namespace blok
