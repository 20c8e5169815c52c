// Runtime of the layer-stack models (stack.h): weight loading into padded device matrices, caches and recurrent states per
// layer run, and the launches of a step or a prompt chunk.
//
// Padding.  Heads' dimensions, ranks, widths and rows are padded with zero rows and columns when the weights are loaded
// (a head's key size to 16, its value size to 16, everything a product contracts to 32), so that every activation is
// aligned and the kernels need no bounds inside a head.  Padded values come out as zeros at every stage.
//
// A layer run is: residual + norm -> mixer -> residual + norm -> feed-forward.  The residual's update by a sublayer's output is
// fused with the norm in front of the next one (residual_streams.cu, residual_norm.cu), across layer borders too.
#include <algorithm>
#include <cmath>
#include <cstring>
#include <map>
#include <memory>
#include <new>
#include <utility>

#include "gemm_tma.h"
#include "prompt_attn_tc.h"
#include "safetensors.h"
#include "stack.h"
#include "stack_kernels.h"
#include "synth_fill.cuh"
#include "wgemm.h"

namespace blok {

size_t bf16_gemv_splitk_workspace_bytes(int rows);
int launch_bf16_gemv_splitk(const uint16_t *w, const uint16_t *x, uint16_t *y_bf16, float *y_f32, int rows, int cols, int T, void *ws, size_t ws_bytes,
                            cudaStream_t stream);
int launch_head_gemv(const uint16_t *w, long w_head_stride, const uint16_t *x, long x_tok_stride, long x_head_stride, uint16_t *y, long y_tok_stride,
                     long y_head_stride, int rows, int cols, int heads, int T, cudaStream_t stream);
int launch_bf16_gateup(const uint16_t *gate, const uint16_t *up, const uint16_t *x, uint16_t *mid, int ffn, int cols, int T, cudaStream_t stream);
int mla_attend_tc_take_error(unsigned *out);
int launch_argmax_f32(const float *logits, int vocab, int pitch, int T, uint32_t *ids, cudaStream_t stream);

namespace {

constexpr int kHeadRows = 64;       // rows of the vocabulary product per call
constexpr int kShortPortion = 32;   // portions of up to this many tokens attend in the absorbed form
constexpr int kSyntheticBuckets = 32; // distance buckets of a model without stored weights
constexpr int kGemvAssignments = 64;  // up to this many (token, expert) pairs go through the mat-vec kernel

int pad(int n, int to) { return (n + to - 1) / to * to; }

struct Mat {
  uint16_t *w = nullptr;
  int R = 0, K = 0;  // padded; experts: R per expert
  CUtensorMap m128, m256;
};
struct Norm {
  float *w = nullptr, *b = nullptr, alpha = 0.f;
};
struct Hyper {
  float *in = nullptr, *out = nullptr, *mix = nullptr;
};
struct LayerState {
  Norm norm1, norm2;
  Hyper hc1, hc2;
  float *post1 = nullptr, *post2 = nullptr;  // sandwich: the norms behind the sublayers
  Mat qkvg, o;                       // linear; state: everything that is projected in; grouped: q, k, v (unless borrowed), gates
  float *decay_pow = nullptr, *norm_w = nullptr;
  LinearAttn lin;                    // sizes only
  LatentShape lat;                   // latent
  Mat dqkv, uq, kvb;
  uint16_t *wuk_t = nullptr;         // [heads, rank, dim]
  float *q_norm = nullptr, *kv_norm = nullptr;
  StateInputs inputs;                // state: sizes and weights
  int step_at = 0;                   // state: column of the step sizes
  GroupedShape grp;                  // grouped
  float *k_norm = nullptr;
  int gate_at = 0;                   // grouped: column of the head gates
  Mat up, down;                      // experts; dense: gate and up rows in `up`
  int *table = nullptr;
  ExpertPlan plan;
  int plan_index = -1;
};
struct Run {
  int layer = 0;
  float *state = nullptr;  // linear, state: [slots, heads, dim, vdim]
  void *pool = nullptr;    // latent, grouped: Act [pages, page_rows, row]; possibly an earlier run's
  void *ring = nullptr;    // state: Act [slots, taps, channels]
};

struct StackModel {
  StackSpec spec;
  bool f32 = false;
  int W = 0, V = 0;  // padded width and vocabulary
  std::vector<LayerState> layers;
  std::vector<Run> runs;
  uint16_t *embed = nullptr, *bigram = nullptr;
  double *turns = nullptr;       // sinusoid: turns per position of every pair of columns
  uint32_t *last_ids = nullptr;  // [slots] newest token
  Norm final_norm;
  Mat head;
  ExpertPlanArgs *plans_dev = nullptr;
  int n_plans = 0, max_top = 1;
  // step buffers (Act: bf16 or fp32)
  float *x = nullptr, *y = nullptr, *ckr = nullptr, *lin_o = nullptr, *chunk_state = nullptr, *logits = nullptr;
  float4 *token = nullptr;
  void *xbc = nullptr;
  void *h = nullptr, *proj = nullptr, *cq = nullptr, *q_abs = nullptr, *o_lat = nullptr, *mix = nullptr, *mid = nullptr, *h_final = nullptr,
       *h_sel = nullptr;
  float *part_o = nullptr, *part_ml = nullptr;  // parts of split contexts
  uint16_t *c_all = nullptr, *kr_all = nullptr, *kv_all = nullptr;
  int *sel_rows = nullptr;
  void *gemv_ws = nullptr;
  size_t gemv_ws_bytes = 0;
  float *splitk_ws = nullptr;
  size_t splitk_bytes = 0;
  std::map<std::pair<const void *, int>, CUtensorMap> x_maps;
  std::map<const void *, size_t> buffer_bytes;
};
StackModel *stack(blok_model *m) { return static_cast<StackModel *>(m->impl); }

// ---- weights ----

// Where the rows and columns of a stored matrix go: groups of `row_group` rows are `row_pad` apart, columns alike; inside a
// group, rows from `split` on start at `split_at`.
struct Place {
  int rows, row_group, row_pad, cols, col_group, col_pad, split, split_at;
  static Place plain(int rows, int cols) { return {rows, rows, rows, cols, cols, cols, rows, rows}; }
  static Place out_heads(int heads, int n, int padded, int cols) { return {heads * n, n, padded, cols, cols, cols, n, n}; }
  static Place in_heads(int rows, int heads, int n, int padded) { return {rows, rows, rows, heads * n, n, padded, rows, rows}; }
  // `groups` groups of two parts of a and b rows, padded to pa and pb
  static Place two_parts(int groups, int a, int pa, int b, int pb, int cols) { return {groups * (a + b), a + b, pa + pb, cols, cols, cols, a, pa}; }
  __host__ __device__ long row(long r) const {
    const int in = (int)(r % row_group);
    return r / row_group * row_pad + (in < split ? in : in - split + split_at);
  }
  __host__ __device__ int col(int c) const { return c / col_group * col_pad + c % col_group; }
};

__global__ void fill_placed_kernel(uint16_t *p, int ld, Place at, uint64_t key, float std) {
  const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= (size_t)at.rows * at.cols) return;
  p[at.row((long)(i / at.cols)) * ld + at.col((int)(i % at.cols))] = f32_to_bf16_bits(unit_normal(key, i) * std);
}

// out[h][c][d] = uk[h][d][c]
__global__ void transpose_heads_kernel(const uint16_t *__restrict__ uk, uint16_t *__restrict__ out, int heads, int dim, int rank) {
  const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x, n = (size_t)heads * rank * dim;
  if (i >= n) return;
  const int d = (int)(i % dim), c = (int)(i / dim % rank);
  const size_t h = i / ((size_t)dim * rank);
  out[i] = uk[(h * dim + d) * rank + c];
}

float bf16_value(uint16_t b) {
  const uint32_t u = (uint32_t)b << 16;
  float f;
  memcpy(&f, &u, 4);
  return f;
}

class Weights {
 public:
  Weights(blok_model *m, uint64_t seed) : m_(m), seed_(seed) {}
  int open(const char *dir) {
    if (!dir) return BLOK_OK;
    from_file_ = true;
    return file_.open(std::string(dir) + "/model.safetensors");
  }
  int zeroed(size_t bytes, void **out) {
    if (int rc = dev_alloc(m_, bytes, out)) return rc;
    BLOK_CUDA(cudaMemset(*out, 0, bytes ? bytes : 16));
    return BLOK_OK;
  }
  // `groups` matrices [R, K] behind one another (experts), or one.
  int make(Mat *t, int R, int K, int groups = 1) {
    t->R = R;
    t->K = K;
    void *p;
    // at least 256 rows, so that no copied box is taller than the matrix
    const size_t rows = std::max((size_t)groups * R, (size_t)256);
    if (int rc = zeroed(rows * K * 2, &p)) return rc;
    t->w = static_cast<uint16_t *>(p);
    if (m_->dtype == BLOK_DTYPE_F32) return BLOK_OK;
    if (int rc = gemm_operand_map(t->w, (long)rows, K, K, 128, &t->m128)) return rc;
    return gemm_operand_map(t->w, (long)rows, K, K, 256, &t->m256);
  }
  // The stored matrix `name` (or rows of it, see fill_rows) into rows row0.. of t.
  int fill(const Mat &t, long row0, const std::string &name, const Place &at, float std, long from = 0, long total = 0) {
    return fill_rows(t.w + (size_t)row0 * t.K, t.K, name, at, std, from, total);
  }
  // Of a stored matrix of `total` rows, those from `from` on (total 0: all of it).
  int fill_rows(uint16_t *dst, int ld, const std::string &name, const Place &at, float std, long from = 0, long total = 0) {
    if (!from_file_) {
      const size_t n = (size_t)at.rows * at.cols;
      fill_placed_kernel<<<(unsigned)((n + 255) / 256), 256>>>(dst, ld, at, next_key(), std);
      return launch_status("fill_placed_kernel");
    }
    const StoredTensor *t;
    if (int rc = file_.need(name, "BF16", {total ? total : at.rows, at.cols}, &t)) return rc;
    std::vector<uint16_t> raw((size_t)at.rows * at.cols);
    if (int rc = file_.read(*t, raw.data(), (uint64_t)from * at.cols * 2, raw.size() * 2)) return rc;
    const size_t prows = (size_t)at.row(at.rows - 1) + 1;
    std::vector<uint16_t> placed(prows * ld, 0);
    for (long r = 0; r < at.rows; ++r)
      for (int c = 0; c < at.cols; ++c) placed[(size_t)at.row(r) * ld + at.col(c)] = raw[(size_t)r * at.cols + c];
    BLOK_CUDA(cudaMemcpy(dst, placed.data(), placed.size() * 2, cudaMemcpyHostToDevice));
    return BLOK_OK;
  }
  // Rows of a stored matrix of `cols` columns; `synthetic` without a file.
  int stored_rows(const std::string &name, long cols, int synthetic, int *rows) {
    *rows = synthetic;
    if (!from_file_) return BLOK_OK;
    const StoredTensor *t = file_.find(name);
    BLOK_REQUIRE(t && t->shape.size() == 2 && t->shape[0] >= 1 && t->shape[0] < (1 << 20) && t->shape[1] == cols, BLOK_ERR_SHAPE,
                 "tensor %s is missing or has not %ld columns", name.c_str(), cols);
    *rows = (int)t->shape[0];
    return BLOK_OK;
  }
  int host_vector(const std::string &name, const std::vector<long> &shape, float mean, float dev, std::vector<float> *out) {
    long n = 1;
    for (long d : shape) n *= d;
    out->resize((size_t)n);
    if (!from_file_) {
      uint64_t k = next_key();
      for (float &v : *out) {
        k = k * 6364136223846793005ull + 1442695040888963407ull;
        v = mean + dev * ((float)(k >> 40) / 8388608.0f - 1.0f);
      }
      return BLOK_OK;
    }
    const StoredTensor *t;
    if (int rc = file_.need(name, "BF16", shape, &t)) return rc;
    std::vector<uint16_t> raw((size_t)n);
    if (int rc = file_.read(*t, raw.data())) return rc;
    for (long i = 0; i < n; ++i) (*out)[i] = bf16_value(raw[i]);
    return BLOK_OK;
  }
  int upload(const std::vector<float> &v, float **out) {
    if (int rc = dev_alloc_as(m_, v.size(), out)) return rc;
    BLOK_CUDA(cudaMemcpy(*out, v.data(), v.size() * 4, cudaMemcpyHostToDevice));
    return BLOK_OK;
  }
  // [n] as groups of `group` values `gpad` apart, zero in between and up to `total`.
  int vector(const std::string &name, int n, int group, int gpad, int total, float mean, float dev, float **out) {
    std::vector<float> v, p((size_t)total, 0.f);
    if (int rc = host_vector(name, {n}, mean, dev, &v)) return rc;
    for (int i = 0; i < n; ++i) p[i / group * gpad + i % group] = v[i];
    return upload(p, out);
  }
  int norm(const std::string &name, int width, int padded, bool dynamic_tanh, Norm *out) {
    std::vector<float> a;
    int rc;
    if (!dynamic_tanh) return vector(name, width, width, padded, padded, 1.f, 0.1f, &out->w);
    if ((rc = vector(name, width, width, padded, padded, 1.f, 0.1f, &out->w)) || (rc = vector(name + ".b", width, width, padded, padded, 0.f, 0.1f, &out->b)) ||
        (rc = host_vector(name + ".alpha", {}, 0.8f, 0.1f, &a)))
      return rc;
    out->alpha = a[0];
    return BLOK_OK;
  }
  int hyper(const std::string &name, int s, Hyper *out) {
    std::vector<float> mix;
    int rc;
    if ((rc = vector(name + ".in", s, s, s, s, 1.f / s, 0.1f, &out->in)) || (rc = vector(name + ".out", s, s, s, s, 1.f, 0.1f, &out->out)) ||
        (rc = host_vector(name + ".mix", {s, s}, 0.f, 0.05f, &mix)))
      return rc;
    if (!from_file_)
      for (int i = 0; i < s; ++i) mix[(size_t)i * s + i] += 0.9f;
    return upload(mix, &out->mix);
  }
  int table(const std::string &name, int vocab, int top, int experts, int **out) {
    std::vector<int> v((size_t)vocab * top);
    if (!from_file_) {
      for (int i = 0; i < vocab; ++i) {
        const uint64_t k = (seed_ + 1 + i) * 0x9e3779b97f4a7c15ull;
        const int step = 1 + (int)(k >> 20) % std::max(1, experts / top);  // distinct: top * step <= experts
        for (int j = 0; j < top; ++j) v[(size_t)i * top + j] = (int)(((k >> 40) + (uint64_t)j * step) % experts);
      }
    } else {
      const StoredTensor *t;
      if (int rc = file_.need(name, "I32", {vocab, top}, &t)) return rc;
      if (int rc = file_.read(*t, v.data())) return rc;
      for (int e : v) BLOK_REQUIRE(e >= 0 && e < experts, BLOK_ERR_ROUTE, "%s names expert %d of %d", name.c_str(), e, experts);
    }
    if (int rc = dev_alloc_as(m_, v.size(), out)) return rc;
    BLOK_CUDA(cudaMemcpy(*out, v.data(), v.size() * 4, cudaMemcpyHostToDevice));
    return BLOK_OK;
  }

 private:
  blok_model *m_;
  uint64_t seed_, counter_ = 0;
  bool from_file_ = false;
  Safetensors file_;
  uint64_t next_key() { return seed_ * 0x100000001b3ull + (++counter_) * 0x9e3779b97f4a7c15ull; }
};

#define TRY(call)                 \
  do {                            \
    if (int rc_ = (call)) return rc_; \
  } while (0)

float fan(int cols) { return 1.0f / std::sqrt((float)cols); }

int load_linear(blok_model *m, Weights &w, const std::string &p, const LinearMixer &x, LayerState &L) {
  StackModel *S = stack(m);
  const int W = S->spec.width, d = pad(x.dim, 16), dv = pad(x.vdim, 16), hd = x.heads * d, hv = x.heads * dv;
  BLOK_REQUIRE(d <= kLinMaxDim, BLOK_ERR_SHAPE, "%s: heads of %d keys, at most %d are supported", p.c_str(), x.dim, kLinMaxDim);
  L.lin.heads = x.heads;
  L.lin.dim = d;
  L.lin.vdim = dv;
  L.lin.silu_qkv = x.silu_qkv;
  L.lin.k_scale = (float)x.k_scale;
  TRY(w.make(&L.qkvg, 2 * hd + 2 * hv, S->W));
  TRY(w.fill(L.qkvg, 0, p + "q", Place::out_heads(x.heads, x.dim, d, W), fan(W)));
  TRY(w.fill(L.qkvg, hd, p + "k", Place::out_heads(x.heads, x.dim, d, W), fan(W)));
  TRY(w.fill(L.qkvg, 2 * hd, p + "v", Place::out_heads(x.heads, x.vdim, dv, W), fan(W)));
  TRY(w.fill(L.qkvg, 2 * hd + hv, p + "g", Place::out_heads(x.heads, x.vdim, dv, W), fan(W)));
  TRY(w.make(&L.o, S->W, pad(hv, 32)));
  TRY(w.fill(L.o, 0, p + "o", Place::in_heads(W, x.heads, x.vdim, dv), fan(hv)));
  if (x.norm_weight) TRY(w.vector(p + "norm", x.heads * x.vdim, x.vdim, dv, hv, 1.f, 0.1f, &L.norm_w));
  std::vector<float> pw((size_t)x.heads * (kLinChunk + 1));
  for (int h = 0; h < x.heads; ++h)
    for (int i = 0; i <= kLinChunk; ++i) pw[(size_t)h * (kLinChunk + 1) + i] = (float)std::pow(x.decay[h], i);
  return w.upload(pw, &L.decay_pow);
}

int load_latent(blok_model *m, Weights &w, const std::string &p, const LatentMixer &x, LayerState &L) {
  StackModel *S = stack(m);
  const int W = S->spec.width;
  LatentShape &s = L.lat;
  s.heads = x.heads;
  s.dim = pad(x.dim, 32);
  s.rot = pad(x.rot_dim, 32);
  s.vdim = pad(x.vdim, 16);
  s.rank = pad(x.kv_rank, 32);
  s.q_rank = pad(x.q_rank, 32);
  s.true_rot = x.rot_dim;
  s.true_rank = x.kv_rank;
  s.true_q_rank = x.q_rank;
  s.rot_dims = x.rot_dims;
  s.scale = (float)x.scale;
  s.eps = (float)S->spec.eps;
  std::vector<double> turns(x.rot_dims / 2 + 1);
  for (int i = 0; i < x.rot_dims / 2; ++i) turns[i] = std::pow(x.rot_base, -2.0 * i / x.rot_dims) / 6.28318530717958647693;
  double *turns_dev = nullptr;
  TRY(dev_alloc_as(m, turns.size(), &turns_dev));
  BLOK_CUDA(cudaMemcpy(turns_dev, turns.data(), turns.size() * sizeof(double), cudaMemcpyHostToDevice));
  s.turns = turns_dev;
  TRY(w.make(&L.dqkv, s.q_rank + s.row(), S->W));
  TRY(w.fill(L.dqkv, 0, p + "dq", Place::plain(x.q_rank, W), fan(W)));
  TRY(w.fill(L.dqkv, s.q_rank, p + "dkv", Place::two_parts(1, x.kv_rank, s.rank, x.rot_dim, s.rot, W), fan(W)));
  TRY(w.vector(p + "dq.norm", x.q_rank, x.q_rank, s.q_rank, s.q_rank, 1.f, 0.1f, &L.q_norm));
  TRY(w.vector(p + "dkv.norm", x.kv_rank, x.kv_rank, s.rank, s.rank, 1.f, 0.1f, &L.kv_norm));
  TRY(w.make(&L.uq, x.heads * s.head(), s.q_rank));
  TRY(w.fill(L.uq, 0, p + "uq", Place::two_parts(x.heads, x.dim, s.dim, x.rot_dim, s.rot, x.q_rank), fan(x.q_rank)));
  TRY(w.make(&L.kvb, x.heads * (s.dim + s.vdim), s.rank));
  TRY(w.fill(L.kvb, 0, p + "uk", Place::out_heads(x.heads, x.dim, s.dim, x.kv_rank), fan(x.kv_rank)));
  TRY(w.fill(L.kvb, (long)x.heads * s.dim, p + "uv", Place::out_heads(x.heads, x.vdim, s.vdim, x.kv_rank), fan(x.kv_rank)));
  const size_t n = (size_t)x.heads * s.rank * s.dim;
  TRY(dev_alloc_as(m, n, &L.wuk_t));
  transpose_heads_kernel<<<(unsigned)((n + 255) / 256), 256>>>(L.kvb.w, L.wuk_t, x.heads, s.dim, s.rank);
  TRY(launch_status("transpose_heads_kernel"));
  TRY(w.make(&L.o, S->W, pad(x.heads * s.vdim, 32)));
  return w.fill(L.o, 0, p + "o", Place::in_heads(W, x.heads, x.vdim, s.vdim), fan(x.heads * x.vdim));
}

int load_state(blok_model *m, Weights &w, const std::string &p, const StateMixer &x, LayerState &L) {
  StackModel *S = stack(m);
  const int W = S->spec.width, dv = pad(x.vdim, 16), n = pad(x.state, 16);
  const int inner = x.heads * x.vdim, hv = x.heads * dv, bc = x.groups * x.state, bcp = x.groups * n, channels = hv + 2 * bcp;
  BLOK_REQUIRE(n <= kLinMaxDim, BLOK_ERR_SHAPE, "%s: a state of %d rows, at most %d are supported", p.c_str(), x.state, kLinMaxDim);
  L.lin.heads = x.heads;
  L.lin.dim = n;
  L.lin.vdim = dv;
  L.lin.share = x.heads / x.groups;
  L.lin.v_first = true;
  L.step_at = 2 * hv + 2 * bcp;
  // z | x | B | C | steps
  const long total = 2l * inner + 2 * bc + x.heads;
  TRY(w.make(&L.qkvg, L.step_at + pad(x.heads, 16), S->W));
  TRY(w.fill(L.qkvg, 0, p + "in", Place::out_heads(2 * x.heads, x.vdim, dv, W), fan(W), 0, total));
  TRY(w.fill(L.qkvg, 2 * hv, p + "in", Place::out_heads(2 * x.groups, x.state, n, W), fan(W), 2l * inner, total));
  TRY(w.fill(L.qkvg, L.step_at, p + "in", Place::plain(x.heads, W), fan(W), 2l * inner + 2 * bc, total));
  TRY(w.make(&L.o, S->W, pad(hv, 32)));
  TRY(w.fill(L.o, 0, p + "o", Place::in_heads(W, x.heads, x.vdim, dv), fan(inner)));
  TRY(w.vector(p + "norm", inner, x.vdim, dv, hv, 1.f, 0.1f, &L.norm_w));
  std::vector<float> conv, bias, placed_conv((size_t)x.taps * channels, 0.f), placed_bias((size_t)channels, 0.f);
  TRY(w.host_vector(p + "conv", {inner + 2 * bc, x.taps}, 0.f, 1.f / std::sqrt((float)x.taps), &conv));
  TRY(w.host_vector(p + "conv.b", {inner + 2 * bc}, 0.f, 0.1f, &bias));
  for (int c = 0; c < inner + 2 * bc; ++c) {
    const int at = c < inner ? c / x.vdim * dv + c % x.vdim : hv + (c - inner) / x.state * n + (c - inner) % x.state;
    placed_bias[at] = bias[c];
    for (int j = 0; j < x.taps; ++j) placed_conv[(size_t)j * channels + at] = conv[(size_t)c * x.taps + j];
  }
  float *conv_w = nullptr, *conv_b = nullptr, *dt_bias = nullptr, *rate = nullptr, *skip = nullptr;
  TRY(w.upload(placed_conv, &conv_w));
  TRY(w.upload(placed_bias, &conv_b));
  std::vector<float> a;
  TRY(w.host_vector(p + "A_log", {x.heads}, 0.5f, 0.5f, &a));
  for (float &v : a) v = (float)-std::exp((double)v);
  TRY(w.upload(a, &rate));
  TRY(w.vector(p + "dt_bias", x.heads, x.heads, x.heads, x.heads, -3.f, 1.f, &dt_bias));
  TRY(w.vector(p + "D", x.heads, x.heads, x.heads, x.heads, 1.f, 0.2f, &skip));
  L.lin.skip = skip;
  StateInputs &s = L.inputs;
  s.heads = x.heads;
  s.channels = channels;
  s.taps = x.taps;
  s.conv_w = conv_w;
  s.conv_b = conv_b;
  s.dt_bias = dt_bias;
  s.rate = rate;
  s.ld = L.qkvg.R;
  s.first = hv;
  s.dt_at = L.step_at;
  return BLOK_OK;
}

// The bucket of a distance: itself below half of them, then logarithmic up to `top`.
int distance_bucket(int n, int buckets, double top) {
  const int half = buckets / 2;
  if (n < half) return n;
  const double at = std::log((double)n / half) / std::log(top / half) * (buckets - half);
  return std::min((double)(buckets - 1), half + std::floor(at));
}

int load_grouped(blok_model *m, Weights &w, const std::string &p, const GroupedMixer &x, LayerState &L) {
  StackModel *S = stack(m);
  const int W = S->spec.width;
  GroupedShape &s = L.grp;
  s.heads = x.heads;
  s.kv_heads = x.kv_heads;
  s.dim = pad(x.dim, 32);
  s.vdim = pad(x.vdim, 16);
  s.true_dim = x.dim;
  s.scale = (float)x.scale;
  s.eps = (float)S->spec.eps;
  const bool own = x.kv_from < 0;
  const int nq = x.heads * s.dim, nk = own ? x.kv_heads * s.dim : 0, nv = own ? x.kv_heads * s.vdim : 0;
  L.gate_at = nq + nk + nv;
  TRY(w.make(&L.qkvg, L.gate_at + (x.head_gate ? pad(x.heads, 16) : 0), S->W));
  TRY(w.fill(L.qkvg, 0, p + "q", Place::out_heads(x.heads, x.dim, s.dim, W), fan(W)));
  if (own) {
    TRY(w.fill(L.qkvg, nq, p + "k", Place::out_heads(x.kv_heads, x.dim, s.dim, W), fan(W)));
    TRY(w.fill(L.qkvg, nq + nk, p + "v", Place::out_heads(x.kv_heads, x.vdim, s.vdim, W), fan(W)));
  }
  if (x.head_gate) TRY(w.fill(L.qkvg, L.gate_at, p + "g", Place::plain(x.heads, W), fan(W)));
  if (x.qk_norm) {
    TRY(w.vector(p + "q.norm", x.heads * x.dim, x.dim, s.dim, nq, 1.f, 0.1f, &L.q_norm));
    if (own) TRY(w.vector(p + "k.norm", x.kv_heads * x.dim, x.dim, s.dim, nk, 1.f, 0.1f, &L.k_norm));
  }
  if (x.bias_max > 0) {
    int buckets = 0;
    TRY(w.stored_rows(p + "rel", x.heads, kSyntheticBuckets, &buckets));
    BLOK_REQUIRE(buckets >= 2 && x.bias_max > buckets / 2 && x.bias_max <= (1 << 24), BLOK_ERR_SHAPE, "%srel: %d buckets up to a distance of %g", p.c_str(),
                 buckets, x.bias_max);
    std::vector<float> rel, by_distance;
    TRY(w.host_vector(p + "rel", {buckets, x.heads}, 0.f, 0.5f, &rel));
    s.bias_len = 1;  // up to the first distance of the last bucket
    while (distance_bucket(s.bias_len - 1, buckets, x.bias_max) < buckets - 1) ++s.bias_len;
    by_distance.resize((size_t)x.heads * s.bias_len);
    for (int n = 0; n < s.bias_len; ++n) {
      const int b = distance_bucket(n, buckets, x.bias_max);
      for (int h = 0; h < x.heads; ++h) by_distance[(size_t)h * s.bias_len + n] = rel[(size_t)b * x.heads + h];
    }
    float *bias = nullptr;
    TRY(w.upload(by_distance, &bias));
    s.bias = bias;
  }
  TRY(w.make(&L.o, S->W, pad(x.heads * s.vdim, 32)));
  return w.fill(L.o, 0, p + "o", Place::in_heads(W, x.heads, x.vdim, s.vdim), fan(x.heads * x.vdim));
}

int load_mixer(blok_model *m, Weights &w, const std::string &p, const StackLayer &x, LayerState &L) {
  switch (x.kind) {
    case StackLayer::Linear: return load_linear(m, w, p, x.linear, L);
    case StackLayer::Latent: return load_latent(m, w, p, x.latent, L);
    case StackLayer::State: return load_state(m, w, p, x.state, L);
    case StackLayer::Grouped: return load_grouped(m, w, p, x.grouped, L);
  }
  return BLOK_ERR_STATE;
}

int load_dense(blok_model *m, Weights &w, const std::string &p, const DenseGated &x, LayerState &L) {
  StackModel *S = stack(m);
  const int W = S->spec.width, ff = pad(x.ff, 32);
  TRY(w.make(&L.up, 2 * ff, S->W));
  TRY(w.fill(L.up, 0, p + "gate", Place::plain(x.ff, W), fan(W)));
  TRY(w.fill(L.up, ff, p + "up", Place::plain(x.ff, W), fan(W)));
  TRY(w.make(&L.down, S->W, ff));
  return w.fill(L.down, 0, p + "down", Place::plain(W, x.ff), fan(x.ff));
}

int load_experts(blok_model *m, Weights &w, const std::string &p, const TableExperts &x, LayerState &L) {
  StackModel *S = stack(m);
  const int W = S->spec.width, ff = pad(x.ff, 32);
  BLOK_REQUIRE(x.experts <= kMaxTableExperts && x.top <= x.experts, BLOK_ERR_SHAPE, "%s: %d of %d experts (at most %d)", p.c_str(), x.top, x.experts,
               kMaxTableExperts);
  TRY(w.make(&L.up, ff, S->W, x.experts));
  TRY(w.make(&L.down, S->W, ff, x.experts));
  for (int e = 0; e < x.experts; ++e) {
    const std::string pe = p + "e" + std::to_string(e);
    TRY(w.fill(L.up, (long)e * ff, pe + ".up", Place::plain(x.ff, W), fan(W)));
    TRY(w.fill(L.down, (long)e * S->W, pe + ".down", Place::plain(W, x.ff), fan(x.ff)));
  }
  return w.table(p + "table", S->spec.vocab, x.top, x.experts, &L.table);
}

// A step buffer: zeroed, and remembered so that the copies of a product know how many rows it has.
template <typename T>
int buffer(blok_model *m, size_t bytes, T **out) {
  void *p = nullptr;
  bytes = std::max(bytes, (size_t)16);
  TRY(dev_alloc(m, bytes, &p));
  BLOK_CUDA(cudaMemset(p, 0, bytes));
  stack(m)->buffer_bytes[p] = bytes;
  *out = static_cast<T *>(p);
  return BLOK_OK;
}

// The tensor map of a step buffer read as rows of `cols` bf16.
int x_map(StackModel *S, const void *x, int cols, const CUtensorMap **out) {
  auto it = S->x_maps.find({x, cols});
  if (it == S->x_maps.end()) {
    auto b = S->buffer_bytes.find(x);
    BLOK_REQUIRE(b != S->buffer_bytes.end(), BLOK_ERR_STATE, "stack: not a step buffer");
    CUtensorMap map;
    TRY(gemm_operand_map(x, (long)(b->second / ((size_t)cols * 2)), cols, cols, kGtTileRows, &map));
    it = S->x_maps.emplace(std::make_pair(x, cols), map).first;
  }
  *out = &it->second;
  return BLOK_OK;
}

// y[T, W.R] = x[T, W.K] W^T; y Act, or fp32 with y_f32.  silu: *silu columns go through SiLU if the kernel that is picked can
// do that on the way; *silu becomes 0 then.
int product(StackModel *S, const Mat &w, const void *x, int T, void *y, bool y_f32, cudaStream_t stream, int *silu = nullptr) {
  if (S->f32) {
    GemmF32 g;
    g.w = w.w;
    g.x = static_cast<const float *>(x);
    g.y = static_cast<float *>(y);
    g.R = g.ldy = w.R;
    g.K = g.ldw = g.ldx = w.K;
    g.T = T;
    return launch_gemm_f32(g, stream);
  }
  const uint16_t *xb = static_cast<const uint16_t *>(x);
  uint16_t *yb = y_f32 ? nullptr : static_cast<uint16_t *>(y);
  float *yf = y_f32 ? static_cast<float *>(y) : nullptr;
  if (T <= 8) return launch_bf16_gemv_splitk(w.w, xb, yb, yf, w.R, w.K, T, S->gemv_ws, S->gemv_ws_bytes, stream);
  if (T <= kWgStreamTokens && w.K % 256 == 0 && w.R % 16 == 0)
    return launch_wgemm_rows(WG_BF16_PLAIN, w.w, nullptr, xb, yb, yf, w.R, w.K, T, S->splitk_ws, S->splitk_bytes, stream);
  GemmTma g;
  TRY(x_map(S, x, w.K, &g.x));
  g.w128 = &w.m128;
  g.w256 = &w.m256;
  g.T = T;
  g.R = g.ldo = w.R;
  g.K = w.K;
  g.out = y;
  g.out_f32 = y_f32;
  if (silu && *silu) {
    g.act = GEMM_ACT_SILU;
    g.act_cols = *silu;
    *silu = 0;
  }
  return launch_gemm_tma(g, stream);
}

}  // namespace

int stack_describe(blok_model *m, const StackSpec &spec) {
  BLOK_REQUIRE(spec.sandwich ? spec.streams == 1 : spec.embed_scale == 1 && !spec.bigram_buckets && !spec.sinusoid && spec.logit_scale == 1, BLOK_ERR_ARG,
               "this form of the residual does not go with the other values");
  for (const StackLayer &L : spec.layers)
    BLOK_REQUIRE(!spec.sandwich || L.ff_kind != StackLayer::Experts, BLOK_ERR_ARG, "experts do not go with sandwiched sublayers");
  BLOK_REQUIRE(spec.streams <= kMaxStreams && !spec.order.empty(), BLOK_ERR_SHAPE, "%d residual streams (at most %d), %zu layer runs", spec.streams,
               kMaxStreams, spec.order.size());
  StackModel *S = new (std::nothrow) StackModel();
  BLOK_REQUIRE(S, BLOK_ERR_ARG, "out of host memory");
  S->spec = spec;
  S->f32 = m->dtype == BLOK_DTYPE_F32;
  S->W = pad(spec.width, 32);
  S->V = pad(spec.vocab, 16);
  m->impl = S;
  m->cfg.layers = (int)spec.layers.size();
  m->cfg.hidden = spec.width;
  m->cfg.vocab = spec.vocab;
  m->layer_runs = (int)spec.order.size();
  return BLOK_OK;
}

void stack_destroy(blok_model *m) {
  delete stack(m);
  m->impl = nullptr;
}

int stack_build(blok_model *m, const char *dir, uint64_t seed) {
  StackModel *S = stack(m);
  const StackSpec &spec = S->spec;
  const blok_model_config &c = m->cfg;
  Weights w(m, seed);
  TRY(w.open(dir));
  void *p;
  TRY(w.zeroed((size_t)spec.vocab * S->W * 2, &p));
  S->embed = static_cast<uint16_t *>(p);
  TRY(w.fill_rows(S->embed, S->W, "embed", Place::plain(spec.vocab, spec.width), 1.0f));
  if (spec.bigram_buckets) {
    TRY(w.zeroed(((size_t)spec.bigram_buckets + 1) * S->W * 2, &p));
    S->bigram = static_cast<uint16_t *>(p);
    TRY(w.fill_rows(S->bigram, S->W, "bigram", Place::plain(spec.bigram_buckets + 1, spec.width), 1.0f));
    TRY(w.zeroed((size_t)c.max_batch * 4, &p));
    S->last_ids = static_cast<uint32_t *>(p);
  }
  if (spec.sinusoid) {
    std::vector<double> turns((size_t)S->W / 2);
    for (int i = 0; i < S->W / 2; ++i) turns[i] = std::pow(10000.0, -2.0 * i / spec.width) / 6.28318530717958647693;
    TRY(dev_alloc_as(m, turns.size(), &S->turns));
    BLOK_CUDA(cudaMemcpy(S->turns, turns.data(), turns.size() * sizeof(double), cudaMemcpyHostToDevice));
  }
  if (spec.sandwich) {  // the logits' scale rides on the last norm
    std::vector<float> f, padded((size_t)S->W, 0.f);
    TRY(w.host_vector("final.norm", {spec.width}, 1.f, 0.1f, &f));
    for (int i = 0; i < spec.width; ++i) padded[i] = (float)(f[i] * spec.logit_scale);
    TRY(w.upload(padded, &S->final_norm.w));
  } else {
    TRY(w.norm("final.norm", spec.width, S->W, true, &S->final_norm));
  }
  TRY(w.make(&S->head, S->V, S->W));
  TRY(w.fill(S->head, 0, "head", Place::plain(spec.vocab, spec.width), fan(spec.width)));
  S->layers.resize(spec.layers.size());
  for (size_t i = 0; i < spec.layers.size(); ++i) {
    const StackLayer &x = spec.layers[i];
    LayerState &L = S->layers[i];
    const std::string pl = "l" + std::to_string(i) + ".";
    TRY(w.norm(pl + "norm1", spec.width, S->W, !spec.sandwich, &L.norm1));
    if (spec.sandwich) TRY(w.vector(pl + "norm1b", spec.width, spec.width, S->W, S->W, 1.f, 0.1f, &L.post1));
    else TRY(w.hyper(pl + "hc1", spec.streams, &L.hc1));
    TRY(load_mixer(m, w, pl + "mix.", x, L));
    if (x.ff_kind != StackLayer::NoFf) {
      TRY(w.norm(pl + "norm2", spec.width, S->W, !spec.sandwich, &L.norm2));
      if (spec.sandwich) TRY(w.vector(pl + "norm2b", spec.width, spec.width, S->W, S->W, 1.f, 0.1f, &L.post2));
      else TRY(w.hyper(pl + "hc2", spec.streams, &L.hc2));
      TRY(x.ff_kind == StackLayer::Dense ? load_dense(m, w, pl + "mlp.", x.dense, L) : load_experts(m, w, pl + "mlp.", x.ff, L));
      if (x.ff_kind == StackLayer::Experts) S->max_top = std::max(S->max_top, x.ff.top);
    }
  }

  // caches and states: one per run
  const size_t esz = S->f32 ? 4 : 2, N = (size_t)m->rows;
  std::vector<void *> pool_of(spec.layers.size(), nullptr);
  for (int l : spec.order) {
    Run r;
    r.layer = l;
    const StackLayer &x = spec.layers[l];
    const LayerState &L = S->layers[l];
    const size_t rows = (size_t)c.kv_pages * c.kv_page_rows;
    switch (x.kind) {
      case StackLayer::State:
        TRY(w.zeroed((size_t)c.max_batch * L.inputs.taps * L.inputs.channels * esz, &r.ring));
        // fall through
      case StackLayer::Linear:
        TRY(dev_alloc_as(m, (size_t)c.max_batch * L.lin.heads * L.lin.dim * L.lin.vdim, &r.state));
        break;
      case StackLayer::Latent:
        TRY(dev_alloc(m, rows * L.lat.row() * esz, &r.pool));
        break;
      case StackLayer::Grouped:  // finite from the start: whole boxes are copied from it
        if (x.grouped.kv_from >= 0) r.pool = pool_of[x.grouped.kv_from];
        else TRY(w.zeroed(rows * L.grp.row() * esz, &r.pool));
        BLOK_REQUIRE(r.pool, BLOK_ERR_STATE, "layer %d has no keys to borrow", l);
        break;
    }
    pool_of[l] = r.pool;
    S->runs.push_back(r);
  }

  // step buffers, sized for the largest layer
  size_t proj = 1, ckr = 1, cq = 1, q_abs = 1, o_lat = 1, lin_o = 1, mixw = 1, mid = 1, chunk_state = 1, part_o = 1, part_ml = 1, c_all = 1, kr_all = 1, kv_all = 1, xbc = 1, token = 1;
  int max_R = S->V;
  std::vector<const Mat *> mats = {&S->head};
  for (size_t i = 0; i < spec.layers.size(); ++i) {
    const StackLayer &x = spec.layers[i];
    const LayerState &L = S->layers[i];
    mats.push_back(&L.o);
    mixw = std::max(mixw, (size_t)L.o.K);
    if (x.kind == StackLayer::Grouped) {
      const GroupedShape &s = L.grp;
      mats.push_back(&L.qkvg);
      proj = std::max(proj, (size_t)L.qkvg.R);
      const int short_rows = !S->f32 && grouped_prompt_supports(s) ? std::min(m->rows, std::max(c.max_batch, kShortPortion)) : m->rows;
      const size_t parts = S->f32 ? 0 : grouped_attend_max_parts(s, short_rows, c.max_ctx);
      part_o = std::max(part_o, parts * s.heads * s.vdim);
      part_ml = std::max(part_ml, parts * s.heads * 2);
    } else if (x.kind == StackLayer::Linear || x.kind == StackLayer::State) {
      mats.push_back(&L.qkvg);
      proj = std::max(proj, (size_t)L.qkvg.R);
      if (x.kind == StackLayer::State) {
        xbc = std::max(xbc, (size_t)L.inputs.channels);
        token = std::max(token, (size_t)L.inputs.heads);
      }
      lin_o = std::max(lin_o, (size_t)L.lin.heads * L.lin.vdim);
      if (!S->f32) chunk_state = std::max(chunk_state, linear_chunk_scratch_bytes(L.lin.heads, L.lin.dim, L.lin.vdim, c.prefill_chunk));
    } else {
      const LatentShape &s = L.lat;
      mats.push_back(&L.dqkv);
      mats.push_back(&L.uq);
      proj = std::max(proj, (size_t)L.uq.R);
      ckr = std::max(ckr, (size_t)L.dqkv.R);
      cq = std::max(cq, (size_t)s.q_rank);
      const bool prompt = !S->f32 && latent_prompt_supports(s);
      const int short_rows = prompt ? std::min(m->rows, std::max(c.max_batch, kShortPortion)) : m->rows;
      q_abs = std::max(q_abs, (size_t)short_rows * s.heads * s.row());
      o_lat = std::max(o_lat, (size_t)short_rows * s.heads * s.rank);
      const size_t parts = S->f32 ? 0 : latent_attend_max_parts(s, short_rows, c.max_ctx);
      part_o = std::max(part_o, parts * s.heads * s.rank);
      part_ml = std::max(part_ml, parts * s.heads * 2);
      if (prompt && c.prefill_chunk > kShortPortion) {
        const size_t ctx = pad(c.max_ctx, kGtTileRows);
        c_all = std::max(c_all, ctx * s.rank);
        kr_all = std::max(kr_all, ctx * s.rot);
        kv_all = std::max(kv_all, ctx * L.kvb.R);
      }
    }
    if (x.ff_kind == StackLayer::Experts) mid = std::max(mid, (size_t)x.ff.top * pad(x.ff.ff, 32));
    if (x.ff_kind == StackLayer::Dense) {
      mats.push_back(&L.down);
      mid = std::max(mid, (size_t)L.down.K);
      if (S->f32) proj = std::max(proj, (size_t)L.up.R);
      S->splitk_bytes = std::max(S->splitk_bytes, wgemm_splitk_bytes(WG_BF16_SWIGLU, L.up.K, L.down.K, kWgStreamTokens));
    }
  }
  for (const Mat *t : mats) {
    max_R = std::max(max_R, t->R);
    S->splitk_bytes = std::max(S->splitk_bytes, wgemm_splitk_bytes(WG_BF16_PLAIN, t->K, t->R, kWgStreamTokens));
  }
  const size_t slack = kGtTileRows;  // a product's last tile copies whole boxes of rows
  TRY(buffer(m, N * spec.streams * S->W * 4, &S->x));
  TRY(buffer(m, N * S->max_top * S->W * 4, &S->y));
  TRY(buffer(m, (N * S->max_top + slack) * S->W * esz, &S->h));
  TRY(buffer(m, (N + slack) * proj * esz, &S->proj));
  TRY(buffer(m, N * ckr * 4, &S->ckr));
  TRY(buffer(m, (N + slack) * cq * esz, &S->cq));
  TRY(buffer(m, q_abs * esz, &S->q_abs));
  TRY(buffer(m, o_lat * esz, &S->o_lat));
  TRY(buffer(m, part_o * 4, &S->part_o));
  TRY(buffer(m, part_ml * 4, &S->part_ml));
  TRY(buffer(m, N * lin_o * 4, &S->lin_o));
  TRY(buffer(m, N * xbc * esz, &S->xbc));
  TRY(buffer(m, N * token * sizeof(float4), &S->token));
  TRY(buffer(m, chunk_state, &S->chunk_state));
  TRY(buffer(m, (N + slack) * mixw * esz, &S->mix));
  TRY(buffer(m, (N + slack) * mid * esz, &S->mid));
  TRY(buffer(m, (N + slack) * S->W * esz, &S->h_final));
  TRY(buffer(m, (kHeadRows + slack) * S->W * esz, &S->h_sel));
  TRY(buffer(m, (size_t)kHeadRows * S->V * 4, &S->logits));
  TRY(buffer(m, kHeadRows * 4, &S->sel_rows));
  TRY(buffer(m, c_all * 2, &S->c_all));
  TRY(buffer(m, kr_all * 2, &S->kr_all));
  TRY(buffer(m, kv_all * 2, &S->kv_all));
  S->gemv_ws_bytes = bf16_gemv_splitk_workspace_bytes(pad(max_R, 16));
  TRY(buffer(m, S->gemv_ws_bytes, &S->gemv_ws));
  TRY(buffer(m, S->splitk_bytes, &S->splitk_ws));

  // expert plans, one per layer
  std::vector<ExpertPlanArgs> plans;
  for (size_t i = 0; i < spec.layers.size(); ++i) {
    if (spec.layers[i].ff_kind != StackLayer::Experts || S->f32) continue;
    LayerState &L = S->layers[i];
    const TableExperts &x = spec.layers[i].ff;
    const int tiles = expert_plan_max_tiles(m->rows * x.top, x.experts);
    int *t = nullptr;
    TRY(dev_alloc_as(m, (size_t)m->rows * x.top + 3 * (size_t)tiles + 1, &t));
    L.plan.at = t;
    L.plan.tile_expert = t + (size_t)m->rows * x.top;
    L.plan.tile_start = L.plan.tile_expert + tiles;
    L.plan.tile_count = L.plan.tile_start + tiles;
    L.plan.num_tiles = L.plan.tile_count + tiles;
    L.plan_index = (int)plans.size();
    ExpertPlanArgs a;
    a.table = L.table;
    a.experts = x.experts;
    a.top = x.top;
    a.plan = L.plan;
    plans.push_back(a);
  }
  S->n_plans = (int)plans.size();
  if (S->n_plans) {
    TRY(dev_alloc_as(m, plans.size(), &S->plans_dev));
    BLOK_CUDA(cudaMemcpy(S->plans_dev, plans.data(), plans.size() * sizeof(ExpertPlanArgs), cudaMemcpyHostToDevice));
  }
  TRY(alloc_serving_state(m));
  BLOK_CUDA(cudaDeviceSynchronize());
  return BLOK_OK;
}

namespace {

struct Call {  // of one step or chunk
  blok_model *m;
  StackModel *S;
  int T;
  bool chunk;
  StackRows rows;
  cudaStream_t stream;
};

// S->h -> S->y: the linear-attention mixer of a run.
int run_linear(const Call &c, const LinearMixer &x, const LayerState &L, const Run &r) {
  StackModel *S = c.S;
  const int hd = L.lin.heads * L.lin.dim, hv = L.lin.heads * L.lin.vdim;
  int silu = L.lin.silu_qkv ? 2 * hd + hv : 0;
  TRY(product(S, L.qkvg, S->h, c.T, S->proj, false, c.stream, &silu));
  LinearAttn a = L.lin;
  a.silu_qkv = silu != 0;
  a.qkvg = S->proj;
  a.ld = L.qkvg.R;
  a.f32 = S->f32;
  a.decay_pow = L.decay_pow;
  a.state = r.state;
  a.o = S->lin_o;
  a.chunk_state = S->chunk_state;
  if (c.chunk) TRY(launch_linear_chunk(a, c.m->chunk_slot, c.m->host_pos[c.m->chunk_slot], c.T, c.stream));
  else TRY(launch_linear_step(a, c.rows, c.T, c.stream));
  GatedNorm g;
  g.heads = L.lin.heads;
  g.vdim = L.lin.vdim;
  g.true_vdim = x.vdim;
  g.per_head = x.norm_per_head;
  g.w = L.norm_w;
  g.eps = (float)S->spec.eps;
  g.gate = x.gate;
  g.o = S->lin_o;
  g.g = static_cast<const char *>(S->proj) + (size_t)(2 * hd + hv) * (S->f32 ? 4 : 2);
  g.ldg = L.qkvg.R;
  g.out = S->mix;
  g.ldo = L.o.K;
  g.f32 = S->f32;
  TRY(launch_gated_norm(g, c.T, c.stream));
  return product(S, L.o, S->mix, c.T, S->y, true, c.stream);
}

// One product per head: y[t, h, :] = W_h x[t, h, :].
int head_product(const Call &c, const uint16_t *w, long w_head, const void *x, long x_tok, long x_head, void *y, long y_tok, long y_head, int rows,
                 int cols, int heads) {
  if (!c.S->f32)
    return launch_head_gemv(w, w_head, static_cast<const uint16_t *>(x), x_tok, x_head, static_cast<uint16_t *>(y), y_tok, y_head, rows, cols, heads,
                            c.T, c.stream);
  GemmF32 g;
  g.w = w;
  g.x = static_cast<const float *>(x);
  g.y = static_cast<float *>(y);
  g.R = rows;
  g.K = g.ldw = cols;
  g.T = c.T;
  g.ldx = (int)x_tok;
  g.ldy = (int)y_tok;
  g.batch = heads;
  g.w_stride = w_head;
  g.x_stride = x_head;
  g.y_stride = y_head;
  return launch_gemm_f32(g, c.stream);
}

int run_latent(const Call &c, const LayerState &L, const Run &r) {
  StackModel *S = c.S;
  const LatentShape &s = L.lat;
  TRY(product(S, L.dqkv, S->h, c.T, S->ckr, true, c.stream));
  TRY(launch_latent_append(s, S->ckr, L.q_norm, L.kv_norm, c.rows, c.T, S->cq, r.pool, S->f32, c.stream));
  TRY(product(S, L.uq, S->cq, c.T, S->proj, false, c.stream));
  if (c.chunk && c.T > kShortPortion && !S->f32 && latent_prompt_supports(s)) {
    const int slot = c.m->chunk_slot, n = (int)c.m->host_pos[slot] + c.T;
    TRY(launch_latent_rotate(s, S->proj, c.rows, c.T, S->proj, s.head(), s.dim, false, c.stream));
    TRY(launch_latent_gather(s, static_cast<const uint16_t *>(r.pool), c.rows, slot, n, S->c_all, S->kr_all, c.stream));
    GemmTma g;
    TRY(x_map(S, S->c_all, s.rank, &g.x));
    g.w128 = &L.kvb.m128;
    g.w256 = &L.kvb.m256;
    g.T = n;
    g.R = g.ldo = L.kvb.R;
    g.K = s.rank;
    g.out = S->kv_all;
    TRY(launch_gemm_tma(g, c.stream));
    TRY(launch_latent_prompt(s, static_cast<const uint16_t *>(S->proj), S->kv_all, S->kr_all, c.T, n, static_cast<uint16_t *>(S->mix), L.o.K, c.stream));
  } else {
    const int row = s.row();
    TRY(launch_latent_rotate(s, S->proj, c.rows, c.T, S->q_abs, row, s.rank, S->f32, c.stream));
    TRY(head_product(c, L.wuk_t, (long)s.rank * s.dim, S->proj, (long)s.heads * s.head(), s.head(), S->q_abs, (long)s.heads * row, row, s.rank, s.dim,
                     s.heads));
    TRY(launch_latent_attend(s, S->q_abs, r.pool, c.rows, c.T, c.m->cfg.max_ctx, S->o_lat, S->f32, S->part_o, S->part_ml, c.stream));
    TRY(head_product(c, L.kvb.w + (size_t)s.heads * s.dim * s.rank, (long)s.vdim * s.rank, S->o_lat, (long)s.heads * s.rank, s.rank, S->mix, L.o.K,
                     s.vdim, s.vdim, s.rank, s.heads));
  }
  return product(S, L.o, S->mix, c.T, S->y, true, c.stream);
}

// S->h -> S->y: a selective state space.
int run_state(const Call &c, const StateMixer &x, const LayerState &L, const Run &r) {
  StackModel *S = c.S;
  TRY(product(S, L.qkvg, S->h, c.T, S->proj, false, c.stream));
  StateInputs in = L.inputs;
  in.proj = S->proj;
  in.f32 = S->f32;
  in.ring = r.ring;
  in.out = S->xbc;
  in.token = S->token;
  in.token_ld = c.m->rows;
  TRY(launch_state_inputs(in, c.rows, c.T, c.chunk, c.stream));
  LinearAttn a = L.lin;
  a.qkvg = S->xbc;
  a.ld = in.channels;
  a.f32 = S->f32;
  a.token = S->token;
  a.token_ld = in.token_ld;
  a.state = r.state;
  a.o = S->lin_o;
  a.chunk_state = S->chunk_state;
  if (c.chunk) TRY(launch_linear_chunk(a, c.m->chunk_slot, c.m->host_pos[c.m->chunk_slot], c.T, c.stream));
  else TRY(launch_linear_step(a, c.rows, c.T, c.stream));
  GatedNorm g;
  g.heads = x.heads;
  g.vdim = L.lin.vdim;
  g.true_vdim = x.vdim;
  g.w = L.norm_w;
  g.eps = (float)S->spec.eps;
  g.o = S->lin_o;
  g.g = S->proj;
  g.ldg = L.qkvg.R;
  g.out = S->mix;
  g.ldo = L.o.K;
  g.f32 = S->f32;
  TRY(launch_gate_then_norm(g, x.norm_groups, c.T, c.stream));
  return product(S, L.o, S->mix, c.T, S->y, true, c.stream);
}

template <typename Act>
GroupedQuery<Act> grouped_query(const StackModel *S, const GroupedMixer &x, const LayerState &L) {
  GroupedQuery<Act> q;
  q.q = static_cast<const Act *>(S->proj);
  q.ldq = L.qkvg.R;
  if (x.head_gate) q.gate = q.q + L.gate_at;
  q.ld_gate = L.qkvg.R;
  q.out = static_cast<Act *>(S->mix);
  q.ldo = L.o.K;
  return q;
}

// S->h -> S->y: grouped attention.
int run_grouped(const Call &c, const GroupedMixer &x, const LayerState &L, const Run &r) {
  StackModel *S = c.S;
  const GroupedShape &s = L.grp;
  TRY(product(S, L.qkvg, S->h, c.T, S->proj, false, c.stream));
  if (x.qk_norm || x.kv_from < 0)
    TRY(launch_grouped_append(s, S->proj, L.qkvg.R, L.q_norm, L.k_norm, c.rows, c.T, x.kv_from < 0 ? r.pool : nullptr, S->f32, c.stream));
  if (S->f32) {
    TRY(launch_grouped_attend_f32(s, grouped_query<float>(S, x, L), r.pool, c.rows, c.T, c.stream));
  } else if (c.chunk && c.T > kShortPortion && grouped_prompt_supports(s)) {
    const int slot = c.m->chunk_slot, n = (int)c.m->host_pos[slot] + c.T;
    const long rows = (long)c.m->cfg.kv_pages * c.m->cfg.kv_page_rows;
    TRY(launch_grouped_prompt(s, grouped_query<uint16_t>(S, x, L), r.pool, rows, c.rows, slot, c.T, n, c.stream));
  } else {
    TRY(launch_grouped_attend(s, grouped_query<uint16_t>(S, x, L), r.pool, c.rows, c.T, c.m->cfg.max_ctx, S->part_o, S->part_ml, c.stream));
  }
  return product(S, L.o, S->mix, c.T, S->y, true, c.stream);
}

int run_mixer(const Call &c, const StackLayer &x, const LayerState &L, const Run &r) {
  switch (x.kind) {
    case StackLayer::Linear: return run_linear(c, x.linear, L, r);
    case StackLayer::Latent: return run_latent(c, L, r);
    case StackLayer::State: return run_state(c, x.state, L, r);
    case StackLayer::Grouped: return run_grouped(c, x.grouped, L, r);
  }
  return BLOK_ERR_STATE;
}

// S->h -> S->y: the gated feed-forward.
int run_dense(const Call &c, const LayerState &L) {
  StackModel *S = c.S;
  const int ff = L.down.K;
  const uint16_t *h = static_cast<const uint16_t *>(S->h), *up = L.up.w + (size_t)ff * L.up.K;
  uint16_t *mid = static_cast<uint16_t *>(S->mid);
  if (S->f32) {
    TRY(product(S, L.up, S->h, c.T, S->proj, false, c.stream));
    TRY(launch_swiglu_f32(static_cast<const float *>(S->proj), static_cast<float *>(S->mid), ff, c.T, c.stream));
  } else if (c.T <= 8 && ((size_t)L.up.K * 2 + 64) * c.T <= 200 * 1024) {
    TRY(launch_bf16_gateup(L.up.w, up, h, mid, ff, L.up.K, c.T, c.stream));
  } else if (c.T > 8 && c.T <= kWgStreamTokens && L.up.K % 256 == 0) {
    TRY(launch_wgemm_rows(WG_BF16_SWIGLU, L.up.w, up, h, mid, nullptr, ff, L.up.K, c.T, S->splitk_ws, S->splitk_bytes, c.stream));
  } else {
    GemmTma g;
    TRY(x_map(S, S->h, L.up.K, &g.x));
    g.w128 = &L.up.m128;
    g.T = c.T;
    g.R = g.ldo = g.up_row = ff;
    g.K = L.up.K;
    g.act = GEMM_ACT_SWIGLU;
    g.out = mid;
    TRY(launch_gemm_tma(g, c.stream));
  }
  return product(S, L.down, S->mid, c.T, S->y, true, c.stream);
}

bool planned(const StackModel *S, int T, int top) { return !S->f32 && T * top > kGemvAssignments; }

// S->h (in expert order when planned) -> S->y, one row per assignment.
int run_experts(const Call &c, const TableExperts &x, const LayerState &L) {
  StackModel *S = c.S;
  if (!planned(S, c.T, x.top)) {
    const uint32_t *ids = c.m->ids;
    TRY(launch_expert_gemv(L.up.w, L.up.R, L.up.K, L.table, ids, S->spec.vocab, x.top, c.T, S->h, S->f32, true, true, S->mid, S->f32, c.stream));
    return launch_expert_gemv(L.down.w, L.down.R, L.down.K, L.table, ids, S->spec.vocab, x.top, c.T, S->mid, S->f32, false, false, S->y, true, c.stream);
  }
  GemmTma g;
  g.tile_expert = L.plan.tile_expert;
  g.tile_start = L.plan.tile_start;
  g.tile_count = L.plan.tile_count;
  g.num_tiles = L.plan.num_tiles;
  g.T = c.T * x.top;
  g.max_tiles = expert_plan_max_tiles(g.T, x.experts);
  TRY(x_map(S, S->h, L.up.K, &g.x));
  g.w128 = &L.up.m128;
  g.w256 = &L.up.m256;
  g.R = g.ldo = L.up.R;
  g.K = L.up.K;
  g.act = GEMM_ACT_RELU2;
  g.out = S->mid;
  TRY(launch_gemm_tma(g, c.stream));
  TRY(x_map(S, S->mid, L.down.K, &g.x));
  g.w128 = &L.down.m128;
  g.w256 = &L.down.m256;
  g.R = g.ldo = L.down.R;
  g.K = L.down.K;
  g.act = GEMM_ACT_NONE;
  g.out = S->y;
  g.out_f32 = true;
  return launch_gemm_tma(g, c.stream);
}

// The layers around one residual with a norm on both sides of every sublayer.
int sandwich_layers(const Call &c) {
  blok_model *m = c.m;
  StackModel *S = c.S;
  const StackSpec &spec = S->spec;
  ResidualNorm a;
  a.T = c.T;
  a.width = S->W;
  a.true_width = spec.width;
  a.x = S->x;
  a.embed = S->embed;
  a.vocab = spec.vocab;
  a.embed_scale = (float)spec.embed_scale;
  a.bigram = S->bigram;
  a.buckets = spec.bigram_buckets;
  a.mul_prev = spec.bigram_mul_prev;
  a.mul_cur = spec.bigram_mul_cur;
  a.turns = S->turns;
  a.last_ids = S->last_ids;
  a.pos = c.rows.pos;
  a.slot_of = c.rows.slot_of;
  a.chunk = c.chunk;
  a.mult = (float)spec.residual_mult;
  a.eps = (float)spec.eps;
  a.h = S->h;
  a.h_f32 = S->f32;
  a.ids = m->ids;
  auto step = [&](const Norm &n) {
    a.norm_w = n.w;
    const int rc = launch_residual_norm(a, c.stream);
    a.ids = nullptr;
    a.copy = nullptr;
    a.y = S->y;
    return rc;
  };
  for (size_t i = 0; i < S->runs.size(); ++i) {
    const Run &r = S->runs[i];
    const StackLayer &x = spec.layers[r.layer];
    const LayerState &L = S->layers[r.layer];
    TRY(step(L.norm1));
    TRY(run_mixer(c, x, L, r));
    a.post_w = L.post1;
    if (x.ff_kind == StackLayer::Dense) {
      TRY(step(L.norm2));
      TRY(run_dense(c, L));
      a.post_w = L.post2;
    }
    if (m->trace && c.T <= m->trace_rows) a.copy = m->trace + i * (size_t)m->trace_rows * spec.width;
  }
  a.h = S->h_final;
  if (S->last_ids) a.keep_ids = m->ids;
  return step(S->final_norm);
}

}  // namespace

int stack_layers(blok_model *m, int T, bool chunk, blok_stream_t stream_) {
  StackModel *S = stack(m);
  const StackSpec &spec = S->spec;
  Call c;
  c.m = m;
  c.S = S;
  c.T = T;
  c.chunk = chunk;
  c.stream = (cudaStream_t)stream_;
  c.rows.slot_of = m->slot_of;
  c.rows.pos = m->ctx_b;
  c.rows.table = m->table_dev;
  c.rows.table_stride = m->table_stride;
  c.rows.page_rows = m->cfg.kv_page_rows;
  if (spec.sandwich) return sandwich_layers(c);
  if (S->n_plans) {
    bool any = false;
    for (const StackLayer &L : spec.layers) any = any || (L.ff_kind == StackLayer::Experts && planned(S, T, L.ff.top));
    if (any) TRY(launch_expert_plan(S->plans_dev, S->n_plans, m->ids, spec.vocab, T, c.stream));
  }
  // what the streams have still to take in
  StreamsStep a;
  a.T = T;
  a.width = S->W;
  a.streams = spec.streams;
  a.x = S->x;
  a.ids = m->ids;
  a.embed = S->embed;
  a.vocab = spec.vocab;
  a.h = S->h;
  a.h_f32 = S->f32;
  a.true_width = spec.width;
  auto step = [&](const float *in, const Norm &n) {
    a.in = in;
    a.norm_w = n.w;
    a.norm_b = n.b;
    a.alpha = n.alpha;
    const int rc = launch_streams_step(a, c.stream);
    a.ids = nullptr;
    a.copies = 1;
    a.copy_at = nullptr;
    a.sum = nullptr;
    return rc;
  };
  auto took = [&](const Hyper &h, int parts, const int *part_at) {  // a sublayer left its output in S->y
    a.y_rows = S->y;
    a.parts = parts;
    a.part_at = part_at;
    a.part_scale = 1.0f / (float)parts;
    a.mix = h.mix;
    a.out = h.out;
  };
  for (size_t i = 0; i < S->runs.size(); ++i) {
    const Run &r = S->runs[i];
    const StackLayer &x = spec.layers[r.layer];
    const LayerState &L = S->layers[r.layer];
    TRY(step(L.hc1.in, L.norm1));
    TRY(run_mixer(c, x, L, r));
    took(L.hc1, 1, nullptr);
    if (x.ff_kind == StackLayer::Experts) {
      const bool plan = planned(S, T, x.ff.top);
      if (plan) {
        a.copies = x.ff.top;
        a.copy_at = L.plan.at;
      }
      TRY(step(L.hc2.in, L.norm2));
      TRY(run_experts(c, x.ff, L));
      took(L.hc2, x.ff.top, plan ? L.plan.at : nullptr);
    } else if (x.ff_kind == StackLayer::Dense) {
      TRY(step(L.hc2.in, L.norm2));
      TRY(run_dense(c, L));
      took(L.hc2, 1, nullptr);
    }
    if (m->trace && T <= m->trace_rows) a.sum = m->trace + i * (size_t)m->trace_rows * spec.width;
  }
  a.h = S->h_final;
  a.store_x = false;
  return step(nullptr, S->final_norm);
}

int stack_sample(blok_model *m, int row, int n, uint32_t *next, blok_stream_t stream) {
  StackModel *S = stack(m);
  const char *h = static_cast<const char *>(S->h_final) + (size_t)row * S->W * (S->f32 ? 4 : 2);
  BLOK_REQUIRE(n <= kHeadRows && (row == 0 || n <= 8 || S->f32), BLOK_ERR_SHAPE, "sample: %d rows from row %d", n, row);
  TRY(product(S, S->head, h, n, S->logits, true, (cudaStream_t)stream));
  return launch_argmax_f32(S->logits, S->spec.vocab, S->V, n, next, (cudaStream_t)stream);
}

// Row i of dst is row rows[i] of src; `bytes` per row, a multiple of 16.
__global__ void select_rows_kernel(const uint4 *__restrict__ src, const int *__restrict__ rows, int units, uint4 *__restrict__ dst) {
  for (int u = threadIdx.x; u < units; u += blockDim.x) dst[(size_t)blockIdx.x * units + u] = src[(size_t)rows[blockIdx.x] * units + u];
}

int stack_logits(blok_model *m, const int *rows, int n, float *out, blok_stream_t stream_) {
  StackModel *S = stack(m);
  cudaStream_t stream = (cudaStream_t)stream_;
  const int units = (int)((size_t)S->W * (S->f32 ? 4 : 2) / 16);
  for (int i = 0; i < n; i += kHeadRows) {
    const int k = std::min(kHeadRows, n - i);
    BLOK_CUDA(cudaMemcpyAsync(S->sel_rows, rows + i, (size_t)k * 4, cudaMemcpyHostToDevice, stream));
    select_rows_kernel<<<k, 128, 0, stream>>>(static_cast<const uint4 *>(S->h_final), S->sel_rows, units, static_cast<uint4 *>(S->h_sel));
    TRY(launch_status("select_rows_kernel"));
    TRY(product(S, S->head, S->h_sel, k, S->logits, true, stream));
    const size_t wide = (size_t)S->spec.vocab * 4;
    BLOK_CUDA(cudaMemcpy2DAsync(out + (size_t)i * S->spec.vocab, wide, S->logits, (size_t)S->V * 4, wide, k, cudaMemcpyDeviceToHost, stream));
    BLOK_CUDA(cudaStreamSynchronize(stream));
  }
  return BLOK_OK;
}

int stack_check(blok_model *, blok_stream_t stream) {
  BLOK_CUDA(cudaStreamSynchronize((cudaStream_t)stream));
  unsigned err = 0;
  TRY(gemm_tma_take_error(&err));
  BLOK_REQUIRE(!err, BLOK_ERR_TIMEOUT, "a product gave up on a barrier");
  TRY(prompt_attn_take_error(&err));
  BLOK_REQUIRE(!err, BLOK_ERR_TIMEOUT, "attention over a prompt gave up on a barrier");
  TRY(mla_attend_tc_take_error(&err));
  BLOK_REQUIRE(!err, BLOK_ERR_TIMEOUT, "the attention core gave up on wait %u", err);
  return BLOK_OK;
}

}  // namespace blok
