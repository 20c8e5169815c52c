// Kimi's model: MLA attention over a latent cache and INT4 routed experts (config 4), with seeded synthetic weights or a
// materialised checkpoint.  Reference: generate() and its `run` lambda, src/kimi_exec.cu:780-893 (per-layer body
// :803-878, sampler :880-881).  Weights are resident in HBM; the reference re-reads every tile from storage on every
// use (:608-649).  The serving state around it (slots, pages, steps, generation) is in model.cu.
#include <algorithm>
#include <cstring>
#include <map>
#include <new>
#include <string>
#include <vector>

#include "model.h"
#include "synth_fill.cuh"
#include "wgemm.h"

namespace blok {

// Expert-parallel decode (every rank holds the same rows): the weighted sum of the selected experts THIS rank holds,
// unrounded, rows of experts held elsewhere skipped; the ranks' sums are added by one all-reduce per layer.
__global__ void sharded_partial_kernel(const uint16_t *__restrict__ y_assign, const float *__restrict__ wts,
                                       const int *__restrict__ local_ids, int n_local, int hidden, int topk, float *__restrict__ part) {
  const int t = blockIdx.y;
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * 2;
  if (c >= hidden) return;
  float o0 = 0.f, o1 = 0.f;
  for (int k = 0; k < topk; ++k) {
    const int e = local_ids[(size_t)t * topk + k];
    if (e < 0 || e >= n_local) continue;
    const uint32_t v = *reinterpret_cast<const uint32_t *>(y_assign + ((size_t)t * topk + k) * hidden + c);
    const float w = wts[(size_t)t * topk + k];
    o0 = fmaf(bf16lo(v), w, o0);
    o1 = fmaf(bf16hi(v), w, o1);
  }
  *reinterpret_cast<float2 *>(part + (size_t)t * hidden + c) = make_float2(o0, o1);
}
// out = bf16(bf16(routed sum) + shared), the rounding points of src/kimi_exec.cu:871 and :684.
__global__ void sharded_finish_kernel(const float *__restrict__ part, const uint16_t *__restrict__ shared, int hidden,
                                      uint16_t *__restrict__ out) {
  const int t = blockIdx.y;
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * 2;
  if (c >= hidden) return;
  const float2 v = *reinterpret_cast<const float2 *>(part + (size_t)t * hidden + c);
  float o0 = round_bf16(v.x), o1 = round_bf16(v.y);
  if (shared) {
    const uint32_t s = *reinterpret_cast<const uint32_t *>(shared + (size_t)t * hidden + c);
    o0 = round_bf16(o0 + bf16lo(s));
    o1 = round_bf16(o1 + bf16hi(s));
  }
  *reinterpret_cast<uint32_t *>(out + (size_t)t * hidden + c) = pack_bf16x2(o0, o1);
}

int launch_bf16_gemv(const uint16_t *w, const uint16_t *x, uint16_t *y_bf16, float *y_f32, int rows, int cols, int T,
                     cudaStream_t stream);
int launch_router_topk(const float *logits, const float *bias, int T, int experts, int topk, float routed_scale,
                       uint16_t *ids, float *wts, int *local_ids, int expert_base, cudaStream_t stream);

struct Tensor {
  void *ptr = nullptr;
  size_t bytes = 0;
};

struct LayerWeights {
  std::map<std::string, Tensor> t;
  blok_mla_layer_t *mla = nullptr;
  blok_moe_layer_t *moe = nullptr;
  uint16_t *cache = nullptr;  // [max_batch, max_ctx, kv_rank + qk_rope], or the page pool [kv_pages, kv_page_rows, ...]
};

struct KimiModel {
  std::vector<LayerWeights> layers;
  std::map<std::string, Tensor> top;
  // step buffers
  uint16_t *x = nullptr, *n = nullptr, *tmp = nullptr;  // [rows, hidden]
  bool moe_batched_ok = false;                          // the layer sizes fit the grouped-GEMM kernels
  void *mlp_ws = nullptr;
  size_t mlp_ws_bytes = 0;
  int mlp_rows = 8;            // rows of the dense layer per call
  void *head_ws = nullptr;
  size_t head_ws_bytes = 0;
  uint64_t seed = 0, counter = 0;
  // expert parallelism (cfg.ep_world > 1): this rank holds experts [ep_base, ep_base + ep_local) of every MoE layer
  blok_comm_t *comm = nullptr;
  int ep_base = 0, ep_local = 0;
  float *ep_logits = nullptr;   // [rows, experts]
  float *ep_sk = nullptr;       // K-split partial sums of the router logits over 9..64 rows
  size_t ep_sk_bytes = 0;
  uint16_t *ep_ids = nullptr;   // [rows, topk]
  int *ep_local_ids = nullptr;  // [rows, topk] id - ep_base (outside [0, ep_local): held by another rank)
  int *ep_rows = nullptr;       // [rows * topk] row of assignment a: a / topk
  float *ep_wts = nullptr;      // [rows, topk]
  uint16_t *ep_y = nullptr;     // [rows * topk, hidden] outputs of the assignments held here
  float *ep_part = nullptr;     // [rows, hidden] this rank's weighted sum, then the sum over the ranks
  uint16_t *ep_shared = nullptr;  // [rows, hidden]
};

}  // namespace blok

using namespace blok;

static KimiModel *kimi(blok_model *m) { return static_cast<KimiModel *>(m->impl); }

namespace {
enum Fill { F_NORMAL, F_ABS, F_ONE, F_WORDS, F_F32 };

int make_tensor(blok_model *m, std::map<std::string, Tensor> &into, const char *name, size_t elems, Fill fill, float std,
                size_t first = 0) {
  size_t esz = (fill == F_WORDS || fill == F_F32) ? 4 : 2;
  Tensor t;
  t.bytes = elems * esz;
  int rc = dev_alloc(m, t.bytes, &t.ptr);
  if (rc) return rc;
  const uint64_t key = kimi(m)->seed * 0x100000001b3ull + (++kimi(m)->counter) * 0x9e3779b97f4a7c15ull;
  const unsigned blocks = (unsigned)((elems + 255) / 256);
  if (elems) {
    if (fill == F_WORDS) fill_words_kernel<<<blocks, 256>>>(static_cast<uint32_t *>(t.ptr), elems, key, first);
    else if (fill == F_F32) fill_f32_kernel<<<blocks, 256>>>(static_cast<float *>(t.ptr), elems, key, std);
    else fill_bf16_kernel<<<blocks, 256>>>(static_cast<uint16_t *>(t.ptr), elems, key, fill == F_ONE ? 1.0f : std,
                                           fill == F_ONE ? 2 : (fill == F_ABS ? 1 : 0), first);
    rc = launch_status("synthetic fill");
    if (rc) return rc;
  }
  into[name] = t;
  return BLOK_OK;
}

template <typename T>
T *tp(const std::map<std::string, Tensor> &m, const char *name) {
  auto it = m.find(name);
  return it == m.end() ? nullptr : static_cast<T *>(it->second.ptr);
}


int build(blok_model *m, const char *, uint64_t) {
  KimiModel *K = kimi(m);
  const blok_model_config &c = m->cfg;
  m->rows = c.max_batch > c.prefill_chunk ? c.max_batch : c.prefill_chunk;
  const int world = c.ep_world > 1 ? c.ep_world : 1;
  K->ep_local = c.experts / world;
  K->ep_base = (world > 1 ? c.ep_rank : 0) * K->ep_local;
  // the grouped-GEMM form of the MoE layer (blok_moe_batched) serves prefill chunks and steps of more than 8 sequences
  K->moe_batched_ok = m->rows > 1 && c.first_dense < c.layers && c.hidden % 512 == 0 && c.inter % 512 == 0 &&
                      c.experts % 128 == 0 && c.shared_inter % 512 == 0;
  const size_t H = c.hidden;
  const float wstd = 0.006f;
  int rc;
#define MK(map, name, elems, fill, std) \
  if ((rc = make_tensor(m, map, name, (size_t)(elems), fill, std))) return rc;
  MK(K->top, "embed_tokens", (size_t)c.vocab * H, F_NORMAL, wstd);
  MK(K->top, "norm", H, F_ONE, 1.f);
  MK(K->top, "lm_head", (size_t)c.vocab * H, F_NORMAL, wstd);
  K->layers.resize(c.layers);
  const int qk_head = c.qk_nope + c.qk_rope, lat_w = c.kv_rank + c.qk_rope;
  for (int l = 0; l < c.layers; ++l) {
    auto &t = K->layers[l].t;
    MK(t, "input_layernorm", H, F_ONE, 1.f);
    MK(t, "post_attention_layernorm", H, F_ONE, 1.f);
    MK(t, "q_a_proj", (size_t)c.q_rank * H, F_NORMAL, wstd);
    MK(t, "q_a_layernorm", c.q_rank, F_ONE, 1.f);
    MK(t, "q_b_proj", (size_t)c.heads * qk_head * c.q_rank, F_NORMAL, wstd);
    MK(t, "kv_a_proj_with_mqa", (size_t)lat_w * H, F_NORMAL, wstd);
    MK(t, "kv_a_layernorm", c.kv_rank, F_ONE, 1.f);
    MK(t, "kv_b_proj", (size_t)c.heads * (c.qk_nope + c.v_head) * c.kv_rank, F_NORMAL, wstd);
    MK(t, "o_proj", H * (size_t)c.heads * c.v_head, F_NORMAL, wstd);
    if (l < c.first_dense) {
      MK(t, "gate_proj", (size_t)c.dense_inter * H, F_NORMAL, wstd);
      MK(t, "up_proj", (size_t)c.dense_inter * H, F_NORMAL, wstd);
      MK(t, "down_proj", H * (size_t)c.dense_inter, F_NORMAL, wstd);
    } else {
      const size_t E = c.experts, I = c.inter;
      const size_t El = K->ep_local, E0 = K->ep_base;  // this rank's experts; the values are those of the whole tensor
      MK(t, "router", E * H, F_NORMAL, wstd);
      MK(t, "router_bias", E, F_F32, 0.01f);
#define MKE(name, per_expert, fill, std) \
  if ((rc = make_tensor(m, t, name, El * (size_t)(per_expert), fill, std, E0 * (size_t)(per_expert)))) return rc;
      MKE("gate_w", I * (H / 8), F_WORDS, 0.f);
      MKE("gate_s", I * (H / 32), F_ABS, 0.003f);
      MKE("up_w", I * (H / 8), F_WORDS, 0.f);
      MKE("up_s", I * (H / 32), F_ABS, 0.003f);
      MKE("down_w", H * (I / 8), F_WORDS, 0.f);
      MKE("down_s", H * (I / 32), F_ABS, 0.003f);
#undef MKE
      if (c.shared_inter) {
        MK(t, "shared_gate", (size_t)c.shared_inter * H, F_NORMAL, wstd);
        MK(t, "shared_up", (size_t)c.shared_inter * H, F_NORMAL, wstd);
        MK(t, "shared_down", H * (size_t)c.shared_inter, F_NORMAL, wstd);
      }
    }
    void *cache = nullptr;
    const size_t cache_rows = c.kv_page_rows > 0 ? (size_t)c.kv_pages * c.kv_page_rows : (size_t)c.max_batch * c.max_ctx;
    if ((rc = dev_alloc(m, cache_rows * lat_w * 2, &cache))) return rc;
    K->layers[l].cache = static_cast<uint16_t *>(cache);
  }
#undef MK
  BLOK_CUDA(cudaDeviceSynchronize());
  for (int l = 0; l < c.layers; ++l) {
    auto &L = K->layers[l];
    blok_mla_weights mw;
    memset(&mw, 0, sizeof(mw));
    mw.hidden = c.hidden; mw.heads = c.heads; mw.qk_nope = c.qk_nope; mw.qk_rope = c.qk_rope; mw.v_head = c.v_head;
    mw.q_rank = c.q_rank; mw.kv_rank = c.kv_rank; mw.rms_eps = c.rms_eps; mw.rope_theta = c.rope_theta;
    mw.yarn_factor = c.yarn_factor; mw.yarn_beta_fast = c.yarn_beta_fast; mw.yarn_beta_slow = c.yarn_beta_slow;
    mw.yarn_original_ctx = c.yarn_original_ctx; mw.yarn_mscale_all_dim = c.yarn_mscale_all_dim;
    mw.q_a = tp<uint16_t>(L.t, "q_a_proj"); mw.q_a_ln = tp<uint16_t>(L.t, "q_a_layernorm");
    mw.q_b = tp<uint16_t>(L.t, "q_b_proj"); mw.kv_a = tp<uint16_t>(L.t, "kv_a_proj_with_mqa");
    mw.kv_a_ln = tp<uint16_t>(L.t, "kv_a_layernorm"); mw.kv_b = tp<uint16_t>(L.t, "kv_b_proj");
    mw.o = tp<uint16_t>(L.t, "o_proj");
    if ((rc = blok_mla_layer_create(&mw, m->rows, c.max_ctx, &L.mla))) return rc;
    if (l >= c.first_dense) {
      blok_moe_weights ew;
      memset(&ew, 0, sizeof(ew));
      ew.hidden = c.hidden; ew.inter = c.inter; ew.experts = c.experts; ew.topk = c.topk; ew.shared_inter = c.shared_inter;
      ew.routed_scale = c.routed_scale; ew.router_w = tp<uint16_t>(L.t, "router");
      ew.router_bias = tp<float>(L.t, "router_bias"); ew.expert_base = K->ep_base; ew.experts_local = K->ep_local;
      ew.gate_w = tp<uint32_t>(L.t, "gate_w"); ew.gate_s = tp<uint16_t>(L.t, "gate_s");
      ew.up_w = tp<uint32_t>(L.t, "up_w"); ew.up_s = tp<uint16_t>(L.t, "up_s");
      ew.down_w = tp<uint32_t>(L.t, "down_w"); ew.down_s = tp<uint16_t>(L.t, "down_s");
      ew.shared_gate = tp<uint16_t>(L.t, "shared_gate"); ew.shared_up = tp<uint16_t>(L.t, "shared_up");
      ew.shared_down = tp<uint16_t>(L.t, "shared_down");
      // a sharded layer always runs its experts through the grouped kernels, which need the batched scratch
      const int moe_rows = world > 1 ? (m->rows > 2 ? m->rows : 2) : (K->moe_batched_ok ? m->rows : 1);
      if ((rc = blok_moe_layer_create(&ew, moe_rows, &L.moe))) return rc;
    }
  }
  void *p;
  const size_t act = (size_t)m->rows * c.hidden * 2;
  if ((rc = dev_alloc(m, act, &p))) return rc; K->x = static_cast<uint16_t *>(p);
  if ((rc = dev_alloc(m, act, &p))) return rc; K->n = static_cast<uint16_t *>(p);
  if ((rc = dev_alloc(m, act, &p))) return rc; K->tmp = static_cast<uint16_t *>(p);
  // the dense layer takes up to 64 rows per call where its sizes fit the weight-streaming kernel, else 8
  K->mlp_rows = (c.hidden % 256 == 0 && c.dense_inter % 256 == 0 && c.dense_inter > 0) ? std::min((int)m->rows, kWgStreamTokens) : 8;
  K->mlp_ws_bytes = blok_bf16_mlp_workspace_bytes(c.hidden, c.dense_inter > 0 ? c.dense_inter : 32, std::max(K->mlp_rows, 8));
  if ((rc = dev_alloc(m, K->mlp_ws_bytes, &K->mlp_ws))) return rc;
  K->head_ws_bytes = blok_lm_head_workspace_bytes(c.vocab, c.max_batch);
  if ((rc = dev_alloc(m, K->head_ws_bytes, &K->head_ws))) return rc;
  if (world > 1) {
    if ((rc = dev_alloc(m, (size_t)m->rows * c.experts * 4, &p))) return rc; K->ep_logits = static_cast<float *>(p);
    K->ep_sk_bytes = wgemm_splitk_bytes(WG_BF16_PLAIN, c.hidden, c.experts, std::min((int)m->rows, kWgStreamTokens));
    if ((rc = dev_alloc(m, std::max(K->ep_sk_bytes, (size_t)16), &p))) return rc; K->ep_sk = static_cast<float *>(p);
    if ((rc = dev_alloc(m, (size_t)m->rows * c.topk * 2, &p))) return rc; K->ep_ids = static_cast<uint16_t *>(p);
    if ((rc = dev_alloc(m, (size_t)m->rows * c.topk * 4, &p))) return rc; K->ep_local_ids = static_cast<int *>(p);
    if ((rc = dev_alloc(m, (size_t)m->rows * c.topk * 4, &p))) return rc; K->ep_wts = static_cast<float *>(p);
    if ((rc = dev_alloc(m, (size_t)m->rows * c.topk * 4, &p))) return rc; K->ep_rows = static_cast<int *>(p);
    {
      std::vector<int> rows_of((size_t)m->rows * c.topk);
      for (size_t a = 0; a < rows_of.size(); ++a) rows_of[a] = (int)(a / c.topk);
      BLOK_CUDA(cudaMemcpy(K->ep_rows, rows_of.data(), rows_of.size() * 4, cudaMemcpyHostToDevice));
    }
    if ((rc = dev_alloc(m, (size_t)m->rows * c.topk * c.hidden * 2, &p))) return rc; K->ep_y = static_cast<uint16_t *>(p);
    if ((rc = dev_alloc(m, (size_t)m->rows * c.hidden * 4, &p))) return rc; K->ep_part = static_cast<float *>(p);
    if ((rc = dev_alloc(m, (size_t)m->rows * c.hidden * 2, &p))) return rc; K->ep_shared = static_cast<uint16_t *>(p);
  }
  return alloc_serving_state(m);
}

}  // namespace

static int layers(blok_model *m, int T, bool chunk, blok_stream_t stream);
static int sample(blok_model *m, int row, int n, uint32_t *next, blok_stream_t stream);
static int check(blok_model *m, blok_stream_t stream);
static void destroy(blok_model *m);
// Weights come from blok_model_create_synthetic and blok_model_load_index: no config.json.
static const ModelFamily kKimiFamily = {"KimiK2", kMaxBatch, nullptr, build, destroy, layers, sample, nullptr, check};
static const FamilyRegistration kKimiRegistered(&kKimiFamily);

// The family's state, or NULL (and the error message) for a model of another family.
static KimiModel *kimi_of(blok_model *m, const char *who) {
  if (m && m->family == &kKimiFamily) return kimi(m);
  set_error("%s: %s", who, m ? "not a Kimi model" : "null pointer");
  return nullptr;
}

extern "C" void blok_model_default_config(blok_model_config *c) {
  if (!c) return;
  memset(c, 0, sizeof(*c));
  c->layers = 61; c->first_dense = 1; c->hidden = 7168; c->vocab = 163840; c->dense_inter = 18432;
  c->inter = 2048; c->experts = 384; c->topk = 8; c->shared_inter = 2048; c->routed_scale = 2.827f;
  c->heads = 64; c->qk_nope = 128; c->qk_rope = 64; c->v_head = 128; c->q_rank = 1536; c->kv_rank = 512;
  c->rms_eps = 1.0e-5f; c->final_rms_eps = 1.0e-5f;
  c->rope_theta = 50000.0f; c->yarn_factor = 64.0f; c->yarn_beta_fast = 32.0f; c->yarn_beta_slow = 1.0f;
  c->yarn_original_ctx = 4096.0f; c->yarn_mscale_all_dim = 1.0f;
  c->max_batch = 1; c->max_ctx = 1024; c->eos_id = 163586u;
}

extern "C" int blok_model_create_synthetic(const blok_model_config *cfg, uint64_t seed, blok_model_t **out) {
  BLOK_REQUIRE(cfg && out, BLOK_ERR_ARG, "blok_model_create_synthetic: null pointer");
  BLOK_REQUIRE(cfg->layers >= 1 && cfg->first_dense >= 0 && cfg->first_dense <= cfg->layers && cfg->vocab > 0 &&
                   cfg->hidden % 256 == 0 && cfg->max_batch >= 1 && cfg->max_batch <= kMaxBatch && cfg->max_ctx >= 1 &&
                   cfg->prefill_chunk >= 0 && cfg->prefill_chunk <= kMaxBatch,
               BLOK_ERR_SHAPE, "blok_model_create_synthetic: unsupported configuration");
  BLOK_REQUIRE(cfg->kv_page_rows == 0 || (cfg->kv_page_rows >= 32 && cfg->kv_page_rows % 32 == 0 && cfg->kv_pages >= 1),
               BLOK_ERR_SHAPE, "blok_model_create_synthetic: kv_page_rows %d must be 0 or a multiple of 32 with kv_pages >= 1",
               cfg->kv_page_rows);
  BLOK_REQUIRE(cfg->first_dense == 0 || (cfg->dense_inter > 0 && cfg->dense_inter % 32 == 0), BLOK_ERR_SHAPE,
               "blok_model_create_synthetic: dense_inter %d must be a positive multiple of 32", cfg->dense_inter);
  BLOK_REQUIRE(cfg->ep_world <= 1 || (cfg->ep_rank >= 0 && cfg->ep_rank < cfg->ep_world && cfg->experts % cfg->ep_world == 0 &&
                                       cfg->hidden % 512 == 0 && cfg->inter % 512 == 0 && cfg->kv_page_rows == 0),
               BLOK_ERR_SHAPE, "blok_model_create_synthetic: expert parallelism needs 0 <= ep_rank < ep_world, experts divisible "
                               "by ep_world, hidden and inter multiples of 512 and a dense cache");
  blok_model *m = new (std::nothrow) blok_model();
  KimiModel *K = new (std::nothrow) KimiModel();
  if (!m || !K) {
    delete m;
    delete K;
    set_error("blok_model_create_synthetic: out of host memory");
    return BLOK_ERR_ARG;
  }
  m->family = &kKimiFamily;
  m->impl = K;
  m->cfg = *cfg;
  // a step's launches are replayed from a CUDA graph, the all-reduces of a sharded model among them (measured on 2 GPUs:
  // 5.7 ms against 6.3 ms per token eagerly); BLOK_MODEL_GRAPH=0 keeps every launch eager
  if (const char *g = getenv("BLOK_MODEL_GRAPH")) m->graphs_enabled = strcmp(g, "0") != 0;
  K->seed = seed;
  if (int rc = build(m, nullptr, seed)) {
    blok_model_destroy(m);
    return rc;
  }
  *out = m;
  return BLOK_OK;
}

extern "C" int blok_model_tensor(blok_model_t *m, int layer, const char *name, void **ptr, size_t *bytes) {
  KimiModel *K = kimi_of(m, "blok_model_tensor");
  if (!K) return BLOK_ERR_STATE;
  BLOK_REQUIRE(name && ptr && bytes, BLOK_ERR_ARG, "blok_model_tensor: null pointer");
  const std::map<std::string, Tensor> *map = nullptr;
  if (layer == -1) map = &K->top;
  else if (layer >= 0 && layer < (int)K->layers.size()) map = &K->layers[layer].t;
  BLOK_REQUIRE(map, BLOK_ERR_ARG, "blok_model_tensor: layer %d out of range", layer);
  auto it = map->find(name);
  BLOK_REQUIRE(it != map->end(), BLOK_ERR_ARG, "blok_model_tensor: layer %d has no tensor '%s'", layer, name);
  *ptr = it->second.ptr;
  *bytes = it->second.bytes;
  return BLOK_OK;
}

extern "C" int blok_model_hidden(blok_model_t *m, const blok_bf16_t **ptr, int *rows) {
  KimiModel *K = kimi_of(m, "blok_model_hidden");
  if (!K) return BLOK_ERR_STATE;
  BLOK_REQUIRE(m && ptr && rows, BLOK_ERR_ARG, "blok_model_hidden: null pointer");
  *ptr = K->n;
  *rows = m->rows;
  return BLOK_OK;
}

extern "C" int blok_model_refresh_derived(blok_model_t *m) {
  KimiModel *K = kimi_of(m, "blok_model_refresh_derived");
  if (!K) return BLOK_ERR_STATE;
  BLOK_REQUIRE(m, BLOK_ERR_ARG, "blok_model_refresh_derived: null pointer");
  for (auto &L : K->layers)
    if (L.mla)
      if (int rc = blok_mla_layer_refresh(L.mla)) return rc;
  return BLOK_OK;
}

extern "C" int blok_model_set_comm(blok_model_t *m, blok_comm_t *comm) {
  KimiModel *K = kimi_of(m, "blok_model_set_comm");
  if (!K) return BLOK_ERR_STATE;
  BLOK_REQUIRE(m && comm, BLOK_ERR_ARG, "blok_model_set_comm: null pointer");
  BLOK_REQUIRE(m->cfg.ep_world > 1 && blok_comm_world(comm) == m->cfg.ep_world && blok_comm_rank(comm) == m->cfg.ep_rank, BLOK_ERR_STATE,
               "blok_model_set_comm: the communicator is rank %d of %d, the model was created as rank %d of %d", blok_comm_rank(comm),
               blok_comm_world(comm), m->cfg.ep_rank, m->cfg.ep_world);
  K->comm = comm;
  return BLOK_OK;
}

static int check(blok_model *m, blok_stream_t stream) {
  KimiModel *K = kimi(m);
  int first = BLOK_OK;
  std::string message;
  for (size_t l = 0; l < K->layers.size(); ++l) {
    auto &L = K->layers[l];
    int rc = L.moe ? blok_moe_layer_check(L.moe, stream) : BLOK_OK;
    if (rc == BLOK_OK && L.mla) rc = blok_mla_layer_check(L.mla, stream);
    if (rc != BLOK_OK && first == BLOK_OK) {  // keep checking: every layer's error word is cleared by its check
      first = rc;
      message = "layer " + std::to_string(l) + ": " + blok_last_error();
    }
  }
  if (first == BLOK_OK && K->comm) return blok_comm_check(K->comm);
  if (first != BLOK_OK) set_error("%s", message.c_str());
  return first;
}

extern "C" int blok_model_debug_set_layer_error(blok_model_t *m, int layer, unsigned code, blok_stream_t stream) {
  KimiModel *K = kimi_of(m, "blok_model_debug_set_layer_error");
  if (!K) return BLOK_ERR_STATE;
  BLOK_REQUIRE(layer >= 0 && layer < (int)K->layers.size() && K->layers[layer].moe, BLOK_ERR_ARG,
               "blok_model_debug_set_layer_error: layer %d is not a MoE layer of this model", layer);
  return blok_moe_layer_debug_set_error(K->layers[layer].moe, code, stream);
}

// The MoE layer with the experts split over the ranks, for T rows that every rank holds alike (the attention block is
// replicated): route (replicated, so all ranks agree without talking), run the selected experts this rank holds, add the
// ranks' weighted sums with ONE all-reduce, round, add the shared expert (replicated).  K->n -> K->tmp.
static int moe_sharded_rows(blok_model_t *m, blok::LayerWeights &L, int T, blok_stream_t stream_) {
  KimiModel *K = kimi(m);
  const blok_model_config &c = m->cfg;
  cudaStream_t stream = (cudaStream_t)stream_;
  BLOK_REQUIRE(K->comm, BLOK_ERR_STATE, "blok_model_step: a model with ep_world > 1 needs blok_model_set_comm first");
  const uint16_t *router = tp<uint16_t>(L.t, "router");
  int rc;
  const dim3 grid((c.hidden / 2 + 255) / 256, T);
  if (T <= 3 && blok_moe_layer_has_partial(L.moe)) {
    // steps of up to three sequences: one launch per row does the router, the shared expert and this rank's selected
    // experts (measured on 2 GPUs, 9 layers: 3.0 ms against 3.6 ms through the grouped kernels at batch 2, 4.5 against 4.0
    // at batch 4)
    for (int b = 0; b < T; ++b)
      if ((rc = blok_moe_decode_partial(L.moe, K->n + (size_t)b * c.hidden, K->ep_part + (size_t)b * c.hidden,
                                        K->ep_shared + (size_t)b * c.hidden, nullptr, nullptr, stream_)))
        return rc;
    if ((rc = blok_comm_all_reduce_f32(K->comm, K->ep_part, (long)T * c.hidden, stream_))) return rc;
    sharded_finish_kernel<<<grid, 256, 0, stream>>>(K->ep_part, K->ep_shared, c.hidden, K->tmp);
    return launch_status("sharded_finish_kernel");
  }
  // router logits (fp32): 9..64 rows in one pass of the weight-streaming kernel where the sizes fit it, else 8 rows at a time
  const bool stream_rows = T > 8 && c.experts % 16 == 0 && c.hidden % 256 == 0;
  for (int t0 = 0; t0 < T; t0 += stream_rows ? kWgStreamTokens : 8) {
    const int nrows = std::min(T - t0, stream_rows ? kWgStreamTokens : 8);
    rc = nrows > 8 ? launch_wgemm_rows(WG_BF16_PLAIN, router, nullptr, K->n + (size_t)t0 * c.hidden, nullptr, K->ep_logits + (size_t)t0 * c.experts,
                                       c.experts, c.hidden, nrows, K->ep_sk, K->ep_sk_bytes, stream)
                   : launch_bf16_gemv(router, K->n + (size_t)t0 * c.hidden, nullptr, K->ep_logits + (size_t)t0 * c.experts, c.experts, c.hidden,
                                      nrows, stream);
    if (rc) return rc;
  }
  if ((rc = launch_router_topk(K->ep_logits, tp<float>(L.t, "router_bias"), T, c.experts, c.topk, c.routed_scale, K->ep_ids, K->ep_wts,
                               K->ep_local_ids, K->ep_base, stream)))
    return rc;
  // assignments of experts held elsewhere carry ids outside [0, ep_local): the grouped kernels skip them
  if ((rc = blok_moe_experts_grouped(L.moe, K->n, K->ep_rows, K->ep_local_ids, T * c.topk, K->ep_y, stream_))) return rc;
  sharded_partial_kernel<<<grid, 256, 0, stream>>>(K->ep_y, K->ep_wts, K->ep_local_ids, K->ep_local, c.hidden, c.topk, K->ep_part);
  if ((rc = launch_status("sharded_partial_kernel"))) return rc;
  if ((rc = blok_comm_all_reduce_f32(K->comm, K->ep_part, (long)T * c.hidden, stream_))) return rc;
  const uint16_t *shared = nullptr;
  if (c.shared_inter > 0) {
    if ((rc = blok_moe_shared(L.moe, K->n, T, K->ep_shared, stream_))) return rc;
    shared = K->ep_shared;
  }
  sharded_finish_kernel<<<grid, 256, 0, stream>>>(K->ep_part, shared, c.hidden, K->tmp);
  return launch_status("sharded_finish_kernel");
}

// The feed-forward half of layer l for T rows: K->n -> K->tmp (:829-877 without the residual add).  Steps of up to 3
// sequences take the batch-1 kernels row by row; prefill chunks and larger steps take the grouped kernels for the routed
// experts where the sizes fit them, and the dense layer up to 64 rows at a time.
static int ffn_rows(blok_model_t *m, int l, int T, bool chunk, blok_stream_t stream_) {
  KimiModel *K = kimi(m);
  const blok_model_config &c = m->cfg;
  auto &L = K->layers[l];
  const size_t H = c.hidden;
  // the grouped kernels stream each selected expert once for all rows: from four rows on that is cheaper than a launch
  // of the batch-1 kernel per row (12-layer model, 8 sequences: 10.2 ms a step row by row)
  const bool wide = chunk ? T > 1 : T > 3;
  int rc = BLOK_OK;
  if (l < c.first_dense) {
    // rows per call: up to 8, fewer when 8 rows of the wider of the two vectors would not fit in shared memory
    const size_t row_bytes = (size_t)(c.hidden > c.dense_inter ? c.hidden : c.dense_inter) * 2 + 64;
    int group = wide ? 8 : 1;
    while (group > 1 && row_bytes * group > 200 * 1024) --group;
    if (wide && T > 8 && K->mlp_rows > 8) group = K->mlp_rows;  // one pass over the weights for up to 64 rows
    for (int b = 0; b < T && !rc; b += group)
      rc = blok_bf16_mlp(tp<uint16_t>(L.t, "gate_proj"), tp<uint16_t>(L.t, "up_proj"), tp<uint16_t>(L.t, "down_proj"), K->n + b * H,
                         K->tmp + b * H, c.hidden, c.dense_inter, T - b < group ? T - b : group, K->mlp_ws, K->mlp_ws_bytes, stream_);
    return rc;
  }
  if (c.ep_world > 1) return moe_sharded_rows(m, L, T, stream_);
  if (wide && K->moe_batched_ok) return blok_moe_batched(L.moe, K->n, T, K->tmp, nullptr, nullptr, stream_);
  for (int b = 0; b < T && !rc; ++b) rc = blok_moe_decode(L.moe, K->n + b * H, K->tmp + b * H, nullptr, nullptr, stream_);
  return rc;
}

// Embedding and every layer for T rows of m->ids; leaves the final-normed hidden states in K->n.  chunk: the rows are
// consecutive tokens of sequence 0 (a prefill chunk); otherwise row b is the next token of sequence b.
static int layers(blok_model_t *m, int T, bool chunk, blok_stream_t stream_) {
  KimiModel *K = kimi(m);
  const blok_model_config &c = m->cfg;
  int rc;
  if ((rc = blok_embed(tp<uint16_t>(K->top, "embed_tokens"), m->ids, c.vocab, c.hidden, T, K->x, stream_))) return rc;  // :802
  // Every residual add is fused with the RMSNorm that follows it (blok_add_rmsnorm), so a layer is: attention on n,
  // x += attention | n = norm(x), feed-forward on n, x += feed-forward | n = the next layer's (or the final) norm.
  if ((rc = blok_rmsnorm(K->x, tp<uint16_t>(K->layers[0].t, "input_layernorm"), K->n, T, c.hidden, c.rms_eps, stream_))) return rc;
  for (int l = 0; l < c.layers; ++l) {
    auto &L = K->layers[l];
    // attention block, :812-827
    if (m->pages)  // entry b is slot slot_of[b] at position ctx_b[b], for steps and chunks alike
      rc = blok_mla_decode_paged(L.mla, K->n, L.cache, m->table_dev, m->slot_of, m->table_stride, c.kv_page_rows, m->ctx_b, T, K->tmp,
                                 stream_);
    else
      rc = chunk ? blok_mla_prefill(L.mla, K->n, L.cache, c.max_ctx, m->pos, T, K->tmp, stream_)
                 : blok_mla_decode(L.mla, K->n, L.cache, c.max_ctx, m->pos, T, K->tmp, stream_);
    if (rc) return rc;
    if ((rc = blok_add_rmsnorm(K->x, K->tmp, tp<uint16_t>(L.t, "post_attention_layernorm"), K->n, T, c.hidden, c.rms_eps, stream_)))
      return rc;
    if ((rc = ffn_rows(m, l, T, chunk, stream_))) return rc;  // :829-877
    const bool last = l + 1 == c.layers;
    const uint16_t *next_ln = last ? tp<uint16_t>(K->top, "norm") : tp<uint16_t>(K->layers[l + 1].t, "input_layernorm");  // :812 / :880
    if ((rc = blok_add_rmsnorm(K->x, K->tmp, next_ln, K->n, T, c.hidden, last ? c.final_rms_eps : c.rms_eps, stream_))) return rc;
  }
  return BLOK_OK;
}

// The sampler takes 64 rows per call where the sizes fit the weight-streaming kernel (one pass over the table), else 8.
static int sample(blok_model *m, int row, int n, uint32_t *next, blok_stream_t stream) {
  KimiModel *K = kimi(m);
  const blok_model_config &c = m->cfg;
  const int head_rows = (c.vocab % 16 == 0 && c.hidden % 256 == 0) ? kWgStreamTokens : 8;
  for (int b = 0; b < n; b += head_rows)
    if (int rc = blok_lm_head_argmax(tp<uint16_t>(K->top, "lm_head"), K->n + (size_t)(row + b) * c.hidden, c.vocab, c.hidden,
                                     n - b < head_rows ? n - b : head_rows, next + b, K->head_ws, K->head_ws_bytes, stream))
      return rc;
  return BLOK_OK;
}

static void destroy(blok_model *m) {
  KimiModel *K = kimi(m);
  if (!K) return;
  for (auto &L : K->layers) {
    if (L.mla) blok_mla_layer_destroy(L.mla);
    if (L.moe) blok_moe_layer_destroy(L.moe);
  }
  delete K;
}
