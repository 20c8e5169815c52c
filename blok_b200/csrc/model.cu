// The serving side of a model handle, whatever its family: opening, slots and positions, decode steps (replayed from CUDA
// graphs), prompts in chunks, greedy generation and continuous batching.  Reference: generate() and its `run` lambda,
// src/kimi_exec.cu:780-893 (prompt replay and decode loop :885-890).
#include <algorithm>
#include <cstring>
#include <fstream>
#include <new>
#include <sstream>

#include "model.h"

namespace blok {

__global__ void advance_kernel(int *pos, int n, int by) {
  int i = threadIdx.x;
  if (i < n) pos[i] += by;
}

// Paged model: batch entry b is the sequence in slot slot_of[b].
__global__ void gather_positions_kernel(const int *__restrict__ pos, const int *__restrict__ slot_of, int n, int *__restrict__ ctx) {
  const int b = threadIdx.x;
  if (b < n) ctx[b] = pos[slot_of[b]];
}
__global__ void advance_slots_kernel(int *__restrict__ pos, const int *__restrict__ slot_of, int n) {
  const int b = threadIdx.x;
  if (b < n) pos[slot_of[b]] += 1;  // the slots of a step are distinct
}
// A prompt chunk of the sequence in `slot`: entry i is that slot at position pos[slot] + i.
__global__ void chunk_slots_kernel(const int *__restrict__ pos, int slot, int n, int *__restrict__ ctx, int *__restrict__ slot_of) {
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i < n) {
    ctx[i] = pos[slot] + i;
    slot_of[i] = slot;
  }
}

// ---- registry ----
static std::vector<const ModelFamily *> &families() {
  static std::vector<const ModelFamily *> list;
  return list;
}
FamilyRegistration::FamilyRegistration(const ModelFamily *family) { families().push_back(family); }

int dev_alloc(blok_model *m, size_t bytes, void **out) {
  void *p = nullptr;
  BLOK_CUDA(cudaMalloc(&p, bytes ? bytes : 16));
  m->allocations.push_back(p);
  *out = p;
  return BLOK_OK;
}

int alloc_serving_state(blok_model *m) {
  const blok_model_config &c = m->cfg;
  int rc;
  if ((rc = dev_alloc_as(m, c.max_batch, &m->pos)) || (rc = dev_alloc_as(m, m->rows, &m->ids)) || (rc = dev_alloc_as(m, m->rows, &m->next)) ||
      (rc = dev_alloc_as(m, c.prefill_chunk > 0 ? std::max(c.max_ctx, m->rows) : 1, &m->prompt_ids)))
    return rc;
  BLOK_CUDA(cudaMemset(m->pos, 0, c.max_batch * 4));
  m->host_pos.assign(c.max_batch, 0);
  if (c.kv_page_rows > 0) {
    m->table_stride = (c.max_ctx + c.kv_page_rows - 1) / c.kv_page_rows;
    if ((rc = blok_kv_pages_create(c.kv_pages, c.kv_page_rows, c.max_batch, m->table_stride, &m->pages))) return rc;
    if ((rc = dev_alloc_as(m, (size_t)c.max_batch * m->table_stride, &m->table_dev))) return rc;
    BLOK_CUDA(cudaMemset(m->table_dev, 0, (size_t)c.max_batch * m->table_stride * 4));
    if ((rc = dev_alloc_as(m, m->rows, &m->slot_of)) || (rc = dev_alloc_as(m, m->rows, &m->ctx_b))) return rc;
  }
  return BLOK_OK;
}

}  // namespace blok

using namespace blok;

extern "C" int blok_model_destroy(blok_model_t *m) {
  if (!m) return BLOK_OK;
  for (auto &g : m->step_graph)
    if (g) cudaGraphExecDestroy(g);
  blok_kv_pages_destroy(m->pages);
  if (m->family) m->family->destroy(m);
  if (m->own_stream) cudaStreamDestroy(m->own_stream);
  cudaError_t first = cudaSuccess;
  for (void *p : m->allocations) {
    cudaError_t e = cudaFree(p);
    if (first == cudaSuccess) first = e;
  }
  delete m;
  return first == cudaSuccess ? BLOK_OK : cuda_fail(first, "cudaFree(model)");
}

extern "C" int blok_model_get_config(blok_model_t *m, blok_model_config *cfg) {
  BLOK_REQUIRE(m && cfg, BLOK_ERR_ARG, "blok_model_get_config: null pointer");
  *cfg = m->cfg;
  return BLOK_OK;
}

extern "C" int blok_model_check(blok_model_t *m, blok_stream_t stream) {
  BLOK_REQUIRE(m, BLOK_ERR_ARG, "blok_model_check: null pointer");
  return m->family->check(m, stream);
}

// ---- models described by a config.json ----
extern "C" const char *blok_model_architectures(void) {
  static const std::string names = [] {
    std::string s;
    for (const ModelFamily *f : families())
      if (f->configure) s += (s.empty() ? "" : " ") + std::string(f->architecture);
    return s;
  }();
  return names.c_str();
}

extern "C" void blok_model_default_options(blok_model_options *o) {
  if (!o) return;
  memset(o, 0, sizeof(*o));
  o->dtype = BLOK_DTYPE_BF16;
  o->max_batch = 1;
  o->max_ctx = 4096;
  o->prefill_chunk = 1024;
  o->kv_page_rows = 64;
  o->eos_id = 0xffffffffu;
}

// `text` is a config.json; dir: the folder the weights lie in, NULL for seeded ones.
static int open_config(const std::string &text, const char *dir, uint64_t seed, const blok_model_options *opt, blok_model_t **out) {
  Json j;
  JsonParser parser(text.data(), text.data() + text.size());
  BLOK_REQUIRE(parser.parse(&j) && j.kind == Json::Object, BLOK_ERR_ARG, "config.json: %s",
               parser.error().empty() ? "not an object" : parser.error().c_str());
  const Json *arch = j.find("architecture");
  BLOK_REQUIRE(arch && arch->kind == Json::String, BLOK_ERR_ARG, "config.json: no \"architecture\"");
  const ModelFamily *family = nullptr;
  for (const ModelFamily *f : families())
    if (f->configure && arch->text == f->architecture) family = f;
  BLOK_REQUIRE(family, BLOK_ERR_ARG, "config.json: architecture \"%s\" is not one of: %s", arch->text.c_str(), blok_model_architectures());
  blok_model_options o;
  if (opt) o = *opt;
  else blok_model_default_options(&o);
  BLOK_REQUIRE(o.dtype == BLOK_DTYPE_BF16 || o.dtype == BLOK_DTYPE_F32, BLOK_ERR_ARG, "blok_model_open: unknown dtype %d", o.dtype);
  BLOK_REQUIRE(o.max_batch >= 1 && o.max_batch <= kMaxBatch && o.max_ctx >= 1 && o.prefill_chunk >= 1 && o.prefill_chunk <= family->max_chunk &&
                   o.kv_page_rows >= 32 && o.kv_page_rows % 32 == 0 && o.kv_pages >= 0,
               BLOK_ERR_SHAPE, "blok_model_open: need 1 <= max_batch <= %d, max_ctx >= 1, 1 <= prefill_chunk <= %d and kv_page_rows a multiple of 32",
               kMaxBatch, family->max_chunk);
  blok_model *m = new (std::nothrow) blok_model();
  BLOK_REQUIRE(m, BLOK_ERR_ARG, "blok_model_open: out of host memory");
  m->family = family;
  m->dtype = o.dtype;
  m->cfg.max_batch = o.max_batch;
  m->cfg.max_ctx = o.max_ctx;
  m->cfg.prefill_chunk = o.prefill_chunk;
  m->cfg.eos_id = o.eos_id;
  m->cfg.kv_page_rows = o.kv_page_rows;
  // 0 pages: enough for every slot at max_ctx
  m->cfg.kv_pages = o.kv_pages ? o.kv_pages : o.max_batch * ((o.max_ctx + o.kv_page_rows - 1) / o.kv_page_rows);
  m->rows = std::max(o.max_batch, o.prefill_chunk);
  if (const char *g = getenv("BLOK_MODEL_GRAPH")) m->graphs_enabled = strcmp(g, "0") != 0;
  int rc = family->configure(m, j);
  if (!rc) rc = family->build(m, dir, seed);
  if (rc) {
    blok_model_destroy(m);
    return rc;
  }
  *out = m;
  return BLOK_OK;
}

extern "C" int blok_model_open(const char *dir, const blok_model_options *opt, blok_model_t **out) {
  BLOK_REQUIRE(dir && out, BLOK_ERR_ARG, "blok_model_open: null pointer");
  const std::string path = std::string(dir) + "/config.json";
  std::ifstream in(path);
  BLOK_REQUIRE(in.good(), BLOK_ERR_ARG, "cannot open %s", path.c_str());
  std::stringstream text;
  text << in.rdbuf();
  return open_config(text.str(), dir, 0, opt, out);
}

extern "C" int blok_model_open_synthetic(const char *config_json, uint64_t seed, const blok_model_options *opt, blok_model_t **out) {
  BLOK_REQUIRE(config_json && out, BLOK_ERR_ARG, "blok_model_open_synthetic: null pointer");
  return open_config(config_json, nullptr, seed, opt, out);
}

extern "C" int blok_model_reset(blok_model_t *m) {
  BLOK_REQUIRE(m, BLOK_ERR_ARG, "blok_model_reset: null pointer");
  BLOK_CUDA(cudaMemset(m->pos, 0, m->cfg.max_batch * 4));
  for (int s = 0; s < m->cfg.max_batch; ++s) {
    m->host_pos[s] = 0;
    if (m->pages) blok_kv_pages_release(m->pages, s);
  }
  return BLOK_OK;
}

// The launches of one decode step on `stream`, reading m->ids and writing m->next; every position and length is device
// resident, so the same sequence of launches serves every step and can be replayed from a graph.
static int step_body(blok_model_t *m, int B, blok_stream_t stream_) {
  cudaStream_t stream = (cudaStream_t)stream_;
  int rc;
  if (m->pages) {
    gather_positions_kernel<<<1, 64, 0, stream>>>(m->pos, m->slot_of, B, m->ctx_b);
    if ((rc = launch_status("gather_positions_kernel"))) return rc;
  }
  if ((rc = m->family->layers(m, B, false, stream_))) return rc;
  if ((rc = m->family->sample(m, 0, B, m->next, stream_))) return rc;
  if (m->pages) advance_slots_kernel<<<1, 64, 0, stream>>>(m->pos, m->slot_of, B);
  else advance_kernel<<<1, 64, 0, stream>>>(m->pos, B, 1);
  return launch_status("advance_kernel");
}

// step_body, eagerly or from the batch size's graph.  The first step of a batch size runs eagerly, the second is captured
// (nothing executes during capture) and replayed at once, later steps replay the graph.  The legacy default stream cannot
// be captured.
static int run_step(blok_model_t *m, int B, blok_stream_t stream_) {
  cudaStream_t stream = (cudaStream_t)stream_;
  int rc = BLOK_OK;
  const bool can_graph = m->graphs_enabled && !m->trace && stream != nullptr && stream != cudaStreamLegacy;
  if (can_graph && m->step_graph[B]) {
    BLOK_CUDA(cudaGraphLaunch(m->step_graph[B], stream));
    count_launches(m->graph_launches[B]);
  } else if (can_graph && m->steps_seen[B] >= 1) {
    cudaGraph_t graph = nullptr;
    cudaError_t e = cudaStreamBeginCapture(stream, cudaStreamCaptureModeThreadLocal);
    if (e == cudaSuccess) {
      const long long before = launches_so_far();
      rc = step_body(m, B, stream_);
      m->graph_launches[B] = launches_so_far() - before;
      count_launches(-m->graph_launches[B]);  // nothing ran during the capture
      cudaError_t e2 = cudaStreamEndCapture(stream, &graph);
      if (rc == BLOK_OK && e2 == cudaSuccess && graph) e = cudaGraphInstantiate(&m->step_graph[B], graph, 0);
      else e = e2 == cudaSuccess ? cudaErrorUnknown : e2;
      if (graph) cudaGraphDestroy(graph);
    }
    if (e != cudaSuccess || !m->step_graph[B]) {  // capture is not possible here: stay with eager launches
      cudaGetLastError();
      m->step_graph[B] = nullptr;
      m->graphs_enabled = false;
      rc = step_body(m, B, stream_);
    } else {
      BLOK_CUDA(cudaGraphLaunch(m->step_graph[B], stream));
      count_launches(m->graph_launches[B]);
      rc = BLOK_OK;
    }
  } else {
    rc = step_body(m, B, stream_);
    ++m->steps_seen[B];
  }
  if (rc) return rc;
  return rc;
}

extern "C" int blok_model_step_slots(blok_model_t *m, const int *slots, int B, const uint32_t *ids, uint32_t *next_ids,
                                     blok_stream_t stream_) {
  BLOK_REQUIRE(m && slots && ids && next_ids, BLOK_ERR_ARG, "blok_model_step_slots: null pointer");
  const blok_model_config &c = m->cfg;
  BLOK_REQUIRE(B >= 1 && B <= c.max_batch, BLOK_ERR_SHAPE, "blok_model_step_slots: B=%d outside [1, %d]", B, c.max_batch);
  bool identity = true;
  for (int b = 0; b < B; ++b) {
    BLOK_REQUIRE(slots[b] >= 0 && slots[b] < c.max_batch, BLOK_ERR_ARG, "blok_model_step_slots: slot %d outside [0, %d)", slots[b],
                 c.max_batch);
    for (int a = 0; a < b; ++a) BLOK_REQUIRE(slots[a] != slots[b], BLOK_ERR_ARG, "blok_model_step_slots: slot %d named twice", slots[b]);
    BLOK_REQUIRE(m->host_pos[slots[b]] + 1 <= c.max_ctx, BLOK_ERR_SHAPE,
                 "blok_model_step_slots: the sequence in slot %d already holds max_ctx = %d tokens", slots[b], c.max_ctx);  // :205
    identity = identity && slots[b] == b;
  }
  if (!m->pages) {
    BLOK_REQUIRE(identity, BLOK_ERR_STATE, "blok_model_step_slots: a model with a dense cache steps slots 0..B-1 only");
    return blok_model_step(m, ids, B, next_ids, stream_);
  }
  cudaStream_t stream = (cudaStream_t)stream_;
  int rc;
  for (int b = 0; b < B; ++b)
    if ((rc = blok_kv_pages_reserve(m->pages, slots[b], m->host_pos[slots[b]] + 1))) return rc;
  if ((rc = blok_kv_pages_upload(m->pages, m->table_dev, stream_))) return rc;
  BLOK_CUDA(cudaMemcpyAsync(m->slot_of, slots, (size_t)B * 4, cudaMemcpyHostToDevice, stream));
  if (ids != m->ids) BLOK_CUDA(cudaMemcpyAsync(m->ids, ids, (size_t)B * 4, cudaMemcpyDeviceToDevice, stream));
  if ((rc = run_step(m, B, stream_))) return rc;
  for (int b = 0; b < B; ++b) ++m->host_pos[slots[b]];
  if (next_ids != m->next) BLOK_CUDA(cudaMemcpyAsync(next_ids, m->next, (size_t)B * 4, cudaMemcpyDeviceToDevice, stream));
  return BLOK_OK;
}

extern "C" int blok_model_step(blok_model_t *m, const uint32_t *ids, int B, uint32_t *next_ids, blok_stream_t stream_) {
  BLOK_REQUIRE(m && ids && next_ids, BLOK_ERR_ARG, "blok_model_step: null pointer");
  BLOK_REQUIRE(B >= 1 && B <= m->cfg.max_batch, BLOK_ERR_SHAPE, "blok_model_step: B=%d outside [1, %d]", B, m->cfg.max_batch);
  if (m->pages) {
    int slots[kMaxBatch];
    for (int b = 0; b < B; ++b) slots[b] = b;
    return blok_model_step_slots(m, slots, B, ids, next_ids, stream_);
  }
  for (int b = 0; b < B; ++b)
    BLOK_REQUIRE(m->host_pos[b] + 1 <= m->cfg.max_ctx, BLOK_ERR_SHAPE, "blok_model_step: sequence %d already holds max_ctx = %d tokens", b,
                 m->cfg.max_ctx);  // the reference's capacity check, :205
  for (int b = 0; b < B; ++b) ++m->host_pos[b];
  cudaStream_t stream = (cudaStream_t)stream_;
  if (ids != m->ids) BLOK_CUDA(cudaMemcpyAsync(m->ids, ids, (size_t)B * 4, cudaMemcpyDeviceToDevice, stream));
  if (int rc = run_step(m, B, stream_)) return rc;
  if (next_ids != m->next) BLOK_CUDA(cudaMemcpyAsync(next_ids, m->next, (size_t)B * 4, cudaMemcpyDeviceToDevice, stream));
  return BLOK_OK;
}

// One chunk of a prompt: the layers over the T next tokens of the sequence in `slot`, then (after whatever reads the rows)
// the position's advance.  The pages are reserved and the table is on the device.
static int begin_chunk(blok_model_t *m, int slot, const uint32_t *ids, int T, blok_stream_t stream_) {
  cudaStream_t stream = (cudaStream_t)stream_;
  if (ids != m->ids) BLOK_CUDA(cudaMemcpyAsync(m->ids, ids, (size_t)T * 4, cudaMemcpyDeviceToDevice, stream));
  m->chunk_slot = slot;
  if (m->pages) {
    chunk_slots_kernel<<<(T + 63) / 64, 64, 0, stream>>>(m->pos, slot, T, m->ctx_b, m->slot_of);
    if (int rc = launch_status("chunk_slots_kernel")) return rc;
  }
  return m->family->layers(m, T, true, stream_);
}
static int end_chunk(blok_model_t *m, int slot, int T, blok_stream_t stream_) {
  advance_kernel<<<1, 64, 0, (cudaStream_t)stream_>>>(m->pos + slot, 1, T);
  if (int rc = launch_status("advance_kernel")) return rc;
  m->host_pos[slot] += T;
  return BLOK_OK;
}

extern "C" int blok_model_prefill_slot(blok_model_t *m, int slot, const uint32_t *ids, int n, uint32_t *next_id, blok_stream_t stream_) {
  BLOK_REQUIRE(m && ids && next_id, BLOK_ERR_ARG, "blok_model_prefill: null pointer");
  BLOK_REQUIRE(m->cfg.prefill_chunk >= 1, BLOK_ERR_STATE, "blok_model_prefill: the model was created with prefill_chunk = 0");
  BLOK_REQUIRE(n >= 1, BLOK_ERR_ARG, "blok_model_prefill: no tokens");
  const blok_model_config &c = m->cfg;
  BLOK_REQUIRE(slot >= 0 && slot < c.max_batch && (m->pages || slot == 0), BLOK_ERR_ARG,
               "blok_model_prefill: slot %d (a model with a dense cache prefills sequence 0 only)", slot);
  BLOK_REQUIRE(m->host_pos[slot] + n <= c.max_ctx, BLOK_ERR_SHAPE, "blok_model_prefill: %ld cached + %d new tokens exceed max_ctx = %d",
               m->host_pos[slot], n, c.max_ctx);  // :205
  cudaStream_t stream = (cudaStream_t)stream_;
  int rc;
  if (m->pages && (rc = blok_kv_pages_reserve(m->pages, slot, m->host_pos[slot] + n))) return rc;  // all or nothing, before any launch
  if (m->pages && (rc = blok_kv_pages_upload(m->pages, m->table_dev, stream_))) return rc;
  for (int at = 0; at < n; at += c.prefill_chunk) {
    const int T = n - at < c.prefill_chunk ? n - at : c.prefill_chunk;
    if ((rc = begin_chunk(m, slot, ids + at, T, stream_))) return rc;
    if (at + T == n && (rc = m->family->sample(m, T - 1, 1, m->next, stream_))) return rc;  // only the last token is sampled (:886)
    if ((rc = end_chunk(m, slot, T, stream_))) return rc;
  }
  if (next_id != m->next) BLOK_CUDA(cudaMemcpyAsync(next_id, m->next, 4, cudaMemcpyDeviceToDevice, stream));
  return BLOK_OK;
}

extern "C" int blok_model_prefill(blok_model_t *m, const uint32_t *ids, int n, uint32_t *next_id, blok_stream_t stream) {
  return blok_model_prefill_slot(m, 0, ids, n, next_id, stream);
}

extern "C" int blok_model_extend_slot(blok_model_t *m, int slot, const uint32_t *ids, int n, const int *want, int n_want, float *logits,
                                      blok_stream_t stream_) {
  BLOK_REQUIRE(m && ids && n >= 1 && n_want >= 0 && (n_want == 0 || (want && logits)), BLOK_ERR_ARG, "blok_model_extend_slot: null pointer or no tokens");
  BLOK_REQUIRE(m->family->logits && m->pages, BLOK_ERR_STATE, "blok_model_extend_slot: models of the family %s do not offer logits",
               m->family->architecture);
  const blok_model_config &c = m->cfg;
  BLOK_REQUIRE(slot >= 0 && slot < c.max_batch, BLOK_ERR_ARG, "blok_model_extend_slot: slot %d outside [0, %d)", slot, c.max_batch);
  BLOK_REQUIRE(m->host_pos[slot] + n <= c.max_ctx, BLOK_ERR_SHAPE, "blok_model_extend_slot: %ld cached + %d new tokens exceed max_ctx = %d",
               m->host_pos[slot], n, c.max_ctx);
  for (int i = 0; i < n; ++i)
    BLOK_REQUIRE(ids[i] < (uint32_t)c.vocab, BLOK_ERR_ARG, "blok_model_extend_slot: token %u outside the vocabulary", ids[i]);
  for (int i = 0; i < n_want; ++i)
    BLOK_REQUIRE(want[i] >= 0 && want[i] < n, BLOK_ERR_ARG, "blok_model_extend_slot: place %d outside the %d tokens", want[i], n);
  cudaStream_t stream = (cudaStream_t)stream_;
  BLOK_CUDA(cudaMemcpyAsync(m->prompt_ids, ids, (size_t)n * 4, cudaMemcpyHostToDevice, stream));
  int rc;
  if (n == 1) {  // the decode step, and the logits of the row it left
    if ((rc = blok_model_step_slots(m, &slot, 1, m->prompt_ids, m->next, stream_))) return rc;
    const int row = 0;
    for (int i = 0; i < n_want; ++i)
      if ((rc = m->family->logits(m, &row, 1, logits + (size_t)i * c.vocab, stream_))) return rc;
    return BLOK_OK;
  }
  if ((rc = blok_kv_pages_reserve(m->pages, slot, m->host_pos[slot] + n))) return rc;
  if ((rc = blok_kv_pages_upload(m->pages, m->table_dev, stream_))) return rc;
  std::vector<int> rows, places;
  std::vector<float> got;
  for (int at = 0; at < n; at += c.prefill_chunk) {
    const int T = std::min(n - at, c.prefill_chunk);
    if ((rc = begin_chunk(m, slot, m->prompt_ids + at, T, stream_))) return rc;
    rows.clear(), places.clear();
    for (int i = 0; i < n_want; ++i)
      if (want[i] >= at && want[i] < at + T) rows.push_back(want[i] - at), places.push_back(i);
    if (!rows.empty()) {
      got.resize(rows.size() * (size_t)c.vocab);
      if ((rc = m->family->logits(m, rows.data(), (int)rows.size(), got.data(), stream_))) return rc;
      for (size_t i = 0; i < rows.size(); ++i)
        memcpy(logits + (size_t)places[i] * c.vocab, got.data() + i * (size_t)c.vocab, (size_t)c.vocab * sizeof(float));
    }
    if ((rc = end_chunk(m, slot, T, stream_))) return rc;
  }
  return BLOK_OK;
}

extern "C" int blok_model_trace_layers(blok_model_t *m, float *buffer, int max_rows, int *runs) {
  BLOK_REQUIRE(m && runs && (!buffer || max_rows >= 1), BLOK_ERR_ARG, "blok_model_trace_layers: null pointer or max_rows < 1");
  BLOK_REQUIRE(m->layer_runs > 0, BLOK_ERR_STATE, "blok_model_trace_layers: models of the family %s do not offer it", m->family->architecture);
  m->trace = buffer;
  m->trace_rows = buffer ? max_rows : 0;
  *runs = m->layer_runs;
  return BLOK_OK;
}

extern "C" int blok_model_slot_release(blok_model_t *m, int slot, blok_stream_t stream) {
  BLOK_REQUIRE(m, BLOK_ERR_ARG, "blok_model_slot_release: null pointer");
  BLOK_REQUIRE(slot >= 0 && slot < m->cfg.max_batch, BLOK_ERR_ARG, "blok_model_slot_release: slot %d outside [0, %d)", slot,
               m->cfg.max_batch);
  BLOK_CUDA(cudaMemsetAsync(m->pos + slot, 0, 4, (cudaStream_t)stream));
  m->host_pos[slot] = 0;
  return m->pages ? blok_kv_pages_release(m->pages, slot) : BLOK_OK;
}

extern "C" long blok_model_slot_length(blok_model_t *m, int slot) {
  return (m && slot >= 0 && slot < m->cfg.max_batch) ? m->host_pos[slot] : -1;
}

extern "C" int blok_model_free_pages(blok_model_t *m) { return (m && m->pages) ? blok_kv_pages_free_count(m->pages) : -1; }

// The stream generation runs on.  It is a blocking stream: copies and memsets on the legacy default stream are ordered with
// it.
static int generation_stream(blok_model_t *m, blok_stream_t *out) {
  if (!m->own_stream) BLOK_CUDA(cudaStreamCreate(&m->own_stream));
  *out = (blok_stream_t)m->own_stream;
  return BLOK_OK;
}

extern "C" int blok_model_generate(blok_model_t *m, const uint32_t *prompt, int n_prompt, int max_new, uint32_t *out,
                                   int *n_out) {
  BLOK_REQUIRE(m && prompt && out && n_out, BLOK_ERR_ARG, "blok_model_generate: null pointer");
  BLOK_REQUIRE(n_prompt >= 1 && max_new >= 1, BLOK_ERR_ARG, "blok_model_generate: empty prompt or max_new < 1");
  BLOK_REQUIRE((long)n_prompt + max_new <= m->cfg.max_ctx, BLOK_ERR_SHAPE,
               "blok_model_generate: requested sequence exceeds the model's context (%d)", m->cfg.max_ctx);  // :784
  for (int i = 0; i < n_prompt; ++i)
    BLOK_REQUIRE(prompt[i] < (uint32_t)m->cfg.vocab, BLOK_ERR_ARG, "blok_model_generate: prompt token outside vocabulary");
  int rc = blok_model_reset(m);
  if (rc) return rc;
  blok_stream_t stream;
  if ((rc = generation_stream(m, &stream))) return rc;
  *n_out = 0;
  uint32_t next = prompt[0];
  if (m->cfg.prefill_chunk >= 1) {
    // the prompt in chunks: every layer's weights are read once per chunk instead of once per token
    BLOK_CUDA(cudaMemcpyAsync(m->prompt_ids, prompt, (size_t)n_prompt * 4, cudaMemcpyHostToDevice, nullptr));
    if ((rc = blok_model_prefill(m, m->prompt_ids, n_prompt, m->next, stream))) return rc;
  } else {
    // prompt replay, token by token; only the last step's sample is used (:886)
    for (int i = 0; i < n_prompt; ++i) {
      BLOK_CUDA(cudaMemcpyAsync(m->ids, prompt + i, 4, cudaMemcpyHostToDevice, nullptr));
      if ((rc = blok_model_step(m, m->ids, 1, m->next, stream))) return rc;
    }
  }
  BLOK_CUDA(cudaMemcpy(&next, m->next, 4, cudaMemcpyDeviceToHost));
  for (int i = 0; i < max_new && next != m->cfg.eos_id; ++i) {  // :887-890
    out[(*n_out)++] = next;
    if (i + 1 < max_new) {
      if ((rc = blok_model_step(m, m->next, 1, m->next, stream))) return rc;
      BLOK_CUDA(cudaMemcpy(&next, m->next, 4, cudaMemcpyDeviceToHost));
    }
  }
  // a bounded device-side wait that gave up (or a position outside a cache) in any layer makes the tokens void
  return blok_model_check(m, stream);
}

// The serving loop of blok_model_generate_many over an existing batcher (the caller destroys it).
static int serve_requests(blok_model_t *m, blok_batcher_t *bt, const uint32_t *prompts, const int *prompt_offsets, int n_requests,
                          int max_new, uint32_t *out, int *n_out) {
  const blok_model_config &c = m->cfg;
  blok_stream_t stream;
  int rc = generation_stream(m, &stream);
  for (int r = 0; r < n_requests && !rc; ++r) {
    int id = -1;
    rc = blok_batcher_submit(bt, prompt_offsets[r + 1] - prompt_offsets[r], max_new, &id);
    n_out[r] = 0;
  }
  std::vector<int> admit_slots(c.max_batch), admit_req(c.max_batch), decode_slots(c.max_batch), slot_req(c.max_batch, -1);
  std::vector<uint32_t> last(c.max_batch, 0), ids(c.max_batch), sampled(c.max_batch);
  // one sampled token of the sequence in `slot`: emitted unless it is EOS (:887); the batcher says whether the sequence ended
  auto take = [&](int slot, uint32_t tok) -> int {
    const int r = slot_req[slot];
    const int eos = tok == c.eos_id;
    if (!eos) out[(size_t)r * max_new + n_out[r]++] = tok;
    last[slot] = tok;
    int finished = 0;
    int e = blok_batcher_token(bt, slot, eos, &finished);
    if (e) return e;
    if (finished) {
      slot_req[slot] = -1;
      return blok_model_slot_release(m, slot, stream);
    }
    return BLOK_OK;
  };
  while (!rc && blok_batcher_unfinished(bt) > 0) {
    int n_admit = 0, n_decode = 0;
    if ((rc = blok_batcher_plan(bt, admit_slots.data(), admit_req.data(), &n_admit, decode_slots.data(), &n_decode))) break;
    if (n_admit == 0 && n_decode == 0) {  // cannot happen: submit refused what can never fit, and finished sequences free their budget
      set_error("blok_model_generate_many: no sequence can make progress");
      rc = BLOK_ERR_STATE;
      break;
    }
    if (n_decode) {  // the running sequences step together; their ids come back for the EOS test, as at :882
      for (int b = 0; b < n_decode; ++b) ids[b] = last[decode_slots[b]];
      BLOK_CUDA(cudaMemcpyAsync(m->prompt_ids, ids.data(), (size_t)n_decode * 4, cudaMemcpyHostToDevice, nullptr));
      if ((rc = blok_model_step_slots(m, decode_slots.data(), n_decode, m->prompt_ids, m->next, stream))) break;
      BLOK_CUDA(cudaMemcpy(sampled.data(), m->next, (size_t)n_decode * 4, cudaMemcpyDeviceToHost));
      for (int b = 0; b < n_decode && !rc; ++b) rc = take(decode_slots[b], sampled[b]);
      if (rc) break;
    }
    for (int a = 0; a < n_admit && !rc; ++a) {  // arrivals: the prompt in chunks, its last token sampled
      const int slot = admit_slots[a], r = admit_req[a];
      const int n = prompt_offsets[r + 1] - prompt_offsets[r];
      slot_req[slot] = r;
      BLOK_CUDA(cudaMemcpyAsync(m->prompt_ids, prompts + prompt_offsets[r], (size_t)n * 4, cudaMemcpyHostToDevice, nullptr));
      if ((rc = blok_model_prefill_slot(m, slot, m->prompt_ids, n, m->next, stream))) break;
      uint32_t tok = 0;
      BLOK_CUDA(cudaMemcpy(&tok, m->next, 4, cudaMemcpyDeviceToHost));
      rc = take(slot, tok);
    }
  }
  return rc;
}

extern "C" int blok_model_generate_many(blok_model_t *m, const uint32_t *prompts, const int *prompt_offsets, int n_requests,
                                        int max_new, uint32_t *out, int *n_out) {
  BLOK_REQUIRE(m && prompts && prompt_offsets && out && n_out, BLOK_ERR_ARG, "blok_model_generate_many: null pointer");
  BLOK_REQUIRE(m->pages && m->cfg.prefill_chunk >= 1, BLOK_ERR_STATE,
               "blok_model_generate_many: needs a paged model (kv_page_rows > 0) with prefill_chunk >= 1");
  BLOK_REQUIRE(n_requests >= 1 && max_new >= 1, BLOK_ERR_ARG, "blok_model_generate_many: no requests or max_new < 1");
  const blok_model_config &c = m->cfg;
  for (int r = 0; r < n_requests; ++r) {
    BLOK_REQUIRE(prompt_offsets[r + 1] > prompt_offsets[r], BLOK_ERR_ARG, "blok_model_generate_many: request %d has an empty prompt", r);
    for (int i = prompt_offsets[r]; i < prompt_offsets[r + 1]; ++i)
      BLOK_REQUIRE(prompts[i] < (uint32_t)c.vocab, BLOK_ERR_ARG, "blok_model_generate_many: prompt token outside vocabulary");  // :552
  }
  int rc = blok_model_reset(m);
  if (rc) return rc;
  blok_batcher_t *bt = nullptr;
  if ((rc = blok_batcher_create(c.max_batch, c.kv_pages, c.kv_page_rows, c.max_ctx, &bt))) return rc;
  rc = serve_requests(m, bt, prompts, prompt_offsets, n_requests, max_new, out, n_out);
  blok_batcher_destroy(bt);
  return rc ? rc : blok_model_check(m, (blok_stream_t)m->own_stream);
}
