// The serving state every model of the library shares, and the registry of model families.
//
// A blok_model handle owns the sequence slots, their positions, the page table of the caches, the token buffers and the
// CUDA graphs of its decode steps (model.cu); what runs between a step's token ids and its logits belongs to the
// handle's family: Kimi's blocks (model_kimi.cu) or a stack of layers described by a config.json (model_stack.cu).
#pragma once
#include <string>
#include <vector>

#include "common.cuh"
#include "json_reader.h"

namespace blok {

constexpr int kMaxBatch = 64;  // sequences per step

struct ModelFamily {
  const char *architecture;  // "architecture" of config.json
  int max_chunk;             // most tokens of a prompt per pass
  // From config.json: fills m->cfg's sizes and the family's own description.  NULL: models of this family are not opened
  // from a folder (they have entry points of their own).  No device memory is taken.
  int (*configure)(blok_model *m, const Json &config);
  // Takes device memory and fills the weights: from `dir` (weights beside config.json), or seeded when dir is NULL.
  int (*build)(blok_model *m, const char *dir, uint64_t seed);
  void (*destroy)(blok_model *m);
  // Embedding and every layer for the T rows of m->ids.  chunk: the rows are the next T tokens of the sequence in slot
  // m->chunk_slot; otherwise row b is the next token of the b-th sequence of the step.
  int (*layers)(blok_model *m, int T, bool chunk, blok_stream_t stream);
  // Greedy ids of rows [row, row + n) of the last `layers` call.
  int (*sample)(blok_model *m, int row, int n, uint32_t *next, blok_stream_t stream);
  // Logits of the rows listed on the host, fp32 [n, vocab] in host memory; synchronises.  NULL: not offered.
  int (*logits)(blok_model *m, const int *rows, int n, float *out, blok_stream_t stream);
  int (*check)(blok_model *m, blok_stream_t stream);
};

// Families register themselves at start-up: what is linked in can be opened.
struct FamilyRegistration {
  explicit FamilyRegistration(const ModelFamily *family);
};

}  // namespace blok

struct blok_model {
  const blok::ModelFamily *family = nullptr;
  void *impl = nullptr;  // the family's own state
  blok_model_config cfg{};
  int dtype = BLOK_DTYPE_BF16;
  std::vector<void *> allocations;
  int rows = 0;                    // max(max_batch, prefill_chunk)
  uint32_t *prompt_ids = nullptr;  // [max(max_ctx, rows)] token ids given on the host (prefill_chunk >= 1)
  std::vector<long> host_pos;      // tokens cached per sequence (host mirror of pos)
  // paged cache (cfg.kv_page_rows > 0): one table for all layers' pools
  blok_kv_pages_t *pages = nullptr;
  int table_stride = 0;
  int *table_dev = nullptr;                  // [max_batch, table_stride]
  int *slot_of = nullptr, *ctx_b = nullptr;  // [rows] slot and position of every batch entry of the call in flight
  int chunk_slot = 0;                        // slot of the prompt chunk in flight
  int *pos = nullptr;                        // [max_batch]
  uint32_t *ids = nullptr, *next = nullptr;  // [rows]
  // One CUDA graph of the whole step per batch size: a step is many small launches per layer and the host cannot issue
  // them as fast as the GPU runs them.  steps_seen counts eager steps (the first one also sets kernel attributes).
  cudaGraphExec_t step_graph[blok::kMaxBatch + 1] = {};
  long long graph_launches[blok::kMaxBatch + 1] = {};  // kernels in each graph, added to the launch counter at every replay
  int steps_seen[blok::kMaxBatch + 1] = {};
  bool graphs_enabled = true;
  cudaStream_t own_stream = nullptr;  // generation runs here: unlike the legacy default stream it can be captured
  // blok_model_trace_layers: fp32 [layer_runs, trace_rows, hidden]; layer_runs is set by the family's configure
  float *trace = nullptr;
  int trace_rows = 0, layer_runs = 0;
};

namespace blok {

int dev_alloc(blok_model *m, size_t bytes, void **out);
template <typename T>
int dev_alloc_as(blok_model *m, size_t count, T **out) {
  void *p = nullptr;
  if (int rc = dev_alloc(m, count * sizeof(T), &p)) return rc;
  *out = static_cast<T *>(p);
  return BLOK_OK;
}
// Token buffers, positions and, for a paged model, the page table; m->cfg and m->rows are set.
int alloc_serving_state(blok_model *m);

}  // namespace blok
