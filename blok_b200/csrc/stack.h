// Models that are a stack of layers between an embedding and a vocabulary product, described by values: every layer is a
// token mixer and, usually, a feed-forward, around residual streams that mix (hyper-connections) with a Dynamic-Tanh norm
// in front of every sublayer.  A design (nomozen.cu) turns its config.json into a StackSpec; the runtime is model_stack.cu.
#pragma once
#include <vector>

#include "model.h"

namespace blok {

// Linear attention with a fixed decay per head, then a norm, a gate and the output product.
struct LinearMixer {
  int heads = 0, dim = 0, vdim = 0;
  std::vector<double> decay;  // per head
  double k_scale = 1;
  bool silu_qkv = false;      // SiLU on q, k and v
  bool norm_per_head = false; // else one norm over all heads
  bool norm_weight = false;   // tensor '.norm'
  int gate = 0;               // GATE_SILU or GATE_SIGMOID of W_g h
};

// Multi-head attention over cached latents with a shared rotated key part (interleaved pairs).
struct LatentMixer {
  int heads = 0, dim = 0, rot_dim = 0, vdim = 0, kv_rank = 0, q_rank = 0, rot_dims = 0;
  double rot_base = 1, scale = 1;
};

// Squared-ReLU experts chosen by a table of token ids, each with weight 1 / top.
struct TableExperts {
  int experts = 0, top = 0, ff = 0;
};

struct StackLayer {
  enum Kind { Linear, Latent } kind = Linear;
  LinearMixer linear;
  LatentMixer latent;
  bool has_ff = false;
  TableExperts ff;
};

struct StackSpec {
  int vocab = 0, width = 0, streams = 1;
  double eps = 0;
  std::vector<StackLayer> layers;
  std::vector<int> order;  // layer of every run, in the order they run (a looped layer appears several times)
};

// The hooks of ModelFamily for a stack.  stack_describe takes over the specification (the family's configure ends with it).
int stack_describe(blok_model *m, const StackSpec &spec);
int stack_build(blok_model *m, const char *dir, uint64_t seed);
void stack_destroy(blok_model *m);
int stack_layers(blok_model *m, int T, bool chunk, blok_stream_t stream);
int stack_sample(blok_model *m, int row, int n, uint32_t *next, blok_stream_t stream);
int stack_logits(blok_model *m, const int *rows, int n, float *out, blok_stream_t stream);
int stack_check(blok_model *m, blok_stream_t stream);

}  // namespace blok
