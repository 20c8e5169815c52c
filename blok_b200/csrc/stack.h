// Models that are a stack of layers between an embedding and a vocabulary product, described by values: every layer is a
// token mixer and, usually, a feed-forward, each behind a norm and added to the residual.  Two forms of residual:
//   streams    several streams that mix (hyper-connections), a Dynamic-Tanh norm in front of every sublayer
//   sandwich   one residual, x <- x + mult * post_norm(sublayer(norm(x))), layer norms
// A design (nomozen.cu, pamopel.cu) turns its config.json into a StackSpec; the runtime is model_stack.cu.
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

// Selective state space with a scalar decay per head and token (Mamba-2): convolved inputs, the recurrence, a SiLU gate in
// front of a norm over `norm_groups` equal parts.  `groups` sets of (B, C) are shared by heads / groups heads each.
struct StateMixer {
  int heads = 0, vdim = 0, state = 0, groups = 1, taps = 1, norm_groups = 1;
};

// Softmax attention with heads / kv_heads query heads per key head.
struct GroupedMixer {
  int heads = 0, kv_heads = 0, dim = 0, vdim = 0;
  double scale = 1;
  bool qk_norm = false;  // RMS norm over all of q and all of k: tensors '.q.norm', '.k.norm'
  double bias_max = 0;   // > 0: tensor '.rel' [buckets, heads] is added to the scores by distance; it saturates here
  bool head_gate = false;  // tensor '.g': every head's output times a sigmoid
  int kv_from = -1;      // >= 0: the keys and values are this earlier layer's
};

// Squared-ReLU experts chosen by a table of token ids, each with weight 1 / top.
struct TableExperts {
  int experts = 0, top = 0, ff = 0;
};

// W_down (silu(W_gate h) * (W_up h))
struct DenseGated {
  int ff = 0;
};

struct StackLayer {
  enum Kind { Linear, Latent, State, Grouped } kind = Linear;
  LinearMixer linear;
  LatentMixer latent;
  StateMixer state;
  GroupedMixer grouped;
  enum FfKind { NoFf, Experts, Dense } ff_kind = NoFf;
  TableExperts ff;
  DenseGated dense;
};

struct StackSpec {
  int vocab = 0, width = 0, streams = 1;
  double eps = 0;
  // embedding: embed_scale * embed[token] (+ a row of 'bigram' chosen by the previous and the current token, or its last row
  // at a sequence's start) (+ a sinusoidal vector of the position); the last two with the sandwich form only
  double embed_scale = 1;
  int bigram_buckets = 0;  // 0: none
  long bigram_mul_prev = 0, bigram_mul_cur = 0;
  bool sinusoid = false;
  bool sandwich = false;
  double residual_mult = 1;  // sandwich
  double logit_scale = 1;    // sandwich
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
