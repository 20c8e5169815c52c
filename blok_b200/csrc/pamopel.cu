// The Pamopel design: its config.json as a StackSpec.
//
//   layers[i].type  "mamba2":     selective state space, the gate in front of a norm over parts
//                   "attention":  grouped softmax attention, norms over all of q and k, a learned bias per distance, a gate per
//                                 head; "kv_from" borrows an earlier layer's keys and values
//   layers[i].mlp   null, or {"kind": "dense"}: SiLU-gated feed-forward
//   embedding       scaled, plus a row chosen by the previous and the current token, plus a sinusoid of the position
#include "config_fields.h"
#include "stack.h"

namespace blok {
namespace {

int read_state(const Json *mixer, const std::string &where, StateMixer *out) {
  Fields f(mixer, where);
  out->heads = f.size("heads");
  out->vdim = f.size("vdim");
  out->state = f.size("state");
  out->groups = f.size("groups");
  out->taps = f.size("conv");
  out->norm_groups = f.size("norm_groups");
  if (f.rc()) return f.rc();
  if (out->heads % out->groups) f.fail("groups", "does not divide the heads");
  if (out->heads * out->vdim % out->norm_groups) f.fail("norm_groups", "does not divide the inner size");
  return f.rc();
}

int read_grouped(const Json *mixer, const std::string &where, const std::vector<StackLayer> &before, GroupedMixer *out) {
  Fields f(mixer, where);
  out->heads = f.size("heads");
  out->kv_heads = f.size("kv_heads");
  out->dim = f.size("dim");
  out->vdim = f.size("vdim");
  out->scale = f.number("scale");
  out->bias_max = f.number("bias_max");
  out->qk_norm = out->head_gate = true;
  if (f.rc()) return f.rc();
  if (out->heads % out->kv_heads) f.fail("kv_heads", "does not divide the heads");
  if (out->bias_max < 1) f.fail("bias_max", "is not a distance");
  if (f.has("kv_from")) {
    const double j = f.number("kv_from");
    if (f.rc()) return f.rc();
    const bool known = j >= 0 && j == std::floor(j) && j < (double)before.size() && before[(size_t)j].kind == StackLayer::Grouped;
    const GroupedMixer *from = known ? &before[(size_t)j].grouped : nullptr;
    if (!from || from->kv_from >= 0 || from->kv_heads != out->kv_heads || from->dim != out->dim || from->vdim != out->vdim)
      f.fail("kv_from", "names no earlier attention layer with keys and values of these sizes");
    out->kv_from = (int)j;
  }
  return f.rc();
}

int configure(blok_model *m, const Json &config) {
  Fields top(&config, "the model");
  StackSpec s;
  s.vocab = top.size("vocab");
  s.width = top.size("width");
  s.sandwich = true;
  s.sinusoid = true;
  s.residual_mult = top.number("residual_mult");
  s.logit_scale = top.number("logit_scale");
  Fields norm = top.object("norm"), embedding = top.object("embedding");
  s.eps = norm.number("eps");
  s.embed_scale = embedding.number("scale");
  Fields bigram = embedding.object("bigram");
  s.bigram_buckets = bigram.size("buckets");
  s.bigram_mul_prev = (long)bigram.number("mul_prev");
  s.bigram_mul_cur = (long)bigram.number("mul_cur");
  for (const Fields *f : {&top, &norm, &embedding, &bigram})
    if (f->rc()) return f->rc();
  BLOK_REQUIRE(s.bigram_mul_prev >= 0 && s.bigram_mul_cur >= 0, BLOK_ERR_ARG, "config.json: embedding.bigram: a factor is negative");
  const Json *layers = config.find("layers");
  BLOK_REQUIRE(layers && layers->kind == Json::Array && !layers->items.empty(), BLOK_ERR_ARG, "config.json: no layers");
  for (size_t i = 0; i < layers->items.size(); ++i) {
    const std::string where = "layer " + std::to_string(i);
    const Json &j = layers->items[i];
    Fields f(&j, where);
    const std::string type = f.text("type");
    if (f.rc()) return f.rc();
    StackLayer L;
    const Json *mixer = j.find("mixer"), *mlp = j.find("mlp");
    int rc;
    if (type == "attention") {
      L.kind = StackLayer::Grouped;
      rc = read_grouped(mixer, where + ".mixer", s.layers, &L.grouped);
    } else {
      BLOK_REQUIRE(type == "mamba2", BLOK_ERR_ARG, "config.json: %s: unknown type \"%s\"", where.c_str(), type.c_str());
      L.kind = StackLayer::State;
      rc = read_state(mixer, where + ".mixer", &L.state);
    }
    if (rc) return rc;
    if (mlp && !mlp->is_null()) {
      Fields ff(mlp, where + ".mlp");
      const std::string kind = ff.text("kind");
      if (ff.rc()) return ff.rc();
      BLOK_REQUIRE(kind == "dense", BLOK_ERR_ARG, "config.json: %s: unknown feed-forward \"%s\"", where.c_str(), kind.c_str());
      L.ff_kind = StackLayer::Dense;
      L.dense.ff = ff.size("ff");
      if (ff.rc()) return ff.rc();
    }
    s.layers.push_back(L);
    s.order.push_back((int)i);
  }
  return stack_describe(m, s);
}

const ModelFamily kPamopel = {"Pamopel", 2048, configure, stack_build, stack_destroy, stack_layers, stack_sample, stack_logits, stack_check};
const FamilyRegistration kRegistered(&kPamopel);

}  // namespace
}  // namespace blok
