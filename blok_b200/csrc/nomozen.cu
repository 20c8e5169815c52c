// The Nomozen design: its config.json as a StackSpec.
//
//   layers[i].type  "retention":        linear attention, keys times dim^-1/2, a norm per head without weight, SiLU gate
//                   "lightning":        linear attention over SiLU projections, one weighted norm over all heads, sigmoid gate
//                   "latent_attention": attention over latents with a rotated key part shared by the heads
//   layers[i].mlp   null, or {"kind": "moe"}: squared-ReLU experts that a table of token ids chooses
//   loop            layers start .. stop - 1 run `times` times in a row with the same weights and caches of their own
#include <cmath>

#include "config_fields.h"
#include "stack.h"
#include "stack_kernels.h"

namespace blok {
namespace {

int read_linear(const Json *mixer, const std::string &where, bool lightning, LinearMixer *out) {
  Fields f(mixer, where);
  out->heads = f.size("heads");
  out->dim = f.size("dim");
  out->vdim = f.size("vdim");
  out->decay = f.numbers("decay");
  if (!f.rc() && (int)out->decay.size() != out->heads) f.fail("decay", "has not one entry per head");
  if (f.rc()) return f.rc();
  out->silu_qkv = lightning;
  out->k_scale = lightning ? 1.0 : 1.0 / std::sqrt((double)out->dim);
  out->norm_per_head = !lightning;
  out->norm_weight = lightning;
  out->gate = lightning ? GATE_SIGMOID : GATE_SILU;
  return BLOK_OK;
}

int read_latent(const Json *mixer, const std::string &where, LatentMixer *out) {
  Fields f(mixer, where);
  out->heads = f.size("heads");
  out->dim = f.size("dim");
  out->rot_dim = f.size("rot_dim");
  out->vdim = f.size("vdim");
  out->kv_rank = f.size("kv_rank");
  out->q_rank = f.size("q_rank");
  out->scale = f.number("scale");
  Fields rot = f.object("rot");
  out->rot_dims = rot.size("dims");
  out->rot_base = rot.number("base");
  if (f.rc()) return f.rc();
  if (!rot.rc() && (out->rot_dims > out->rot_dim || out->rot_dims % 2 || out->rot_base <= 0)) rot.fail("dims", "or base does not fit");
  return rot.rc();
}

int configure(blok_model *m, const Json &config) {
  Fields top(&config, "the model");
  StackSpec s;
  s.vocab = top.size("vocab");
  s.width = top.size("width");
  s.streams = top.size("streams");
  Fields norm = top.object("norm");
  s.eps = norm.number("eps");
  if (top.rc()) return top.rc();
  if (norm.rc()) return norm.rc();
  const Json *layers = config.find("layers");
  BLOK_REQUIRE(layers && layers->kind == Json::Array && !layers->items.empty(), BLOK_ERR_ARG, "config.json: no layers");
  for (size_t i = 0; i < layers->items.size(); ++i) {
    const std::string where = "layer " + std::to_string(i);
    const Json &j = layers->items[i];
    Fields f(&j, where);
    const std::string type = f.text("type");
    if (f.rc()) return f.rc();
    StackLayer L;
    const Json *mixer = j.find("mixer");
    int rc;
    if (type == "latent_attention") {
      L.kind = StackLayer::Latent;
      rc = read_latent(mixer, where + ".mixer", &L.latent);
    } else {
      BLOK_REQUIRE(type == "retention" || type == "lightning", BLOK_ERR_ARG, "config.json: %s: unknown type \"%s\"", where.c_str(), type.c_str());
      L.kind = StackLayer::Linear;
      rc = read_linear(mixer, where + ".mixer", type == "lightning", &L.linear);
    }
    if (rc) return rc;
    const Json *mlp = j.find("mlp");
    if (mlp && !mlp->is_null()) {
      Fields ff(mlp, where + ".mlp");
      const std::string kind = ff.text("kind");
      Fields router = ff.object("router"), expert = ff.object("expert");
      L.ff_kind = StackLayer::Experts;
      L.ff.experts = router.size("experts");
      L.ff.top = router.size("top");
      L.ff.ff = expert.size("ff");
      if (ff.rc()) return ff.rc();
      if (router.rc()) return router.rc();
      if (expert.rc()) return expert.rc();
      BLOK_REQUIRE(kind == "moe", BLOK_ERR_ARG, "config.json: %s: unknown feed-forward \"%s\"", where.c_str(), kind.c_str());
    }
    s.layers.push_back(L);
  }
  const int n = (int)s.layers.size();
  const Json *loop = config.find("loop");
  int start = 0, stop = 0, times = 1;
  if (loop && !loop->is_null()) {
    Fields f(loop, "loop");
    start = (int)f.number("start");
    stop = (int)f.number("stop");
    times = (int)f.number("times");
    if (f.rc()) return f.rc();
    BLOK_REQUIRE(start >= 0 && start <= stop && stop <= n && times >= 0, BLOK_ERR_ARG, "config.json: the loop does not fit %d layers", n);
  }
  for (int i = 0; i < start; ++i) s.order.push_back(i);
  for (int t = 0; t < times; ++t)
    for (int i = start; i < stop; ++i) s.order.push_back(i);
  for (int i = stop; i < n; ++i) s.order.push_back(i);
  return stack_describe(m, s);
}

const ModelFamily kNomozen = {"Nomozen", 2048, configure, stack_build, stack_destroy, stack_layers, stack_sample, stack_logits, stack_check};
const FamilyRegistration kRegistered(&kNomozen);

}  // namespace
}  // namespace blok
