// Model registry: which architectures a config.json may name, and how each one's configuration becomes a ModelConfig.
// A design is described by its layers; nothing below or after this file depends on a particular model's sizes.
#include <algorithm>
#include <cmath>

#include "gcore/greta_b200.hpp"
#include "host_util.hpp"
#include "json.hpp"

namespace gcore::inference {

using gcore::host::fail;
using gcore::host::Json;

namespace {

bool need_u32(const Json *o, const char *key, const std::string &where, uint32_t *out, std::string *err) {
  const Json *v = o ? o->get(key) : nullptr;
  if (!v || !v->as_u32(out) || *out == 0) return fail(err, "config.json: " + where + "." + key + " must be a positive whole number");
  return true;
}
bool optional_u32(const Json *o, const char *key, const std::string &where, uint32_t *out, std::string *err) {
  const Json *v = o ? o->get(key) : nullptr;
  if (v && !v->as_u32(out)) return fail(err, "config.json: " + where + "." + key + " must be a whole number");
  return true;
}
bool optional_float(const Json *o, const char *key, const std::string &where, float *out, std::string *err) {
  const Json *v = o ? o->get(key) : nullptr;
  if (v && !v->as_float(out)) return fail(err, "config.json: " + where + "." + key + " must be a number");
  return true;
}

bool attention_spec(const Json *m, const std::string &where, const std::string &pre, const ShapeOf &shape_of, MixerSpec *s, std::string *err) {
  s->kind = MixerKind::WINDOW_ATTENTION;
  if (!need_u32(m, "heads", where, &s->heads, err) || !need_u32(m, "dim", where, &s->dim, err)) return false;
  s->kv_heads = s->heads;
  s->vdim = s->dim;
  s->scale = 1.0f / std::sqrt((float)s->dim);
  if (!optional_u32(m, "kv_heads", where, &s->kv_heads, err) || !optional_u32(m, "vdim", where, &s->vdim, err) ||
      !optional_u32(m, "conv", where, &s->taps, err) || !optional_float(m, "scale", where, &s->scale, err) ||
      !optional_float(m, "softcap", where, &s->softcap, err))
    return false;
  if (const Json *mask = m->get("mask")) {
    if (!need_u32(mask, "size", where + ".mask", &s->window, err) || !optional_u32(mask, "keep_first", where + ".mask", &s->keep_first, err)) return false;
  }
  if (s->kv_heads == 0 || s->heads % s->kv_heads || s->vdim == 0)
    return fail(err, "config.json: " + where + ": heads must be a multiple of kv_heads, vdim positive");
  s->temp = s->distance_bias = s->sink = true;
  if (shape_of) {
    s->temp = shape_of(pre + "temp") != nullptr;
    s->distance_bias = shape_of(pre + "r1") != nullptr;
    s->sink = shape_of(pre + "sink") != nullptr;
    const std::vector<size_t> *conv = shape_of(pre + "q.conv");
    const uint32_t taps = conv && conv->size() == 2 ? (uint32_t)(*conv)[1] : 0;
    if (s->taps && taps != s->taps) return fail(err, "config.json: " + where + ".conv does not match " + pre + "q.conv");
    s->taps = taps;
  }
  return true;
}

bool delta_spec(const Json *m, const std::string &where, const std::string &pre, const ShapeOf &shape_of, MixerSpec *s, std::string *err) {
  s->kind = MixerKind::GENERAL_DELTA;
  if (!need_u32(m, "heads", where, &s->heads, err) || !need_u32(m, "dim", where, &s->dim, err)) return false;
  s->kv_heads = s->heads;
  s->vdim = s->dim;
  if (shape_of) {
    const std::vector<size_t> *w1 = shape_of(pre + "w1");
    if (!w1 || w1->size() != 2) return fail(err, "missing tensor " + pre + "w1");
    s->rank = (uint32_t)(*w1)[0];
    return true;
  }
  s->rank = std::max(16u, s->dim / 2);  // no file to ask: a width for synthetic weights
  return optional_u32(m, "rank", where, &s->rank, err);
}

// "Bidonex": learned positions, parallel layers of windowed attention or generalised delta rule beside a gelu feed-forward.
bool configure_bidonex(const Json &j, const ShapeOf &shape_of, ModelConfig *c, std::string *err) {
  c->arch = ModelArch::HYBRID;
  c->weight_type = c->lm_head_type = gcore::rt::GretaDataType::BF16;
  if (!need_u32(&j, "width", "model", &c->dim, err) || !need_u32(&j, "vocab", "model", &c->vocab_size, err) ||
      !need_u32(&j, "max_positions", "model", &c->max_seq_len, err))
    return false;
  const Json *norm = j.get("norm"), *layers = j.get("layers");
  const Json *eps = norm ? norm->get("eps") : nullptr;
  if (!eps || !eps->as_float(&c->rms_eps)) return fail(err, "config.json: norm.eps must be a number");
  if (!layers || layers->kind != Json::ARRAY || layers->items.empty()) return fail(err, "config.json: layers must be a list");
  c->layers.clear();
  for (size_t i = 0; i < layers->items.size(); ++i) {
    const Json &l = layers->items[i];
    const std::string where = "layers[" + std::to_string(i) + "]", pre = "l" + std::to_string(i) + ".mix.";
    const Json *type = l.get("type"), *mixer = l.get("mixer"), *mlp = l.get("mlp");
    if (!type || type->kind != Json::STRING || !mixer || mixer->kind != Json::OBJECT) return fail(err, "config.json: " + where + " needs a type and a mixer");
    LayerSpec s;
    if (type->string == "attention") {
      if (!attention_spec(mixer, where + ".mixer", pre, shape_of, &s.mixer, err)) return false;
    } else if (type->string == "general_delta") {
      if (!delta_spec(mixer, where + ".mixer", pre, shape_of, &s.mixer, err)) return false;
    } else {
      return fail(err, "config.json: " + where + ": unknown layer type \"" + type->string + "\"");
    }
    if (mlp) {
      const Json *kind = mlp->get("kind");
      if (!kind || kind->kind != Json::STRING || kind->string != "dense") return fail(err, "config.json: " + where + ".mlp: unknown kind");
      if (!need_u32(mlp, "ff", where + ".mlp", &s.ff, err)) return false;
    }
    c->layers.push_back(s);
  }
  c->num_layers = (uint32_t)c->layers.size();
  c->num_heads = c->layers[0].mixer.heads;
  c->num_heads_kv = c->layers[0].mixer.kv_heads;
  c->head_dim = c->layers[0].mixer.dim;
  c->hidden_dim = c->layers[0].ff;
  return true;
}

struct Family {
  const char *name;
  bool (*configure)(const Json &, const ShapeOf &, ModelConfig *, std::string *);
};
const Family kFamilies[] = {{"Bidonex", configure_bidonex}};

}  // namespace

std::vector<std::string> registered_architectures() {
  std::vector<std::string> v;
  for (const Family &f : kFamilies) v.push_back(f.name);
  return v;
}

bool config_from_json(const std::string &text, const ShapeOf &shape_of, ModelConfig *out, std::string *err) {
  Json j;
  if (!Json::parse(text, &j, err)) return false;
  const Json *arch = j.get("architecture");
  if (!arch || arch->kind != Json::STRING) return fail(err, "config.json: no architecture");
  for (const Family &f : kFamilies)
    if (arch->string == f.name) {
      *out = ModelConfig{};
      out->architecture = f.name;
      return f.configure(j, shape_of, out, err);
    }
  return fail(err, "config.json: architecture \"" + arch->string + "\" is not registered");
}

}  // namespace gcore::inference
