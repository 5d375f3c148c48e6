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

bool need_float(const Json *o, const char *key, const std::string &where, float *out, std::string *err) {
  const Json *v = o ? o->get(key) : nullptr;
  if (!v || !v->as_float(out)) return fail(err, "config.json: " + where + "." + key + " must be a number");
  return true;
}
bool need_positive(const Json *o, const char *key, const std::string &where, double *out, std::string *err) {
  const Json *v = o ? o->get(key) : nullptr;
  if (!v || v->kind != Json::NUMBER || !(v->number > 0)) return fail(err, "config.json: " + where + "." + key + " must be a positive number");
  *out = v->number;
  return true;
}
// Rows of a tensor of the file, which has to be two-dimensional; with no file to ask, an optional key or a default.
bool rows_of(const ShapeOf &shape_of, const std::string &name, const Json *m, const char *key, const std::string &where, uint32_t fallback, uint32_t *out,
             std::string *err) {
  if (shape_of) {
    const std::vector<size_t> *s = shape_of(name);
    if (!s || s->size() != 2) return fail(err, "missing tensor " + name);
    *out = (uint32_t)(*s)[0];
    return true;
  }
  *out = fallback;
  return optional_u32(m, key, where, out, err);
}
bool taps_of(const ShapeOf &shape_of, const std::string &pre, const std::string &where, uint32_t *taps, std::string *err) {
  if (!shape_of) return true;
  const std::vector<size_t> *conv = shape_of(pre + "q.conv");
  const uint32_t n = conv && conv->size() == 2 ? (uint32_t)(*conv)[1] : 0;
  if (*taps && n != *taps) return fail(err, "config.json: " + where + ".conv does not match " + pre + "q.conv");
  *taps = n;
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
  }
  return taps_of(shape_of, pre, where, &s->taps, err);
}

bool delta_spec(const Json *m, const std::string &where, const std::string &pre, const ShapeOf &shape_of, MixerSpec *s, std::string *err) {
  s->kind = MixerKind::GENERAL_DELTA;
  if (!need_u32(m, "heads", where, &s->heads, err) || !need_u32(m, "dim", where, &s->dim, err)) return false;
  s->kv_heads = s->heads;
  s->vdim = s->dim;
  return rows_of(shape_of, pre + "w1", m, "rank", where, std::max(16u, s->dim / 2), &s->rank, err);
}

bool rotary_spec(const Json *r, const std::string &where, RotarySpec *s, std::string *err) {
  if (!need_u32(r, "dims", where, &s->dims, err) || !need_positive(r, "base", where, &s->base, err)) return false;
  if (s->dims % 2) return fail(err, "config.json: " + where + ".dims must be even");
  if (const Json *y = r->get("scaling"))
    return need_positive(y, "factor", where + ".scaling", &s->factor, err) && need_positive(y, "original", where + ".scaling", &s->original, err) &&
           need_positive(y, "fast", where + ".scaling", &s->fast, err) && need_positive(y, "slow", where + ".scaling", &s->slow, err);
  return true;
}

// Latent attention; low_rank_q: the queries pass a normed latent as well; gate: sigmoid gate on the output.
bool latent_spec(const Json *m, const std::string &where, const std::string &pre, const ShapeOf &shape_of, bool low_rank_q, bool sink, bool gate,
                 bool interleaved, MixerSpec *s, std::string *err) {
  s->kind = MixerKind::LATENT_ATTENTION;
  if (!need_u32(m, "heads", where, &s->heads, err) || !need_u32(m, "dim", where, &s->dim, err) || !need_u32(m, "rot_dim", where, &s->rot_dim, err) ||
      !need_u32(m, "vdim", where, &s->vdim, err) || !need_u32(m, "kv_rank", where, &s->kv_rank, err) || !need_float(m, "scale", where, &s->scale, err))
    return false;
  s->kv_heads = s->heads;
  if (low_rank_q) {
    if (!optional_u32(m, "q_rank", where, &s->q_rank, err)) return false;
    uint32_t rows = 0;
    if (!rows_of(shape_of, pre + "dq", m, "q_rank", where, s->q_rank, &rows, err)) return false;
    if (!rows || (s->q_rank && s->q_rank != rows)) return fail(err, "config.json: " + where + ".q_rank does not match " + pre + "dq");
    s->q_rank = rows;
  }
  s->sink = sink;
  s->gate = gate;
  const Json *rot = m->get("rot");
  if (!rot || !rotary_spec(rot, where + ".rot", &s->rotary, err)) return rot ? false : fail(err, "config.json: " + where + ".rot is missing");
  if (s->rotary.dims > s->rot_dim) return fail(err, "config.json: " + where + ".rot.dims exceeds rot_dim");
  s->rotary.interleaved = interleaved;
  return true;
}

// Gated delta rule with a decay per key channel.
bool gated_delta_spec(const Json *m, const std::string &where, const std::string &pre, const ShapeOf &shape_of, MixerSpec *s, std::string *err) {
  s->kind = MixerKind::GATED_DELTA;
  if (!need_u32(m, "heads", where, &s->heads, err) || !need_u32(m, "dim", where, &s->dim, err)) return false;
  s->kv_heads = s->heads;
  s->vdim = s->dim;
  if (!optional_u32(m, "kv_heads", where, &s->kv_heads, err) || !optional_u32(m, "vdim", where, &s->vdim, err) ||
      !optional_u32(m, "conv", where, &s->taps, err) || !taps_of(shape_of, pre, where, &s->taps, err))
    return false;
  if (s->kv_heads == 0 || s->heads % s->kv_heads || s->vdim == 0)
    return fail(err, "config.json: " + where + ": heads must be a multiple of kv_heads, vdim positive");
  if (s->taps == 0) return fail(err, "config.json: " + where + ".conv must be positive");
  const uint32_t fallback = std::max(16u, s->dim / 2);
  return rows_of(shape_of, pre + "a1", m, "decay_rank", where, fallback, &s->rank, err) &&
         rows_of(shape_of, pre + "g1", m, "gate_rank", where, fallback, &s->gate_rank, err);
}

// What the designs share: width, vocabulary, epsilon, and the list of layers; mixer_of reads a layer's mixer by its type.
using MixerOf = std::function<bool(const std::string &type, const Json *mixer, const std::string &where, const std::string &pre, MixerSpec *s, std::string *err)>;
bool configure_layers(const Json &j, const MixerOf &mixer_of, int ff_act, bool parallel, ModelConfig *c, std::string *err) {
  c->arch = ModelArch::HYBRID;
  c->weight_type = c->lm_head_type = gcore::rt::GretaDataType::BF16;
  if (!need_u32(&j, "width", "model", &c->dim, err) || !need_u32(&j, "vocab", "model", &c->vocab_size, err)) return false;
  const Json *layers = j.get("layers");
  if (!need_float(j.get("norm"), "eps", "norm", &c->rms_eps, err)) return false;
  if (!layers || layers->kind != Json::ARRAY || layers->items.empty()) return fail(err, "config.json: layers must be a list");
  c->layers.clear();
  for (size_t i = 0; i < layers->items.size(); ++i) {
    const Json &l = layers->items[i];
    const std::string where = "layers[" + std::to_string(i) + "]", pre = "l" + std::to_string(i) + ".mix.";
    const Json *type = l.get("type"), *mixer = l.get("mixer"), *mlp = l.get("mlp");
    if (!type || type->kind != Json::STRING || !mixer || mixer->kind != Json::OBJECT) return fail(err, "config.json: " + where + " needs a type and a mixer");
    LayerSpec s;
    s.ff_act = ff_act;
    s.parallel = parallel;
    if (!mixer_of(type->string, mixer, where + ".mixer", pre, &s.mixer, err)) return false;
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
bool unknown_type(const std::string &type, const std::string &where, std::string *err) {
  return fail(err, "config.json: " + where + ": unknown layer type \"" + type + "\"");
}

// "Bidonex": learned positions, parallel layers of windowed attention or generalised delta rule beside a gelu feed-forward.
bool configure_bidonex(const Json &j, const ShapeOf &shape_of, ModelConfig *c, std::string *err) {
  auto mixer_of = [&](const std::string &type, const Json *m, const std::string &where, const std::string &pre, MixerSpec *s, std::string *e) {
    if (type == "attention") return attention_spec(m, where, pre, shape_of, s, e);
    if (type == "general_delta") return delta_spec(m, where, pre, shape_of, s, e);
    return unknown_type(type, where, e);
  };
  return need_u32(&j, "max_positions", "model", &c->max_seq_len, err) && configure_layers(j, mixer_of, GRETA_ACT_GELU_ERF, true, c, err);
}

// "Tetilorn": scaled embedding tied to the LM head, root-mean-square norms, sequential layers of latent attention (two forms) or gated
// delta rule with a decay per channel, each with an optional squared-relu feed-forward behind it.
bool configure_tetilorn(const Json &j, const ShapeOf &shape_of, ModelConfig *c, std::string *err) {
  auto mixer_of = [&](const std::string &type, const Json *m, const std::string &where, const std::string &pre, MixerSpec *s, std::string *e) {
    if (type == "latent_attention") return latent_spec(m, where, pre, shape_of, true, true, true, false, s, e);
    if (type == "latent_attention_2") return latent_spec(m, where, pre, shape_of, false, false, false, true, s, e);
    if (type == "channel_delta") return gated_delta_spec(m, where, pre, shape_of, s, e);
    return unknown_type(type, where, e);
  };
  c->max_seq_len = 1u << 20;  // nothing in the design bounds it
  c->default_seq_len = 8192;
  c->learned_positions = false;
  c->rms_norms = c->tied_head = true;
  return need_float(j.get("embedding"), "scale", "embedding", &c->embed_scale, err) && configure_layers(j, mixer_of, GRETA_ACT_RELU2, false, c, err);
}

struct Family {
  const char *name;
  bool (*configure)(const Json &, const ShapeOf &, ModelConfig *, std::string *);
};
const Family kFamilies[] = {{"Bidonex", configure_bidonex}, {"Tetilorn", configure_tetilorn}};

}  // namespace

std::vector<double> RotarySpec::frequencies(double *amplitude) const {
  std::vector<double> f(dims / 2);
  for (size_t i = 0; i < f.size(); ++i) f[i] = std::pow(base, -2.0 * (double)i / dims);
  *amplitude = 1.0;
  if (factor <= 0) return f;
  // YaRN: pairs that turn fewer than `slow` times over the original context are slowed by the factor, those above `fast` are left.
  auto where = [&](double turns) { return dims * std::log(original / (2.0 * 3.14159265358979323846 * turns)) / (2.0 * std::log(base)); };
  const double lo = std::max(std::floor(where(fast)), 0.0), hi = std::min(std::ceil(where(slow)), dims - 1.0);
  for (size_t i = 0; i < f.size(); ++i) {
    const double ramp = std::min(std::max(((double)i - lo) / std::max(hi - lo, 0.001), 0.0), 1.0);
    f[i] = f[i] / factor * ramp + f[i] * (1.0 - ramp);
  }
  *amplitude = 0.1 * std::log(factor) + 1.0;
  return f;
}

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
