// BlockScheduler, hybrid designs: x += mixer(LN(x)) + ff(LN(x)) with attention or recurrent mixers over unquantised weights.
//
// Both sublayers read the same norm, so a layer is two matrix products around the mixer's core:
//   1. LN -> every input projection of mixer and feed-forward (w_in), activations in the epilogue
//   2. the mixer's core: windowed attention over the cache, or the delta rule over the state
//   3. [mixer | feed-forward] columns -> both output projections and the residual (w_out)
// For a single row (decode; up to 8 in fp32) 1 and 3 are GEMVs with the norm fused in: three kernels per layer and decode
// step.  More rows run on the tensor cores (bf16) behind one layer-norm kernel.  The residual stream, the projections that enter a
// mixer, scores, states and norms are fp32 in either mode.
//
// Caches and states belong to the scheduler's sequence slots and hold no trace of earlier sequences: positions in front of a
// sequence's start are never read, and a delta state starts from zero at position 0.
#include <algorithm>
#include <cmath>
#include <cstring>

#include "gcore/greta_b200.hpp"
#include "host_util.hpp"

namespace gcore::inference {

using gcore::host::fail;
using gcore::rt::GretaDataType;
using gcore::rt::cuda::Buffer;
using gcore::rt::cuda::BufferUsage;
using gcore::rt::cuda::GretaStreamCuda;

namespace {

inline cudaStream_t H(gcore::rt::GretaStream *s) { return static_cast<GretaStreamCuda *>(s)->handle(); }
inline uint32_t up(uint32_t n, uint32_t to) { return (n + to - 1) / to * to; }
constexpr uint32_t FEW_ROWS = 8;       // fp32 weights: rows up to which the linears run as GEMVs
constexpr uint32_t FEW_ROWS_BF16 = 1;  // bf16: the tensor-core kernel streams the weights as fast for two rows as the GEMV for one
constexpr uint32_t MMA_MIN_ROWS = 16;  // portions from which attention runs on the tensor cores

#define GRETA_TRY(call, what)                                                \
  do {                                                                       \
    if ((call) != GRETA_OK) return fail(err, gcore::host::cuda_error(what)); \
  } while (0)

uint16_t f32_to_bf16(float f) {  // round to nearest even
  uint32_t x;
  std::memcpy(&x, &f, 4);
  if ((x & 0x7FFFFFFFu) > 0x7F800000u) return (uint16_t)((x >> 16) | 0x40u);
  return (uint16_t)((x + 0x7FFFu + ((x >> 16) & 1u)) >> 16);
}

// A weight packed on the host: [rows][ld] in bf16 or fp32, zero where nothing is put.
struct Packed {
  bool bf16;
  uint32_t rows, ld;
  std::vector<uint16_t> h;
  std::vector<float> f;
  Packed(bool b, uint32_t r, uint32_t l) : bf16(b), rows(r), ld(l) {
    if (b) h.assign((size_t)r * l, 0);
    else f.assign((size_t)r * l, 0.f);
  }
  void put(const std::vector<float> &src, uint32_t r, uint32_t cols, uint32_t row0, uint32_t col0) {
#pragma omp parallel for schedule(static)
    for (uint32_t i = 0; i < r; ++i)
      for (uint32_t j = 0; j < cols; ++j) {
        const size_t at = (size_t)(row0 + i) * ld + col0 + j;
        if (bf16) h[at] = f32_to_bf16(src[(size_t)i * cols + j]);
        else f[at] = src[(size_t)i * cols + j];
      }
  }
  bool upload(Buffer &b, std::string *err) const {
    const size_t bytes = (size_t)rows * ld * (bf16 ? 2 : 4);
    if (!b.allocate(bytes, BufferUsage::DeviceOnly, bf16 ? GretaDataType::BF16 : GretaDataType::FP32, err)) return false;
    return b.copy_to_device(bf16 ? (const void *)h.data() : (const void *)f.data(), bytes, err);
  }
};

bool upload_f32(Buffer &b, const std::vector<float> &v, std::string *err) {
  return b.allocate(std::max<size_t>(16, v.size() * 4), BufferUsage::DeviceOnly, GretaDataType::FP32, err) && b.copy_to_device(v.data(), v.size() * 4, err);
}
const float *fp(const Buffer &b) { return static_cast<const float *>(b.data()); }

}  // namespace

// Where the weights come from: values(name) as fp32, checked against the expected shape.
class BlockScheduler::TensorSource {
public:
  virtual ~TensorSource() = default;
  virtual bool values(const std::string &name, const std::vector<size_t> &shape, std::vector<float> *out, std::string *err) = 0;
};

struct BlockScheduler::FileSource : BlockScheduler::TensorSource {
  SafetensorsLoader &loader;
  explicit FileSource(SafetensorsLoader &l) : loader(l) {}
  bool values(const std::string &name, const std::vector<size_t> &shape, std::vector<float> *out, std::string *err) override {
    const TensorInfo *t = loader.find(name);
    if (!t) return fail(err, "load_weights: missing tensor " + name);
    if (t->shape != shape) return fail(err, "load_weights: unexpected shape of " + name);
    return loader.read_floats(name, out, err);
  }
};

// Seeded normal weights scaled by their fan-in, norms near one: the layers stay of order one whatever their sizes.
struct BlockScheduler::SynthSource : BlockScheduler::TensorSource {
  uint64_t seed;
  explicit SynthSource(uint64_t s) : seed(s) {}
  bool values(const std::string &name, const std::vector<size_t> &shape, std::vector<float> *out, std::string *) override {
    size_t n = 1;
    for (size_t d : shape) n *= d;
    uint64_t stream = 0x5bd1e995u;  // FNV-style hash of the name
    for (char c : name) stream = (stream ^ (uint8_t)c) * 0x100000001b3ull;
    auto ends = [&](const char *s) { const size_t k = std::strlen(s); return name.size() >= k && name.compare(name.size() - k, k, s) == 0; };
    float sigma = shape.size() == 2 ? 1.f / std::sqrt((float)shape[1]) : 0.1f, mean = 0.f;
    if (name == "embed") sigma = 1.f;
    if (name == "pos") sigma = 0.1f;
    if (ends("norm") || ends("norm1") || ends(".temp")) mean = 1.f;
    if (ends(".r1")) mean = 0.5f;
    if (ends(".r2")) mean = 1.f;
    out->resize(n);
    synth::normal_f32(seed, stream, sigma, out->data(), 0, n);
    if (mean != 0.f)
      for (float &v : *out) v = std::fabs(v + mean);
    return true;
  }
};

bool BlockScheduler::init_hybrid(std::string *err) {
  const ModelConfig &c = config_;
  if (c.tp_size != 1) return fail(err, "init: hybrid designs run on one GPU (no tensor parallelism)");
  if (c.weight_type != GretaDataType::BF16 && c.weight_type != GretaDataType::FP32) return fail(err, "init: a hybrid design's weight_type must be BF16 or FP32");
  if (c.layers.empty() || c.layers.size() != c.num_layers || !c.dim || !c.vocab_size || !c.prefill_chunk) return fail(err, "init: incomplete hybrid configuration");
  for (const LayerSpec &l : c.layers) {
    const MixerSpec &m = l.mixer;
    if (m.dim > 256 || m.vdim > 256) return fail(err, "init: head sizes above 256 are not supported");
    if (m.kind == MixerKind::GENERAL_DELTA && (!m.rank || m.rank > 8192)) return fail(err, "init: general delta needs a low-rank width of 1..8192");
  }
  if (gcore::rt::GretaContext::instance().initialize() != gcore::rt::GretaResult::SUCCESS)
    return fail(err, "init: no usable CUDA device (this path has no CPU fallback)");
  vocab_l_ = c.vocab_size;
  stream_ = gcore::rt::GretaContext::instance().create_stream();
  blocks_.clear();
  hybrid_.clear();
  initialized_ = true;
  return true;
}

bool BlockScheduler::load_hybrid_file(SafetensorsLoader &loader, std::string *err) {
  FileSource src(loader);
  return load_hybrid(src, err);
}
bool BlockScheduler::load_hybrid_synthetic(uint64_t seed, std::string *err) {
  SynthSource src(seed);
  return load_hybrid(src, err);
}

bool BlockScheduler::load_hybrid(TensorSource &src, std::string *err) {
  const ModelConfig &c = config_;
  if (hybrid_.size() != c.num_layers) return fail(err, "load_weights: allocate_weights first");
  const bool bf16 = c.weight_type == GretaDataType::BF16;
  const uint32_t D = c.dim;
  std::vector<float> v;
  weight_bytes_ = 0;
  auto vec = [&](const std::string &name, uint32_t n, Buffer &b) { return src.values(name, {n}, &v, err) && upload_f32(b, v, err); };
  for (uint32_t l = 0; l < c.num_layers; ++l) {
    const LayerSpec &s = c.layers[l];
    const MixerSpec &m = s.mixer;
    HybridLayerBuffers &b = hybrid_[l];
    const std::string pre = "l" + std::to_string(l) + ".", mix = pre + "mix.";
    const bool delta = m.kind == MixerKind::GENERAL_DELTA;
    const uint32_t HD = m.heads * m.dim, HV = m.out_cols(), GD = m.kv_heads * m.dim, GV = m.kv_heads * m.vdim;
    if (!vec(pre + "norm1", D, b.norm_w) || !vec(pre + "norm1.b", D, b.norm_b)) return false;
    b.in_rows = m.proj_cols() + (delta ? m.rank : 0) + s.ff;
    b.in_ld = up(D, 64);
    b.ff_col = up(HV, 64);
    b.out_cols = s.ff ? b.ff_col + s.ff : HV;
    b.out_ld = up(b.out_cols, 64);
    Packed in(bf16, b.in_rows, b.in_ld), out(bf16, D, b.out_ld);
    uint32_t row = 0;
    auto rows = [&](const std::string &name, uint32_t n) {
      if (!src.values(name, {n, D}, &v, err)) return false;
      in.put(v, n, D, row, 0);
      row += n;
      return true;
    };
    auto cols = [&](const std::string &name, uint32_t n, uint32_t col) {
      if (!src.values(name, {D, n}, &v, err)) return false;
      out.put(v, D, n, 0, col);
      return true;
    };
    if (delta) {
      for (const char *n : {"r", "k", "v", "g", "a"})
        if (!rows(mix + n, HD)) return false;
      if (!rows(mix + "w1", m.rank)) return false;
      if (!vec(mix + "a.b", HD, b.a_bias) || !vec(mix + "w0", HD, b.w0) || !vec(mix + "norm", HD, b.out_norm)) return false;
      if (!src.values(mix + "w2", {HD, m.rank}, &v, err) || !upload_f32(b.w2, v, err)) return false;
      // Portions multiply w2 as a dense linear.  In bf16 the activations travel as a pair (hi, lo), so w2 stands there twice.
      const uint32_t second = up(m.rank, 8);
      b.w2_ld = up(bf16 ? 2 * second : m.rank, 64);
      Packed w2(bf16, HD, b.w2_ld);
      w2.put(v, HD, m.rank, 0, 0);
      if (bf16) w2.put(v, HD, m.rank, 0, second);
      if (!w2.upload(b.w2_packed, err)) return false;
      weight_bytes_ += b.w2.size();
    } else {
      if (!rows(mix + "q", HD) || !rows(mix + "k", GD) || !rows(mix + "v", GV)) return false;
      if (m.temp && !vec(mix + "temp", m.heads, b.temp)) return false;
      if (m.distance_bias && (!vec(mix + "r1", m.heads, b.r1) || !vec(mix + "r2", m.heads, b.r2))) return false;
      if (m.sink && !vec(mix + "sink", m.heads, b.sink)) return false;
      if (m.taps) {
        std::vector<float> all;
        const std::pair<const char *, uint32_t> parts[3] = {{"q", HD}, {"k", GD}, {"v", GV}};
        for (const auto &p : parts) {
          if (!src.values(mix + p.first + ".conv", {p.second, m.taps}, &v, err)) return false;
          all.insert(all.end(), v.begin(), v.end());
        }
        if (!upload_f32(b.conv, all, err)) return false;
      }
    }
    if (s.ff && (!rows(pre + "mlp.up", s.ff) || !cols(pre + "mlp.down", s.ff, b.ff_col))) return false;
    if (!cols(mix + "o", HV, 0)) return false;
    if (!in.upload(b.w_in, err) || !out.upload(b.w_out, err)) return false;
    weight_bytes_ += b.w_in.size() + b.w_out.size();
  }
  auto table = [&](const std::string &name, uint32_t n, uint32_t ld, Buffer &b) {
    if (!src.values(name, {n, D}, &v, err)) return false;
    Packed p(bf16, n, ld);
    p.put(v, n, D, 0, 0);
    return p.upload(b, err);
  };
  head_ld_ = up(D, 64);
  if (!table("embed", c.vocab_size, D, token_embd_) || !table("pos", c.max_seq_len, D, pos_embd_) || !table("head", c.vocab_size, head_ld_, output_weight_))
    return false;
  if (!vec("final.norm", D, output_norm_) || !vec("final.norm.b", D, final_norm_b_)) return false;
  weight_bytes_ += output_weight_.size();
  GRETA_TRY(greta_cuda_device_synchronize(), "load_weights");
  return true;
}

bool BlockScheduler::allocate_hybrid_activations(std::string *err) {
  const ModelConfig &c = config_;
  if (max_seq_ == 0 || max_seq_ > c.max_seq_len)
    return fail(err, "allocate_activations: max_seq_len must be 1.." + std::to_string(c.max_seq_len) + " (the model's learned positions)");
  const bool bf16 = c.weight_type == GretaDataType::BF16;
  const uint32_t chunk = (uint32_t)std::min<size_t>(c.prefill_chunk, max_seq_), B = batch_, R = std::max(chunk, B), D = c.dim, cb = bf16 ? 2 : 4;
  ActivationBuffers &a = activations_;
  HybridActivations &w = hact_;
  auto zeroed = [&](Buffer &b, size_t bytes, GretaDataType t = GretaDataType::FP32) {
    if (!b.allocate(std::max<size_t>(bytes, 16), BufferUsage::DeviceOnly, t, err)) return false;
    GRETA_TRY(greta_cuda_memset(b.data(), 0, b.size(), nullptr), "allocate_activations");
    return true;
  };
  uint32_t proj = 4, cat = 64, q = 4, o = 4, rank = 0, hd = 0;
  for (uint32_t l = 0; l < c.num_layers; ++l) {
    const MixerSpec &m = c.layers[l].mixer;
    const uint32_t ff_col = up(m.out_cols(), 64);
    proj = std::max(proj, up(m.proj_cols(), 4));
    cat = std::max(cat, c.layers[l].ff ? ff_col + up(c.layers[l].ff, 64) : ff_col);
    if (m.kind == MixerKind::GENERAL_DELTA) {
      o = std::max(o, m.heads * m.dim);
      rank = std::max(rank, m.rank);
      hd = std::max(hd, m.heads * m.dim);
    } else {
      q = std::max(q, m.heads * up(m.dim, 8));
    }
  }
  w.h_ld = up(D, 64);
  w.proj_ld = proj;
  w.cat_ld = cat;
  w.low_ld = up(rank, 64);
  w.low16_ld = up(2 * up(rank, 8), 64);
  w.decay_ld = up(hd, 4);
  if (!zeroed(a.x, (size_t)R * D * 4) || !zeroed(a.tokens, (size_t)R * 4) || !zeroed(a.d_pos, 2 * (size_t)B * 4) || !zeroed(a.d_next, (size_t)B * 4) ||
      !zeroed(a.out_tokens, (size_t)B * max_seq_ * 4) || !zeroed(logits_, (size_t)B * c.vocab_size * 4))
    return false;
  const size_t few = bf16 ? std::min(R, FEW_ROWS_BF16) : R;
  if (!zeroed(w.h, (size_t)R * w.h_ld * cb) || !zeroed(w.proj, (size_t)R * proj * 4) || !zeroed(w.cat, few * cat * 4) ||
      (bf16 && !zeroed(w.cat16, (size_t)R * cat * 2)) || !zeroed(w.q, (size_t)R * q * 4) || !zeroed(w.x_rows, (size_t)64 * D * 4) ||
      !zeroed(w.logits_rows, (size_t)64 * c.vocab_size * 4))
    return false;
  if (rank && (!zeroed(w.low, (size_t)R * w.low_ld * 4) || (bf16 && !zeroed(w.low16, (size_t)R * w.low16_ld * 2)) ||
               !zeroed(w.decay, (size_t)R * w.decay_ld * 4) || !zeroed(w.o, (size_t)R * o * 4)))
    return false;
  for (uint32_t l = 0; l < c.num_layers; ++l) {
    const MixerSpec &m = c.layers[l].mixer;
    HybridLayerBuffers &b = hybrid_[l];
    if (m.kind == MixerKind::GENERAL_DELTA) {
      if (!zeroed(b.state, B * greta_cuda_delta_state_bytes(m.heads, m.dim))) return false;
      continue;
    }
    // kept rows, then a ring that holds the window in front of a portion and the portion itself
    const size_t keep = std::min<size_t>(m.keep_first, max_seq_), rest = std::max<size_t>(1, max_seq_ - keep);
    b.ring = (uint32_t)(m.window ? std::min(rest, (size_t)m.window - 1 + chunk) : rest);
    const size_t rows = (size_t)B * m.kv_heads * (keep + b.ring);
    const GretaDataType ct = bf16 ? GretaDataType::FP16 : GretaDataType::FP32;
    if (!zeroed(b.k_cache, rows * up(m.dim, 8) * cb, ct) || !zeroed(b.v_cache, rows * up(m.vdim, 8) * cb, ct)) return false;
    if (m.taps && !zeroed(b.history, (size_t)B * m.taps * m.proj_cols() * 4)) return false;
  }
  GRETA_TRY(greta_cuda_device_synchronize(), "allocate_activations");
  invalidate_graph();
  return true;
}

bool BlockScheduler::hybrid_embed(const int32_t *d_tokens, const greta_rows &rows, std::string *err) {
  const ModelConfig &c = config_;
  GRETA_TRY(greta_cuda_embedding_positions(H(stream_), d_tokens, token_embd_.data(), pos_embd_.data(),
                                           c.weight_type == GretaDataType::BF16 ? GRETA_FMT_BF16 : GRETA_FMT_F32, static_cast<float *>(activations_.x.data()),
                                           rows.M, c.dim, c.vocab_size, c.max_seq_len, rows.d_pos, rows.pos0),
            "embedding");
  return true;
}

bool BlockScheduler::hybrid_layer(size_t layer, const greta_rows &rows, std::string *err) {
  const ModelConfig &c = config_;
  const LayerSpec &spec = c.layers[layer];
  const MixerSpec &m = spec.mixer;
  HybridLayerBuffers &b = hybrid_[layer];
  HybridActivations &w = hact_;
  cudaStream_t s = H(stream_);
  const bool bf16 = c.weight_type == GretaDataType::BF16, few = rows.M <= (bf16 ? FEW_ROWS_BF16 : FEW_ROWS), decode = rows.d_pos != nullptr;
  const bool delta = m.kind == MixerKind::GENERAL_DELTA;
  const int fmt = bf16 ? GRETA_FMT_BF16 : GRETA_FMT_F32;
  const uint32_t D = c.dim, HD = m.heads * m.dim;
  float *x = static_cast<float *>(activations_.x.data()), *proj = static_cast<float *>(w.proj.data()), *low = static_cast<float *>(w.low.data());
  const bool cat_bf16 = bf16 && !few, low_pair = cat_bf16 && !decode;
  void *cat = cat_bf16 ? w.cat16.data() : w.cat.data();
  const int cat_fmt = cat_bf16 ? GRETA_OUT_BF16 : GRETA_OUT_F32;

  // 1. norm and input projections
  greta_linear in{};
  in.fmt = fmt;
  in.w = b.w_in.data();
  in.N = b.in_rows;
  in.K = D;
  in.ldw = b.in_ld;
  uint32_t row = 0;
  auto segment = [&](greta_linear &l, uint32_t n, int act, const float *bias, void *out, uint32_t ld, uint32_t col, int out_fmt, uint32_t pair, int add) {
    l.seg[l.n_segments++] = greta_out_segment{row, n, act, out_fmt, add, bias, out, ld, col, pair};
    row += n;
  };
  if (delta) {
    segment(in, 3 * HD, GRETA_ACT_NONE, nullptr, proj, w.proj_ld, 0, GRETA_OUT_F32, 0, 0);
    segment(in, HD, GRETA_ACT_SIGMOID, nullptr, proj, w.proj_ld, 3 * HD, GRETA_OUT_F32, 0, 0);
    segment(in, HD, GRETA_ACT_SIGMOID, fp(b.a_bias), proj, w.proj_ld, 4 * HD, GRETA_OUT_F32, 0, 0);
    if (low_pair)
      segment(in, m.rank, GRETA_ACT_TANH, nullptr, w.low16.data(), w.low16_ld, 0, GRETA_OUT_BF16_PAIR, up(m.rank, 8), 0);
    else
      segment(in, m.rank, GRETA_ACT_TANH, nullptr, low, w.low_ld, 0, GRETA_OUT_F32, 0, 0);
  } else {
    segment(in, m.proj_cols(), GRETA_ACT_NONE, nullptr, proj, w.proj_ld, 0, GRETA_OUT_F32, 0, 0);
  }
  if (spec.ff) segment(in, spec.ff, GRETA_ACT_GELU_ERF, nullptr, cat, w.cat_ld, b.ff_col, cat_fmt, 0, 0);
  if (few) {
    GRETA_TRY(greta_cuda_linear_gemv(s, &in, x, D, fp(b.norm_w), fp(b.norm_b), c.rms_eps, rows.M), "input projections");
  } else {
    GRETA_TRY(greta_cuda_layer_norm(s, x, fp(b.norm_w), fp(b.norm_b), c.rms_eps, w.h.data(), bf16 ? GRETA_OUT_BF16 : GRETA_OUT_F32, rows.M, D, w.h_ld),
              "layer norm");
    GRETA_TRY(greta_cuda_linear_gemm(s, &in, w.h.data(), w.h_ld, rows.M), "input projections");
  }

  // 2. the mixer's core -> columns 0 .. out_cols of cat
  if (delta) {
    greta_delta_rule d{};
    d.heads = m.heads;
    d.dim = m.dim;
    d.rank = m.rank;
    d.ld = w.proj_ld;
    d.eps = c.rms_eps;
    d.r = proj;
    d.k = proj + HD;
    d.v = proj + 2 * HD;
    d.gate = proj + 3 * HD;
    d.a = proj + 4 * HD;
    d.decay = fp(w.decay);
    d.ld_decay = w.decay_ld;
    d.t = low;
    d.ld_t = w.low_ld;
    d.w2 = fp(b.w2);
    d.w0 = fp(b.w0);
    d.norm = fp(b.out_norm);
    d.state = static_cast<float *>(b.state.data());
    if (decode) {
      GRETA_TRY(greta_cuda_delta_step(s, &d, &rows, cat, cat_fmt, w.cat_ld), "delta step");
    } else {
      greta_linear dec{};
      dec.fmt = fmt;
      dec.w = b.w2_packed.data();
      dec.N = HD;
      dec.K = low_pair ? 2 * up(m.rank, 8) : m.rank;
      dec.ldw = b.w2_ld;
      row = 0;
      segment(dec, HD, GRETA_ACT_DELTA_DECAY, fp(b.w0), w.decay.data(), w.decay_ld, 0, GRETA_OUT_F32, 0, 0);
      if (few)
        GRETA_TRY(greta_cuda_linear_gemv(s, &dec, low, w.low_ld, nullptr, nullptr, 0.f, rows.M), "decay");
      else
        GRETA_TRY(greta_cuda_linear_gemm(s, &dec, low_pair ? w.low16.data() : w.low.data(), low_pair ? w.low16_ld : w.low_ld, rows.M), "decay");
      GRETA_TRY(greta_cuda_delta_scan(s, &d, &rows, static_cast<float *>(w.o.data())), "delta scan");
      GRETA_TRY(greta_cuda_delta_output(s, &d, fp(w.o), rows.M, cat, cat_fmt, w.cat_ld), "delta output");
    }
  } else {
    greta_window_attn a{};
    a.heads = m.heads;
    a.kv_heads = m.kv_heads;
    a.dim = m.dim;
    a.vdim = m.vdim;
    a.taps = m.taps;
    a.window = m.window;
    a.keep_first = (uint32_t)std::min<size_t>(m.keep_first, max_seq_);
    a.ring = b.ring;
    a.scale = m.scale;
    a.softcap = m.softcap;
    a.eps = c.rms_eps;
    a.temp = fp(b.temp);
    a.r1 = fp(b.r1);
    a.r2 = fp(b.r2);
    a.sink = fp(b.sink);
    a.conv = fp(b.conv);
    a.proj = proj;
    a.ld_proj = w.proj_ld;
    a.cache_fmt = bf16 ? GRETA_FMT_F16 : GRETA_FMT_F32;
    a.k_cache = b.k_cache.data();
    a.v_cache = b.v_cache.data();
    a.history = static_cast<float *>(b.history.data());
    if (decode) {
      GRETA_TRY(greta_cuda_window_attn(s, &a, &rows, nullptr, cat, cat_fmt, w.cat_ld, (uint32_t)max_seq_), "attention");
    } else {
      float *q = static_cast<float *>(w.q.data());
      GRETA_TRY(greta_cuda_window_attn_prepare(s, &a, &rows, q), "attention inputs");
      if (bf16 && rows.M >= MMA_MIN_ROWS)
        GRETA_TRY(greta_cuda_window_attn_prefill(s, &a, &rows, q, cat, cat_fmt, w.cat_ld), "attention");
      else
        GRETA_TRY(greta_cuda_window_attn(s, &a, &rows, q, cat, cat_fmt, w.cat_ld, rows.pos0 + rows.M), "attention");
    }
  }

  // 3. output projections of both sublayers, added to the residual stream
  greta_linear out{};
  out.fmt = fmt;
  out.w = b.w_out.data();
  out.N = D;
  out.K = b.out_cols;
  out.ldw = b.out_ld;
  row = 0;
  segment(out, D, GRETA_ACT_NONE, nullptr, x, D, 0, GRETA_OUT_F32, 0, 1);
  if (few)
    GRETA_TRY(greta_cuda_linear_gemv(s, &out, static_cast<const float *>(cat), w.cat_ld, nullptr, nullptr, 0.f, rows.M), "output projections");
  else
    GRETA_TRY(greta_cuda_linear_gemm(s, &out, cat, w.cat_ld, rows.M), "output projections");
  return true;
}

// Final norm + LM head for n rows (at most the activations' rows) -> logits [n][vocab].
bool BlockScheduler::hybrid_logits(const float *x, uint32_t n, float *logits, std::string *err) {
  const ModelConfig &c = config_;
  cudaStream_t s = H(stream_);
  const bool bf16 = c.weight_type == GretaDataType::BF16;
  greta_linear head{};
  head.fmt = bf16 ? GRETA_FMT_BF16 : GRETA_FMT_F32;
  head.w = output_weight_.data();
  head.N = c.vocab_size;
  head.K = c.dim;
  head.ldw = head_ld_;
  head.n_segments = 1;
  head.seg[0] = greta_out_segment{0, c.vocab_size, GRETA_ACT_NONE, GRETA_OUT_F32, 0, nullptr, logits, c.vocab_size, 0, 0};
  if (n <= (bf16 ? FEW_ROWS_BF16 : FEW_ROWS)) {
    GRETA_TRY(greta_cuda_linear_gemv(s, &head, x, c.dim, fp(output_norm_), fp(final_norm_b_), c.rms_eps, n), "lm head");
    return true;
  }
  // the hidden rows' own layer-norm buffer is free here; it holds at least the 64 rows a caller may ask for at once
  GRETA_TRY(greta_cuda_layer_norm(s, x, fp(output_norm_), fp(final_norm_b_), c.rms_eps, hact_.h.data(), bf16 ? GRETA_OUT_BF16 : GRETA_OUT_F32, n, c.dim,
                                  hact_.h_ld),
            "final norm");
  GRETA_TRY(greta_cuda_linear_gemm(s, &head, hact_.h.data(), hact_.h_ld, n), "lm head");
  return true;
}

bool BlockScheduler::hybrid_run(const int32_t *tokens, size_t seq_start, size_t seq_len, const std::function<bool(size_t, size_t)> &after,
                                std::string *err) {
  ActivationBuffers &a = activations_;
  cudaStream_t s = H(stream_);
  const size_t chunk = std::min<size_t>(config_.prefill_chunk, max_seq_);
  if (hybrid_.empty() || !hybrid_[0].w_in.data()) return fail(err, "forward: load weights first");
  for (size_t first = 0; first < seq_len; first += chunk) {
    const size_t n = std::min(chunk, seq_len - first);
    greta_rows rows{(uint32_t)n, cur_seq_, (uint32_t)(seq_start + first), nullptr};
    GRETA_TRY(greta_cuda_memcpy_h2d(a.tokens.data(), tokens + first, n * 4, s), "token upload");
    if (n == 1) {  // a single token takes the decode form
      GRETA_TRY(greta_cuda_memcpy_h2d(a.d_pos.data(), &rows.pos0, 4, s), "position upload");
      GRETA_TRY(greta_cuda_stream_synchronize(s), "position upload");  // it lives on this stack frame
      rows.d_pos = static_cast<const uint32_t *>(a.d_pos.data());
    }
    if (!hybrid_embed(static_cast<const int32_t *>(a.tokens.data()), rows, err)) return false;
    for (size_t l = 0; l < hybrid_.size(); ++l)
      if (!hybrid_layer(l, rows, err)) return false;
    if (!after(first, n)) return false;
  }
  return true;
}

}  // namespace gcore::inference
