// BlockScheduler, hybrid designs: layers with attention or recurrent mixers and feed-forwards over unquantised weights.
//
// A mixer is two matrix products around its core:
//   1. norm -> every input projection (w_in), activations in the epilogue
//   2. the core: windowed or latent attention over the cache, or a delta rule over the state
//   3. its columns -> output projection, added to the residual (w_out)
// Parallel layers, x += mixer(N(x)) + ff(N(x)), have the feed-forward in the same two products (its columns stand behind the mixer's);
// sequential ones, x += mixer(N1(x)); x += ff(N2(x)), have two more.
// For a single row (decode; up to 8 in fp32) the products are GEMVs with the norm fused in.  More rows run on the tensor cores (bf16)
// behind one norm kernel.  The residual stream, the projections that enter a mixer, scores, states and norms are fp32 in either mode.
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
constexpr uint32_t MMA_MIN_ROWS = 16;  // portions from which attention runs on the tensor cores (latent attention: in its expanded form)

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

uint16_t f32_to_f16(float f) {  // round to nearest even; too large saturates
  uint32_t x;
  std::memcpy(&x, &f, 4);
  const uint16_t sign = (uint16_t)((x >> 16) & 0x8000u);
  const float a = std::fabs(f);
  if (!(a < 65520.f)) return (uint16_t)(sign | (a != a ? 0x7E00u : 0x7BFFu));
  if (a < 6.103515625e-05f) return (uint16_t)(sign | (uint16_t)std::lrintf(a * 16777216.f));  // subnormal: units of 2^-24
  x &= 0x7FFFFFFFu;
  return (uint16_t)(sign | ((x - 0x38000000u + 0xFFFu + ((x >> 13) & 1u)) >> 13));
}

// A weight packed on the host: [rows][ld] in bf16, fp16 or fp32, zero where nothing is put.
struct Packed {
  GretaDataType type;
  uint32_t rows, ld;
  std::vector<uint16_t> h;
  std::vector<float> f;
  Packed(GretaDataType t, uint32_t r, uint32_t l) : type(t), rows(r), ld(l) {
    if (t != GretaDataType::FP32) h.assign((size_t)r * l, 0);
    else f.assign((size_t)r * l, 0.f);
  }
  Packed(bool bf16, uint32_t r, uint32_t l) : Packed(bf16 ? GretaDataType::BF16 : GretaDataType::FP32, r, l) {}
  void put(const std::vector<float> &src, uint32_t r, uint32_t cols, uint32_t row0, uint32_t col0) {
#pragma omp parallel for schedule(static)
    for (uint32_t i = 0; i < r; ++i)
      for (uint32_t j = 0; j < cols; ++j) {
        const size_t at = (size_t)(row0 + i) * ld + col0 + j;
        if (type == GretaDataType::BF16) h[at] = f32_to_bf16(src[(size_t)i * cols + j]);
        else if (type == GretaDataType::FP16) h[at] = f32_to_f16(src[(size_t)i * cols + j]);
        else f[at] = src[(size_t)i * cols + j];
      }
  }
  bool upload(Buffer &b, std::string *err) const {
    const bool wide = type == GretaDataType::FP32;
    const size_t bytes = (size_t)rows * ld * (wide ? 4 : 2);
    return b.allocate(bytes, BufferUsage::DeviceOnly, type, err) && b.copy_to_device(wide ? (const void *)f.data() : (const void *)h.data(), bytes, err);
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
    if (ends("norm") || ends("norm1") || ends("norm2") || ends(".temp")) mean = 1.f;
    if (ends(".r1")) mean = 0.5f;
    if (ends(".r2")) mean = 1.f;
    out->resize(n);
    synth::normal_f32(seed, stream, sigma, out->data(), 0, n);
    if (mean != 0.f)
      for (float &v : *out) v = std::fabs(v + mean);
    if (ends(".dt_bias") || ends(".A_log"))
      for (float &v : *out) v = 10.f * v - 2.f;  // decays from slow to quick
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
    if (m.kind == MixerKind::GATED_DELTA && (!m.rank || !m.gate_rank || m.rank + m.gate_rank > 8192))
      return fail(err, "init: gated delta needs low-rank widths that add up to 2..8192");
    if (m.kind == MixerKind::LATENT_ATTENTION && (!m.kv_rank || m.kv_rank > 1024 || !m.rot_dim || m.rot_dim > 128))
      return fail(err, "init: latent attention needs a latent of 1..1024 and a rotated part of 1..128");
  }
  rotations_.clear();
  for (const LayerSpec &l : c.layers)
    if (l.mixer.kind == MixerKind::LATENT_ATTENTION && std::find(rotations_.begin(), rotations_.end(), l.mixer.rotary) == rotations_.end())
      rotations_.push_back(l.mixer.rotary);
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
    const uint32_t HD = m.heads * m.dim, HV = m.out_cols(), GD = m.kv_heads * m.dim, GV = m.kv_heads * m.vdim, low = m.rank + m.gate_rank;
    const uint32_t ff_in = s.parallel ? s.ff : 0;
    uint32_t mix_rows = m.proj_cols();
    if (m.kind == MixerKind::LATENT_ATTENTION) mix_rows = (m.q_rank ? m.q_rank : m.q_cols()) + m.kv_rank + m.rot_dim + (m.gate ? HV : 0);
    if (m.kind == MixerKind::GATED_DELTA) mix_rows = m.conv_cols() + m.heads;
    if (!vec(pre + "norm1", D, b.norm_w) || (!c.rms_norms && !vec(pre + "norm1.b", D, b.norm_b))) return false;
    b.in_rows = mix_rows + low + ff_in;
    b.in_ld = up(D, 64);
    b.ff_col = up(HV, 64);
    b.out_cols = ff_in ? b.ff_col + s.ff : HV;
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
    auto convolution = [&](const std::initializer_list<std::pair<const char *, uint32_t>> &parts) {  // taps of q, k and v below one another
      std::vector<float> all;
      for (const auto &p : parts) {
        if (!src.values(mix + p.first + ".conv", {p.second, m.taps}, &v, err)) return false;
        all.insert(all.end(), v.begin(), v.end());
      }
      return upload_f32(b.conv, all, err);
    };
    if (m.kind == MixerKind::GENERAL_DELTA) {
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
    } else if (m.kind == MixerKind::LATENT_ATTENTION) {
      const uint32_t d8 = up(m.dim, 8), v8 = up(m.vdim, 8);
      if (m.q_rank) {
        b.uq_ld = up(m.q_rank, 64);
        Packed uq(bf16, m.q_cols(), b.uq_ld);
        if (!rows(mix + "dq", m.q_rank) || !vec(mix + "dq.norm", m.q_rank, b.q_norm) || !src.values(mix + "uq", {m.q_cols(), m.q_rank}, &v, err)) return false;
        uq.put(v, m.q_cols(), m.q_rank, 0, 0);
        if (!uq.upload(b.w_uq, err)) return false;
        weight_bytes_ += b.w_uq.size();
      } else if (!rows(mix + "q", m.q_cols())) {
        return false;
      }
      if (!rows(mix + "dkv", m.kv_rank + m.rot_dim) || !vec(mix + "dkv.norm", m.kv_rank, b.kv_norm)) return false;
      if (m.gate && !rows(mix + "g", HV)) return false;
      if (m.sink && !vec(mix + "sink", m.heads, b.sink)) return false;
      // Keys' and values' up-projections meet the fp16 cache, so a bf16 model holds them in fp16 (eight of its eleven bits suffice).
      b.kv_ld = up(m.kv_rank, 64);
      Packed kv(bf16 ? GretaDataType::FP16 : GretaDataType::FP32, m.heads * (d8 + v8), b.kv_ld);
      std::vector<float> head;
      const std::pair<const char *, uint32_t> parts[2] = {{"uk", m.dim}, {"uv", m.vdim}};
      for (int p = 0; p < 2; ++p) {
        const uint32_t n = parts[p].second;
        if (!src.values(mix + parts[p].first, {m.heads * n, m.kv_rank}, &v, err)) return false;
        for (uint32_t h = 0; h < m.heads; ++h) {
          head.assign(v.begin() + (size_t)h * n * m.kv_rank, v.begin() + (size_t)(h + 1) * n * m.kv_rank);
          kv.put(head, n, m.kv_rank, p ? m.heads * d8 + h * v8 : h * d8, 0);
        }
      }
      if (!kv.upload(b.w_kv, err)) return false;
      weight_bytes_ += b.w_kv.size();
      b.rotation = std::find(rotations_.begin(), rotations_.end(), m.rotary) - rotations_.begin();
    } else if (m.kind == MixerKind::GATED_DELTA) {
      if (!rows(mix + "q", GD) || !rows(mix + "k", GD) || !rows(mix + "v", HV) || !rows(mix + "b", m.heads) || !rows(mix + "a1", m.rank) ||
          !rows(mix + "g1", m.gate_rank) || !convolution({{"q", GD}, {"k", GD}, {"v", HV}}) || !vec(mix + "dt_bias", HD, b.w0) ||
          !vec(mix + "norm", m.vdim, b.out_norm))
        return false;
      if (!src.values(mix + "A_log", {m.heads}, &v, err)) return false;
      std::vector<float> rate(HD);
      for (uint32_t i = 0; i < HD; ++i) rate[i] = std::exp(v[i / m.dim]);
      if (!upload_f32(b.rate, rate, err)) return false;
      // Portions take both low-rank paths in one product, [decay | gate] columns; in bf16 the activations of either travel as a pair
      // (hi, lo), so each weight stands there twice.
      const uint32_t a8 = up(m.rank, 8), g8 = up(m.gate_rank, 8), g_col = bf16 ? 2 * a8 : up(m.rank, 4);
      b.w2_ld = up(bf16 ? 2 * a8 + 2 * g8 : g_col + m.gate_rank, 64);
      Packed w2(bf16, HD + HV, b.w2_ld);
      if (!src.values(mix + "a2", {HD, m.rank}, &v, err) || !upload_f32(b.w2, v, err)) return false;
      w2.put(v, HD, m.rank, 0, 0);
      if (bf16) w2.put(v, HD, m.rank, 0, a8);
      if (!src.values(mix + "g2", {HV, m.gate_rank}, &v, err) || !upload_f32(b.g2, v, err)) return false;
      w2.put(v, HV, m.gate_rank, HD, g_col);
      if (bf16) w2.put(v, HV, m.gate_rank, HD, g_col + g8);
      if (!w2.upload(b.w2_packed, err)) return false;
      weight_bytes_ += b.w2.size() + b.g2.size();
    } else {
      if (!rows(mix + "q", HD) || !rows(mix + "k", GD) || !rows(mix + "v", GV)) return false;
      if (m.temp && !vec(mix + "temp", m.heads, b.temp)) return false;
      if (m.distance_bias && (!vec(mix + "r1", m.heads, b.r1) || !vec(mix + "r2", m.heads, b.r2))) return false;
      if (m.sink && !vec(mix + "sink", m.heads, b.sink)) return false;
      if (m.taps && !convolution({{"q", HD}, {"k", GD}, {"v", GV}})) return false;
    }
    if (ff_in && (!rows(pre + "mlp.up", s.ff) || !cols(pre + "mlp.down", s.ff, b.ff_col))) return false;
    if (s.ff && !s.parallel) {
      b.up_ld = up(D, 64);
      b.down_ld = up(s.ff, 64);
      Packed w_up(bf16, s.ff, b.up_ld), w_down(bf16, D, b.down_ld);
      if (!vec(pre + "norm2", D, b.norm2_w) || !src.values(pre + "mlp.up", {s.ff, D}, &v, err)) return false;
      w_up.put(v, s.ff, D, 0, 0);
      if (!src.values(pre + "mlp.down", {D, s.ff}, &v, err)) return false;
      w_down.put(v, D, s.ff, 0, 0);
      if (!w_up.upload(b.w_up, err) || !w_down.upload(b.w_down, err)) return false;
      weight_bytes_ += b.w_up.size() + b.w_down.size();
    }
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
  if (c.tied_head ? !table("embed", c.vocab_size, head_ld_, output_weight_)
                  : !table("embed", c.vocab_size, D, token_embd_) || !table("head", c.vocab_size, head_ld_, output_weight_))
    return false;
  if (c.learned_positions && !table("pos", c.max_seq_len, D, pos_embd_)) return false;
  if (!vec("final.norm", D, output_norm_) || (!c.rms_norms && !vec("final.norm.b", D, final_norm_b_))) return false;
  weight_bytes_ += output_weight_.size();
  GRETA_TRY(greta_cuda_device_synchronize(), "load_weights");
  return true;
}

bool BlockScheduler::allocate_hybrid_activations(std::string *err) {
  const ModelConfig &c = config_;
  if (max_seq_ == 0 || max_seq_ > c.max_seq_len)
    return fail(err, "allocate_activations: max_seq_len must be 1.." + std::to_string(c.max_seq_len) + (c.learned_positions ? " (the model's learned positions)" : ""));
  const bool bf16 = c.weight_type == GretaDataType::BF16;
  const uint32_t chunk = (uint32_t)std::min<size_t>(c.prefill_chunk, max_seq_), B = batch_, R = std::max(chunk, B), D = c.dim, cb = bf16 ? 2 : 4;
  ActivationBuffers &a = activations_;
  HybridActivations &w = hact_;
  auto zeroed = [&](Buffer &b, size_t bytes, GretaDataType t = GretaDataType::FP32) {
    if (!b.allocate(std::max<size_t>(bytes, 16), BufferUsage::DeviceOnly, t, err)) return false;
    GRETA_TRY(greta_cuda_memset(b.data(), 0, b.size(), nullptr), "allocate_activations");
    return true;
  };
  uint32_t proj = 4, cat = 64, q = 4, o = 4, low = 0, low16 = 0, hd = 0, q_latent = 0, u = 0, gate = 0;
  size_t scratch = 0, qx = 0, kx = 0, vx = 0;
  const uint32_t absorbed = bf16 ? std::max(B, std::min(chunk, MMA_MIN_ROWS - 1)) : R;  // rows that latent attention takes in its absorbed form
  for (uint32_t l = 0; l < c.num_layers; ++l) {
    const MixerSpec &m = c.layers[l].mixer;
    const uint32_t ff = c.layers[l].ff, ff_col = up(m.out_cols(), 64), HD = m.heads * m.dim;
    proj = std::max(proj, up(m.proj_cols(), 4));
    cat = std::max({cat, ff_col, c.layers[l].parallel && ff ? ff_col + up(ff, 64) : up(ff, 64)});
    switch (m.kind) {
      case MixerKind::GENERAL_DELTA:
        o = std::max(o, HD);
        low = std::max(low, m.rank);
        low16 = std::max(low16, 2 * up(m.rank, 8));
        hd = std::max(hd, HD);
        break;
      case MixerKind::GATED_DELTA:
        o = std::max(o, m.out_cols());
        low = std::max(low, up(m.rank, 4) + m.gate_rank);
        low16 = std::max(low16, 2 * up(m.rank, 8) + 2 * up(m.gate_rank, 8));
        hd = std::max(hd, HD);
        u = std::max(u, up(m.conv_cols(), 4));
        gate = std::max(gate, up(m.out_cols(), 4));
        break;
      case MixerKind::LATENT_ATTENTION: {
        q = std::max(q, m.q_cols());
        q_latent = std::max(q_latent, up(m.q_rank, 64));
        greta_latent_attn a{};
        a.heads = m.heads, a.rank = m.kv_rank, a.rot_dim = m.rot_dim, a.fmt = bf16 ? GRETA_FMT_F16 : GRETA_FMT_F32;
        scratch = std::max(scratch, greta_cuda_latent_scratch_bytes(&a, absorbed, (uint32_t)max_seq_));
        if (bf16 && chunk >= MMA_MIN_ROWS) {
          qx = std::max(qx, (size_t)R * greta_cuda_latent_query_row(m.heads, m.dim, m.rot_dim) * 2);
          kx = std::max(kx, max_seq_ * m.heads * up(m.dim, 8) * 2);
          vx = std::max(vx, max_seq_ * m.heads * up(m.vdim, 8) * 2);
        }
        break;
      }
      default: q = std::max(q, m.heads * up(m.dim, 8));
    }
  }
  w.h_ld = up(D, 64);
  w.proj_ld = proj;
  w.cat_ld = cat;
  w.low_ld = up(low, 64);
  w.low16_ld = up(low16, 64);
  w.decay_ld = up(hd, 4);
  w.q_latent_ld = q_latent;
  w.u_ld = u;
  w.gate_ld = gate;
  if (!zeroed(a.x, (size_t)R * D * 4) || !zeroed(a.tokens, (size_t)R * 4) || !zeroed(a.d_pos, 2 * (size_t)B * 4) || !zeroed(a.d_next, (size_t)B * 4) ||
      !zeroed(a.out_tokens, (size_t)B * max_seq_ * 4) || !zeroed(logits_, (size_t)B * c.vocab_size * 4))
    return false;
  const size_t few = bf16 ? std::min(R, FEW_ROWS_BF16) : R;
  if (!zeroed(w.h, (size_t)R * w.h_ld * cb) || !zeroed(w.proj, (size_t)R * proj * 4) || !zeroed(w.cat, few * cat * 4) ||
      (bf16 && !zeroed(w.cat16, (size_t)R * cat * 2)) || !zeroed(w.q, (size_t)R * q * 4) || !zeroed(w.x_rows, (size_t)64 * D * 4) ||
      !zeroed(w.logits_rows, (size_t)64 * c.vocab_size * 4))
    return false;
  if (low && (!zeroed(w.low, (size_t)R * w.low_ld * 4) || (bf16 && !zeroed(w.low16, (size_t)R * w.low16_ld * 2)) ||
              !zeroed(w.decay, (size_t)R * w.decay_ld * 4) || !zeroed(w.o, (size_t)R * o * 4)))
    return false;
  if ((u && (!zeroed(w.u, (size_t)R * u * 4) || !zeroed(w.gate, (size_t)R * gate * 4))) || (q_latent && !zeroed(w.q_latent, (size_t)R * q_latent * cb)) ||
      (scratch && !zeroed(w.latent_scratch, scratch)) || (kx && (!zeroed(w.q_tiles, qx, GretaDataType::FP16) || !zeroed(w.k_expanded, kx, GretaDataType::FP16) || !zeroed(w.v_expanded, vx, GretaDataType::FP16))))
    return false;
  rotation_tables_ = std::vector<Buffer>(rotations_.size());
  for (size_t r = 0; r < rotations_.size(); ++r) {  // angles in double: the tables are as exact as their fp32 entries
    double amp = 1.0;
    const std::vector<double> f = rotations_[r].frequencies(&amp);
    std::vector<float> t(max_seq_ * f.size() * 2);
#pragma omp parallel for schedule(static)
    for (size_t p = 0; p < max_seq_; ++p)
      for (size_t i = 0; i < f.size(); ++i) {
        t[(p * f.size() + i) * 2] = (float)(std::cos((double)p * f[i]) * amp);
        t[(p * f.size() + i) * 2 + 1] = (float)(std::sin((double)p * f[i]) * amp);
      }
    if (!upload_f32(rotation_tables_[r], t, err)) return false;
  }
  for (uint32_t l = 0; l < c.num_layers; ++l) {
    const MixerSpec &m = c.layers[l].mixer;
    HybridLayerBuffers &b = hybrid_[l];
    if (m.kind == MixerKind::GENERAL_DELTA) {
      if (!zeroed(b.state, B * greta_cuda_delta_state_bytes(m.heads, m.dim))) return false;
      continue;
    }
    if (m.kind == MixerKind::GATED_DELTA) {
      if (!zeroed(b.state, B * greta_cuda_gated_delta_state_bytes(m.heads, m.dim, m.vdim)) || !zeroed(b.history, (size_t)B * m.taps * m.conv_cols() * 4)) return false;
      continue;
    }
    if (m.kind == MixerKind::LATENT_ATTENTION) {
      if (!zeroed(b.k_cache, B * max_seq_ * greta_cuda_latent_row(m.kv_rank, m.rot_dim) * cb, bf16 ? GretaDataType::FP16 : GretaDataType::FP32)) return false;
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
  const int fmt = c.weight_type == GretaDataType::BF16 ? GRETA_FMT_BF16 : GRETA_FMT_F32;
  float *x = static_cast<float *>(activations_.x.data());
  if (c.learned_positions) {
    GRETA_TRY(greta_cuda_embedding_positions(H(stream_), d_tokens, token_embd_.data(), pos_embd_.data(), fmt, x, rows.M, c.dim, c.vocab_size, c.max_seq_len,
                                             rows.d_pos, rows.pos0),
              "embedding");
    return true;
  }
  GRETA_TRY(greta_cuda_embedding_scaled(H(stream_), d_tokens, c.tied_head ? output_weight_.data() : token_embd_.data(), fmt, c.tied_head ? head_ld_ : c.dim,
                                        c.embed_scale, x, rows.M, c.dim, c.vocab_size),
            "embedding");
  return true;
}

namespace {
// Adds an output segment behind the ones a linear has.
greta_out_segment &segment(greta_linear &l, uint32_t n, int act, const float *bias, void *out, uint32_t ld, uint32_t col, int out_fmt) {
  uint32_t row = l.n_segments ? l.seg[l.n_segments - 1].row0 + l.seg[l.n_segments - 1].rows : 0;
  greta_out_segment &g = l.seg[l.n_segments++];
  g = greta_out_segment{};
  g.row0 = row, g.rows = n, g.act = act, g.bias = bias, g.out = out, g.ld = ld, g.col0 = col, g.out_fmt = out_fmt;
  return g;
}
greta_linear linear(int fmt, const Buffer &w, uint32_t N, uint32_t K, uint32_t ld) {
  greta_linear l{};
  l.fmt = fmt, l.w = w.data(), l.N = N, l.K = K, l.ldw = ld;
  return l;
}
}  // namespace

bool BlockScheduler::few_rows(const greta_rows &rows) const { return rows.M <= (config_.weight_type == GretaDataType::BF16 ? FEW_ROWS_BF16 : FEW_ROWS); }

void *BlockScheduler::cat_buffer(const greta_rows &rows, int *fmt) {
  const bool half = config_.weight_type == GretaDataType::BF16 && !few_rows(rows);
  *fmt = half ? GRETA_OUT_BF16 : GRETA_OUT_F32;
  return half ? hact_.cat16.data() : hact_.cat.data();
}

bool BlockScheduler::x_norm_linear(greta_linear &lin, const Buffer &norm_w, const Buffer &norm_b, const greta_rows &rows, std::string *err) {
  const ModelConfig &c = config_;
  cudaStream_t s = H(stream_);
  const float *x = static_cast<const float *>(activations_.x.data());
  const int out_fmt = c.weight_type == GretaDataType::BF16 ? GRETA_OUT_BF16 : GRETA_OUT_F32;
  if (few_rows(rows)) {
    GRETA_TRY(greta_cuda_linear_gemv(s, &lin, x, c.dim, fp(norm_w), c.rms_norms ? nullptr : fp(norm_b), c.rms_eps, rows.M), "input projections");
    return true;
  }
  if (c.rms_norms)
    GRETA_TRY(greta_cuda_rms_norm(s, x, c.dim, fp(norm_w), c.rms_eps, hact_.h.data(), out_fmt, rows.M, c.dim, hact_.h_ld), "norm");
  else
    GRETA_TRY(greta_cuda_layer_norm(s, x, fp(norm_w), fp(norm_b), c.rms_eps, hact_.h.data(), out_fmt, rows.M, c.dim, hact_.h_ld), "layer norm");
  GRETA_TRY(greta_cuda_linear_gemm(s, &lin, hact_.h.data(), hact_.h_ld, rows.M), "input projections");
  return true;
}

bool BlockScheduler::from_cat(const Buffer &w, uint32_t cols, uint32_t ld, const greta_rows &rows, std::string *err) {
  const ModelConfig &c = config_;
  int cat_fmt;
  const void *cat = cat_buffer(rows, &cat_fmt);
  greta_linear out = linear(c.weight_type == GretaDataType::BF16 ? GRETA_FMT_BF16 : GRETA_FMT_F32, w, c.dim, cols, ld);
  segment(out, c.dim, GRETA_ACT_NONE, nullptr, activations_.x.data(), c.dim, 0, GRETA_OUT_F32).accumulate = 1;
  if (few_rows(rows))
    GRETA_TRY(greta_cuda_linear_gemv(H(stream_), &out, static_cast<const float *>(cat), hact_.cat_ld, nullptr, nullptr, 0.f, rows.M), "output projections");
  else
    GRETA_TRY(greta_cuda_linear_gemm(H(stream_), &out, cat, hact_.cat_ld, rows.M), "output projections");
  return true;
}

bool BlockScheduler::hybrid_layer(size_t layer, const greta_rows &rows, std::string *err) {
  const ModelConfig &c = config_;
  const LayerSpec &spec = c.layers[layer];
  const MixerSpec &m = spec.mixer;
  HybridLayerBuffers &b = hybrid_[layer];
  HybridActivations &w = hact_;
  const bool bf16 = c.weight_type == GretaDataType::BF16, low_pair = bf16 && !few_rows(rows) && !rows.d_pos;
  const int fmt = bf16 ? GRETA_FMT_BF16 : GRETA_FMT_F32;
  const uint32_t HD = m.heads * m.dim;
  float *proj = static_cast<float *>(w.proj.data());
  int cat_fmt;
  void *cat = cat_buffer(rows, &cat_fmt);

  // 1. norm and input projections
  greta_linear in = linear(fmt, b.w_in, b.in_rows, c.dim, b.in_ld);
  auto plain = [&](uint32_t n, uint32_t col, int act = GRETA_ACT_NONE, const float *bias = nullptr) {
    segment(in, n, act, bias, proj, w.proj_ld, col, GRETA_OUT_F32);
  };
  // activations of a low-rank path: fp32 at column col, or as a bf16 pair at column col16
  auto low = [&](uint32_t n, int act, uint32_t col, uint32_t col16) {
    if (low_pair)
      segment(in, n, act, nullptr, w.low16.data(), w.low16_ld, col16, GRETA_OUT_BF16_PAIR).pair_offset = up(n, 8);
    else
      segment(in, n, act, nullptr, w.low.data(), w.low_ld, col, GRETA_OUT_F32);
  };
  switch (m.kind) {
    case MixerKind::GENERAL_DELTA:
      plain(3 * HD, 0);
      plain(HD, 3 * HD, GRETA_ACT_SIGMOID);
      plain(HD, 4 * HD, GRETA_ACT_SIGMOID, fp(b.a_bias));
      low(m.rank, GRETA_ACT_TANH, 0, 0);
      break;
    case MixerKind::LATENT_ATTENTION:
      plain(m.q_rank ? m.q_rank : m.q_cols(), 0);
      plain(m.kv_rank + m.rot_dim, m.down_col());
      if (m.gate) plain(m.out_cols(), m.gate_col(), GRETA_ACT_SIGMOID);
      break;
    case MixerKind::GATED_DELTA:
      plain(m.conv_cols(), 0);
      plain(m.heads, MixerSpec::up4(m.conv_cols()), GRETA_ACT_SIGMOID);
      low(m.rank, GRETA_ACT_NONE, 0, 0);
      low(m.gate_rank, GRETA_ACT_NONE, up(m.rank, 4), 2 * up(m.rank, 8));
      break;
    default: plain(m.proj_cols(), 0);
  }
  if (spec.parallel && spec.ff) segment(in, spec.ff, spec.ff_act, nullptr, cat, w.cat_ld, b.ff_col, cat_fmt);
  if (!x_norm_linear(in, b.norm_w, b.norm_b, rows, err)) return false;

  // 2. the mixer's core -> columns 0 .. out_cols of cat
  switch (m.kind) {
    case MixerKind::GENERAL_DELTA:
      if (!general_delta_core(layer, rows, err)) return false;
      break;
    case MixerKind::LATENT_ATTENTION:
      if (!latent_attention_core(layer, rows, err)) return false;
      break;
    case MixerKind::GATED_DELTA:
      if (!gated_delta_core(layer, rows, err)) return false;
      break;
    default:
      if (!window_attention_core(layer, rows, err)) return false;
  }

  // 3. output projection (parallel layers: of both sublayers), added to the residual stream
  if (!from_cat(b.w_out, b.out_cols, b.out_ld, rows, err)) return false;

  // 4. a feed-forward that follows
  if (spec.parallel || !spec.ff) return true;
  greta_linear ff = linear(fmt, b.w_up, spec.ff, c.dim, b.up_ld);
  segment(ff, spec.ff, spec.ff_act, nullptr, cat, w.cat_ld, 0, cat_fmt);
  return x_norm_linear(ff, b.norm2_w, b.norm_b, rows, err) && from_cat(b.w_down, spec.ff, b.down_ld, rows, err);
}

bool BlockScheduler::general_delta_core(size_t layer, const greta_rows &rows, std::string *err) {
  const ModelConfig &c = config_;
  const MixerSpec &m = c.layers[layer].mixer;
  HybridLayerBuffers &b = hybrid_[layer];
  HybridActivations &w = hact_;
  cudaStream_t s = H(stream_);
  const bool bf16 = c.weight_type == GretaDataType::BF16, few = few_rows(rows), low_pair = bf16 && !few;
  const uint32_t HD = m.heads * m.dim;
  float *proj = static_cast<float *>(w.proj.data()), *low = static_cast<float *>(w.low.data());
  int cat_fmt;
  void *cat = cat_buffer(rows, &cat_fmt);
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
  if (rows.d_pos) {
    GRETA_TRY(greta_cuda_delta_step(s, &d, &rows, cat, cat_fmt, w.cat_ld), "delta step");
    return true;
  }
  greta_linear dec = linear(bf16 ? GRETA_FMT_BF16 : GRETA_FMT_F32, b.w2_packed, HD, low_pair ? 2 * up(m.rank, 8) : m.rank, b.w2_ld);
  segment(dec, HD, GRETA_ACT_DELTA_DECAY, fp(b.w0), w.decay.data(), w.decay_ld, 0, GRETA_OUT_F32);
  if (few)
    GRETA_TRY(greta_cuda_linear_gemv(s, &dec, low, w.low_ld, nullptr, nullptr, 0.f, rows.M), "decay");
  else
    GRETA_TRY(greta_cuda_linear_gemm(s, &dec, low_pair ? w.low16.data() : w.low.data(), low_pair ? w.low16_ld : w.low_ld, rows.M), "decay");
  GRETA_TRY(greta_cuda_delta_scan(s, &d, &rows, static_cast<float *>(w.o.data())), "delta scan");
  GRETA_TRY(greta_cuda_delta_output(s, &d, fp(w.o), rows.M, cat, cat_fmt, w.cat_ld), "delta output");
  return true;
}

bool BlockScheduler::window_attention_core(size_t layer, const greta_rows &rows, std::string *err) {
  const ModelConfig &c = config_;
  const MixerSpec &m = c.layers[layer].mixer;
  HybridLayerBuffers &b = hybrid_[layer];
  HybridActivations &w = hact_;
  cudaStream_t s = H(stream_);
  const bool bf16 = c.weight_type == GretaDataType::BF16;
  int cat_fmt;
  void *cat = cat_buffer(rows, &cat_fmt);
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
  a.proj = static_cast<float *>(w.proj.data());
  a.ld_proj = w.proj_ld;
  a.cache_fmt = bf16 ? GRETA_FMT_F16 : GRETA_FMT_F32;
  a.k_cache = b.k_cache.data();
  a.v_cache = b.v_cache.data();
  a.history = static_cast<float *>(b.history.data());
  if (rows.d_pos) {
    GRETA_TRY(greta_cuda_window_attn(s, &a, &rows, nullptr, cat, cat_fmt, w.cat_ld, (uint32_t)max_seq_), "attention");
    return true;
  }
  float *q = static_cast<float *>(w.q.data());
  GRETA_TRY(greta_cuda_window_attn_prepare(s, &a, &rows, q), "attention inputs");
  if (bf16 && rows.M >= MMA_MIN_ROWS)
    GRETA_TRY(greta_cuda_window_attn_prefill(s, &a, &rows, q, cat, cat_fmt, w.cat_ld), "attention");
  else
    GRETA_TRY(greta_cuda_window_attn(s, &a, &rows, q, cat, cat_fmt, w.cat_ld, rows.pos0 + rows.M), "attention");
  return true;
}

bool BlockScheduler::latent_attention_core(size_t layer, const greta_rows &rows, std::string *err) {
  const ModelConfig &c = config_;
  const MixerSpec &m = c.layers[layer].mixer;
  HybridLayerBuffers &b = hybrid_[layer];
  HybridActivations &w = hact_;
  cudaStream_t s = H(stream_);
  const bool bf16 = c.weight_type == GretaDataType::BF16, few = few_rows(rows);
  const float *proj = fp(w.proj);
  int cat_fmt;
  void *cat = cat_buffer(rows, &cat_fmt);
  greta_latent_attn a{};
  a.heads = m.heads;
  a.dim = m.dim;
  a.rot_dim = m.rot_dim;
  a.vdim = m.vdim;
  a.rank = m.kv_rank;
  a.rot_dims = m.rotary.dims;
  a.interleaved = m.rotary.interleaved;
  a.cap = a.positions = (uint32_t)max_seq_;
  a.scale = m.scale;
  a.eps = c.rms_eps;
  a.rotation = fp(rotation_tables_[b.rotation]);
  a.sink = fp(b.sink);
  a.latent_norm = fp(b.kv_norm);
  a.q = proj;
  a.ld_q = a.ld_down = a.ld_gate = w.proj_ld;
  a.down = proj + m.down_col();
  a.gate = m.gate ? proj + m.gate_col() : nullptr;
  a.fmt = bf16 ? GRETA_FMT_F16 : GRETA_FMT_F32;
  a.w_kv = b.w_kv.data();
  a.ld_w = b.kv_ld;
  a.cache = b.k_cache.data();
  if (m.q_rank) {  // queries through a normed latent
    greta_linear uq = linear(bf16 ? GRETA_FMT_BF16 : GRETA_FMT_F32, b.w_uq, m.q_cols(), m.q_rank, b.uq_ld);
    segment(uq, m.q_cols(), GRETA_ACT_NONE, nullptr, w.q.data(), m.q_cols(), 0, GRETA_OUT_F32);
    if (few) {
      GRETA_TRY(greta_cuda_linear_gemv(s, &uq, proj, w.proj_ld, fp(b.q_norm), nullptr, c.rms_eps, rows.M), "queries");
    } else {
      GRETA_TRY(greta_cuda_rms_norm(s, proj, w.proj_ld, fp(b.q_norm), c.rms_eps, w.q_latent.data(), bf16 ? GRETA_OUT_BF16 : GRETA_OUT_F32, rows.M, m.q_rank,
                                    w.q_latent_ld),
                "query norm");
      GRETA_TRY(greta_cuda_linear_gemm(s, &uq, w.q_latent.data(), w.q_latent_ld, rows.M), "queries");
    }
    a.q = fp(w.q);
    a.ld_q = m.q_cols();
  }
  if (!bf16 || rows.d_pos || rows.M < MMA_MIN_ROWS) {
    GRETA_TRY(greta_cuda_latent_absorbed(s, &a, &rows, w.latent_scratch.data(), cat, cat_fmt, w.cat_ld, rows.d_pos ? (uint32_t)max_seq_ : rows.pos0 + rows.M),
              "attention");
    return true;
  }
  // keys and values of every head for all positions so far, then attention over them
  GRETA_TRY(greta_cuda_latent_prepare(s, &a, &rows, w.q_tiles.data()), "attention inputs");
  const uint32_t Hd = m.heads * up(m.dim, 8), Hv = m.heads * up(m.vdim, 8), ld = greta_cuda_latent_row(m.kv_rank, m.rot_dim);
  greta_linear kv = linear(GRETA_FMT_F16, b.w_kv, Hd + Hv, m.kv_rank, b.kv_ld);
  segment(kv, Hd, GRETA_ACT_NONE, nullptr, w.k_expanded.data(), Hd, 0, GRETA_OUT_F16);
  segment(kv, Hv, GRETA_ACT_NONE, nullptr, w.v_expanded.data(), Hv, 0, GRETA_OUT_F16);
  const uint16_t *latents = static_cast<const uint16_t *>(b.k_cache.data()) + (size_t)rows.slot0 * a.cap * ld;
  GRETA_TRY(greta_cuda_linear_gemm(s, &kv, latents, ld, rows.pos0 + rows.M), "keys and values");
  GRETA_TRY(greta_cuda_latent_prefill(s, &a, &rows, w.q_tiles.data(), w.k_expanded.data(), w.v_expanded.data(), cat, cat_fmt, w.cat_ld), "attention");
  return true;
}

bool BlockScheduler::gated_delta_core(size_t layer, const greta_rows &rows, std::string *err) {
  const ModelConfig &c = config_;
  const MixerSpec &m = c.layers[layer].mixer;
  HybridLayerBuffers &b = hybrid_[layer];
  HybridActivations &w = hact_;
  cudaStream_t s = H(stream_);
  const bool bf16 = c.weight_type == GretaDataType::BF16, few = few_rows(rows), low_pair = bf16 && !few;
  const uint32_t HD = m.heads * m.dim, HV = m.out_cols();
  int cat_fmt;
  void *cat = cat_buffer(rows, &cat_fmt);
  greta_gated_delta d{};
  d.heads = m.heads;
  d.kv_heads = m.kv_heads;
  d.dim = m.dim;
  d.vdim = m.vdim;
  d.taps = m.taps;
  d.rank_a = m.rank;
  d.rank_g = m.gate_rank;
  d.eps = c.rms_eps;
  d.proj = fp(w.proj);
  d.ld_proj = d.ld_beta = w.proj_ld;
  d.conv = fp(b.conv);
  d.history = static_cast<float *>(b.history.data());
  d.beta = d.proj + MixerSpec::up4(m.conv_cols());
  d.norm = fp(b.out_norm);
  d.state = static_cast<float *>(b.state.data());
  d.low = fp(w.low);
  d.ld_low = w.low_ld;
  d.low_g = up(m.rank, 4);
  d.a2 = fp(b.w2);
  d.g2 = fp(b.g2);
  d.rate = fp(b.rate);
  d.dt_bias = fp(b.w0);
  d.u = static_cast<float *>(w.u.data());
  d.ld_u = w.u_ld;
  d.decay = fp(w.decay);
  d.ld_decay = w.decay_ld;
  d.gate = fp(w.gate);
  d.ld_gate = w.gate_ld;
  if (rows.d_pos) {
    GRETA_TRY(greta_cuda_gated_delta_step(s, &d, &rows, cat, cat_fmt, w.cat_ld), "delta step");
    return true;
  }
  const uint32_t K = low_pair ? 2 * up(m.rank, 8) + 2 * up(m.gate_rank, 8) : up(m.rank, 4) + m.gate_rank;
  greta_linear low2 = linear(bf16 ? GRETA_FMT_BF16 : GRETA_FMT_F32, b.w2_packed, HD + HV, K, b.w2_ld);
  segment(low2, HD, GRETA_ACT_SOFTPLUS_DECAY, fp(b.w0), w.decay.data(), w.decay_ld, 0, GRETA_OUT_F32).rate = fp(b.rate);
  segment(low2, HV, GRETA_ACT_SIGMOID, nullptr, w.gate.data(), w.gate_ld, 0, GRETA_OUT_F32);
  if (few)
    GRETA_TRY(greta_cuda_linear_gemv(s, &low2, d.low, w.low_ld, nullptr, nullptr, 0.f, rows.M), "decay and gate");
  else
    GRETA_TRY(greta_cuda_linear_gemm(s, &low2, low_pair ? w.low16.data() : w.low.data(), low_pair ? w.low16_ld : w.low_ld, rows.M), "decay and gate");
  GRETA_TRY(greta_cuda_gated_delta_prepare(s, &d, &rows), "delta inputs");
  GRETA_TRY(greta_cuda_gated_delta_scan(s, &d, &rows, static_cast<float *>(w.o.data())), "delta scan");
  GRETA_TRY(greta_cuda_gated_delta_output(s, &d, fp(w.o), rows.M, cat, cat_fmt, w.cat_ld), "delta output");
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
  segment(head, c.vocab_size, GRETA_ACT_NONE, nullptr, logits, c.vocab_size, 0, GRETA_OUT_F32);
  if (n <= (bf16 ? FEW_ROWS_BF16 : FEW_ROWS)) {
    GRETA_TRY(greta_cuda_linear_gemv(s, &head, x, c.dim, fp(output_norm_), c.rms_norms ? nullptr : fp(final_norm_b_), c.rms_eps, n), "lm head");
    return true;
  }
  // the hidden rows' own layer-norm buffer is free here; it holds at least the 64 rows a caller may ask for at once
  const int out_fmt = bf16 ? GRETA_OUT_BF16 : GRETA_OUT_F32;
  if (c.rms_norms)
    GRETA_TRY(greta_cuda_rms_norm(s, x, c.dim, fp(output_norm_), c.rms_eps, hact_.h.data(), out_fmt, n, c.dim, hact_.h_ld), "final norm");
  else
    GRETA_TRY(greta_cuda_layer_norm(s, x, fp(output_norm_), fp(final_norm_b_), c.rms_eps, hact_.h.data(), out_fmt, n, c.dim, hact_.h_ld), "final norm");
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
