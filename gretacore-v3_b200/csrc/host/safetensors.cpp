// Model folders: config.json + model.safetensors.
#include <fcntl.h>
#include <sys/mman.h>
#include <sys/stat.h>
#include <unistd.h>

#include <cstring>
#include <fstream>
#include <map>
#include <sstream>

#include "gcore/greta_b200.hpp"
#include "host_util.hpp"
#include "json.hpp"

namespace gcore::inference {

using gcore::host::fail;
using gcore::host::Json;
using gcore::rt::GretaDataType;

namespace {
size_t element_bytes(const std::string &dtype) { return dtype == "BF16" || dtype == "F16" ? 2 : dtype == "F32" || dtype == "I32" ? 4 : 0; }
}  // namespace

struct SafetensorsLoader::Impl {
  int fd = -1;
  const uint8_t *map = nullptr;
  size_t map_bytes = 0, data_offset = 0;
  std::vector<TensorInfo> tensors;
  std::map<std::string, size_t> by_name;
  ModelConfig config;

  ~Impl() { close_file(); }
  void close_file() {
    if (map) munmap(const_cast<uint8_t *>(map), map_bytes);
    if (fd >= 0) ::close(fd);
    map = nullptr;
    fd = -1;
  }
};

SafetensorsLoader::SafetensorsLoader() : impl_(new Impl) {}
SafetensorsLoader::~SafetensorsLoader() = default;

bool SafetensorsLoader::open(const std::string &dir, std::string *err) {
  Impl &im = *impl_;
  im.close_file();
  im.tensors.clear();
  im.by_name.clear();
  const std::string path = dir + "/model.safetensors";
  im.fd = ::open(path.c_str(), O_RDONLY);
  if (im.fd < 0) return fail(err, "safetensors: cannot open " + path);
  struct stat st;
  if (fstat(im.fd, &st) != 0 || st.st_size < 8) return fail(err, "safetensors: file too short");
  im.map_bytes = (size_t)st.st_size;
  void *m = mmap(nullptr, im.map_bytes, PROT_READ, MAP_PRIVATE, im.fd, 0);
  if (m == MAP_FAILED) return fail(err, "safetensors: mmap failed");
  im.map = static_cast<const uint8_t *>(m);
  uint64_t header = 0;
  std::memcpy(&header, im.map, 8);
  if (header > im.map_bytes - 8) return fail(err, "safetensors: the header reaches past the end of the file");
  im.data_offset = 8 + (size_t)header;
  Json j;
  if (!Json::parse(reinterpret_cast<const char *>(im.map) + 8, (size_t)header, &j, err)) return false;
  for (const auto &member : j.members) {
    if (member.first == "__metadata__") continue;
    const Json *dt = member.second.get("dtype"), *shape = member.second.get("shape"), *at = member.second.get("data_offsets");
    TensorInfo t;
    t.name = member.first;
    if (!dt || !shape || !at || at->items.size() != 2) return fail(err, "safetensors: malformed entry " + t.name);
    t.dtype = dt->string;
    size_t elems = 1;
    for (const Json &d : shape->items) {
      uint32_t n = 0;
      if (!d.as_u32(&n)) return fail(err, "safetensors: malformed shape of " + t.name);
      t.shape.push_back(n);
      elems *= n;
    }
    const double begin = at->items[0].number, end = at->items[1].number;
    if (begin < 0 || end < begin || end > (double)(im.map_bytes - im.data_offset)) return fail(err, "safetensors: " + t.name + " reaches past the end of the file");
    t.offset = (size_t)begin;
    t.size_bytes = (size_t)end - t.offset;
    if (element_bytes(t.dtype) && t.size_bytes != elems * element_bytes(t.dtype)) return fail(err, "safetensors: size of " + t.name + " does not match its shape");
    im.by_name[t.name] = im.tensors.size();
    im.tensors.push_back(std::move(t));
  }
  std::ifstream cf(dir + "/config.json");
  if (!cf) return fail(err, "cannot open " + dir + "/config.json");
  std::stringstream text;
  text << cf.rdbuf();
  return config_from_json(
      text.str(),
      [this](const std::string &name) {
        const TensorInfo *t = find(name);
        return t ? &t->shape : nullptr;
      },
      &im.config, err);
}

const TensorInfo *SafetensorsLoader::find(const std::string &name) const {
  auto it = impl_->by_name.find(name);
  return it == impl_->by_name.end() ? nullptr : &impl_->tensors[it->second];
}
std::vector<TensorInfo> SafetensorsLoader::list_tensors() const { return impl_->tensors; }
ModelConfig SafetensorsLoader::get_config() const { return impl_->config; }

bool SafetensorsLoader::read_floats(const std::string &name, std::vector<float> *out, std::string *err) const {
  const TensorInfo *t = find(name);
  if (!t) return fail(err, "safetensors: tensor not found: " + name);
  const uint8_t *p = impl_->map + impl_->data_offset + t->offset;
  const size_t eb = element_bytes(t->dtype), n = eb ? t->size_bytes / eb : 0;
  out->resize(n);
  float *o = out->data();
  if (t->dtype == "BF16") {
#pragma omp parallel for schedule(static)
    for (size_t i = 0; i < n; ++i) {
      uint16_t h;
      std::memcpy(&h, p + 2 * i, 2);
      const uint32_t b = (uint32_t)h << 16;
      std::memcpy(o + i, &b, 4);
    }
  } else if (t->dtype == "F16") {
    for (size_t i = 0; i < n; ++i) {
      uint16_t h;
      std::memcpy(&h, p + 2 * i, 2);
      o[i] = host::f16_to_f32(h);
    }
  } else if (t->dtype == "F32") {
    std::memcpy(o, p, n * 4);
  } else {
    return fail(err, "safetensors: " + name + " has type " + t->dtype + ", not a float type that is read here");
  }
  return true;
}

bool SafetensorsLoader::load_tensor(const std::string &name, gcore::rt::cuda::Buffer &buffer, std::string *err) {
  std::vector<float> v;
  if (!read_floats(name, &v, err)) return false;
  if (buffer.size() < v.size() * 4 && !buffer.allocate(v.size() * 4, gcore::rt::cuda::BufferUsage::DeviceOnly, GretaDataType::FP32, err)) return false;
  return buffer.copy_to_device(v.data(), v.size() * 4, err);
}
bool SafetensorsLoader::load_tensor_fp16(const std::string &name, gcore::rt::cuda::Buffer &buffer, std::string *err) {
  std::vector<float> v;
  if (!read_floats(name, &v, err)) return false;
  std::vector<uint16_t> h(v.size());
  for (size_t i = 0; i < v.size(); ++i) h[i] = host::f32_to_f16(v[i]);
  if (buffer.size() < h.size() * 2 && !buffer.allocate(h.size() * 2, gcore::rt::cuda::BufferUsage::DeviceOnly, GretaDataType::FP16, err)) return false;
  return buffer.copy_to_device(h.data(), h.size() * 2, err);
}
bool SafetensorsLoader::load_tensor_int8(const std::string &name, gcore::rt::cuda::Buffer &, gcore::rt::cuda::Buffer &, std::string *err) {
  return fail(err, "safetensors: " + name + " is not re-quantised (load_tensor_int8)");
}
bool SafetensorsLoader::load_tensor_int4(const std::string &name, gcore::rt::cuda::Buffer &, gcore::rt::cuda::Buffer &, gcore::rt::cuda::Buffer &,
                                         std::string *err) {
  return fail(err, "safetensors: " + name + " is not re-quantised (load_tensor_int4)");
}

}  // namespace gcore::inference
