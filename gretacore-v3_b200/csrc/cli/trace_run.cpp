// Replays a trace of token ids through a model and writes logits.
//
//   trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N
//
// Steps come as JSON lines on standard input:
//   {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": ["a"]}
// Every entry brings the next tokens of a request; the logits at the places in `want` go to DIR/<step>.f32 as little-endian
// floats [wanted, vocab], in the order asked; requests in `end` give their sequence slot back.  A line "done <step>" follows.
#include <cstdio>
#include <cstring>
#include <iostream>
#include <map>
#include <numeric>

#include "json.hpp"
#include "model_session.hpp"

using gcore::host::Json;

namespace {

constexpr size_t kSlots = 4;  // requests that may be alive at the same time

struct Live {
  uint32_t slot;
  size_t length;
};

int complain(const std::string &msg, int code = 1) {
  std::fprintf(stderr, "trace_run: %s\n", msg.c_str());
  return code;
}

bool id_of(const Json &v, std::string *out) {
  if (v.kind == Json::STRING) *out = v.string;
  else if (v.kind == Json::NUMBER) *out = std::to_string((long long)v.number);
  else return false;
  return true;
}

}  // namespace

int main(int argc, char **argv) {
  std::string model, out_dir, dtype = "bfloat16", err;
  size_t max_tokens = 0;
  for (int i = 1; i + 1 < argc; i += 2) {
    const std::string k = argv[i], v = argv[i + 1];
    if (k == "--model") model = v;
    else if (k == "--dtype") dtype = v;
    else if (k == "--out") out_dir = v;
    else if (k == "--max-tokens") max_tokens = std::strtoull(v.c_str(), nullptr, 10);
    else return complain("unknown option " + k, 2);
  }
  if (model.empty() || out_dir.empty() || (dtype != "bfloat16" && dtype != "float32"))
    return complain("usage: trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N", 2);
  gcore::cli::Session s;
  if (!s.open(model, dtype == "float32", kSlots, max_tokens, &err, 16384)) return complain(err);
  auto &sched = s.scheduler;
  const size_t V = s.config.vocab_size;

  std::map<std::string, Live> live;
  std::vector<uint32_t> free_slots{3, 2, 1, 0};
  std::string line;
  while (std::getline(std::cin, line)) {
    if (line.find_first_not_of(" \t\r") == std::string::npos) continue;
    Json step;
    if (!Json::parse(line, &step, &err)) return complain(err);
    const Json *number = step.get("step"), *entries = step.get("entries"), *end = step.get("end");
    uint32_t n = 0;
    if (!number || !number->as_u32(&n)) return complain("a step without a number");
    std::vector<float> result;
    for (const Json &e : entries ? entries->items : std::vector<Json>{}) {
      const Json *id = e.get("id"), *tokens = e.get("tokens"), *want = e.get("want");
      std::string name;
      if (!id || !id_of(*id, &name) || !tokens || tokens->items.empty()) return complain("an entry without id or tokens");
      auto it = live.find(name);
      if (it == live.end()) {
        if (free_slots.empty()) return complain("more than " + std::to_string(kSlots) + " requests alive at once");
        it = live.emplace(name, Live{free_slots.back(), 0}).first;
        free_slots.pop_back();
      }
      std::vector<int32_t> ids;
      for (const Json &t : tokens->items) {
        if (t.kind != Json::NUMBER || t.number < 0 || t.number >= (double)V) return complain("a token outside the vocabulary");
        ids.push_back((int32_t)t.number);
      }
      std::vector<uint32_t> places;
      for (const Json &w : want ? want->items : std::vector<Json>{}) {
        uint32_t p = 0;
        if (!w.as_u32(&p) || p >= ids.size()) return complain("a wanted place outside the entry's tokens");
        places.push_back(p);
      }
      std::vector<uint32_t> rows = places;  // ascending and distinct for the scheduler
      std::sort(rows.begin(), rows.end());
      rows.erase(std::unique(rows.begin(), rows.end()), rows.end());
      std::vector<float> z(rows.size() * V);
      if (!sched.set_sequence(it->second.slot, &err) ||
          !sched.forward_logits(ids.data(), it->second.length, ids.size(), rows.data(), rows.size(), z.data(), &err))
        return complain(err);
      it->second.length += ids.size();
      for (uint32_t p : places) {
        const size_t r = (size_t)(std::lower_bound(rows.begin(), rows.end(), p) - rows.begin());
        result.insert(result.end(), z.begin() + r * V, z.begin() + (r + 1) * V);
      }
    }
    if (!result.empty()) {
      const std::string path = out_dir + "/" + std::to_string(n) + ".f32";
      FILE *f = std::fopen(path.c_str(), "wb");
      if (!f || std::fwrite(result.data(), 4, result.size(), f) != result.size() || std::fclose(f) != 0) return complain("cannot write " + path);
    }
    for (const Json &e : end ? end->items : std::vector<Json>{}) {
      std::string name;
      auto it = id_of(e, &name) ? live.find(name) : live.end();
      if (it == live.end()) continue;
      free_slots.push_back(it->second.slot);
      live.erase(it);
    }
    std::printf("done %u\n", n);
    std::fflush(stdout);
  }
  int code = 0;
  if (greta_cuda_linear_gemm_status(&code) != GRETA_OK || code != 0) return complain("a bounded wait of a GEMM kernel gave up (code " + std::to_string(code) + ")");
  return 0;
}
