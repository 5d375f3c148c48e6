// Greedy generation over token ids from the command line (the tokenizer is outside this path).
//
//   greta_infer --model DIR|FILE.gguf --tokens 1,2,3[;4,5] [--max-tokens N] [--dtype bfloat16|float32] [--eos ID] [--max-seq N]
//
// Prompts separated by ';' run as one batch.  Prints one line of generated ids per prompt, then timing on standard error.
// The reference's program of this name is tools/inference/src/greta_infer.cpp.
#include <cstdio>
#include <cstdlib>
#include <sstream>

#include "model_session.hpp"

namespace {
int complain(const std::string &msg, int code = 1) {
  std::fprintf(stderr, "greta_infer: %s\n", msg.c_str());
  return code;
}
}  // namespace

int main(int argc, char **argv) {
  std::string model, dtype = "bfloat16", tokens, err;
  gcore::inference::SamplingParams sp;
  sp.greedy = true;
  sp.max_tokens = 32;
  size_t max_seq = 0;
  for (int i = 1; i + 1 < argc; i += 2) {
    const std::string k = argv[i], v = argv[i + 1];
    if (k == "--model") model = v;
    else if (k == "--dtype") dtype = v;
    else if (k == "--tokens") tokens = v;
    else if (k == "--max-tokens") sp.max_tokens = std::atoi(v.c_str());
    else if (k == "--eos") sp.eos_token_id = std::atoi(v.c_str());
    else if (k == "--max-seq") max_seq = std::strtoull(v.c_str(), nullptr, 10);
    else return complain("unknown option " + k, 2);
  }
  std::vector<std::vector<int32_t>> prompts;
  std::stringstream list(tokens);
  for (std::string part; std::getline(list, part, ';');) {
    prompts.emplace_back();
    std::stringstream ids(part);
    for (std::string id; std::getline(ids, id, ',');) prompts.back().push_back(std::atoi(id.c_str()));
  }
  if (model.empty() || prompts.empty() || (dtype != "bfloat16" && dtype != "float32"))
    return complain("usage: greta_infer --model DIR|FILE.gguf --tokens 1,2,3[;4,5] [--max-tokens N] [--dtype bfloat16|float32] [--eos ID] [--max-seq N]", 2);
  size_t longest = 0;
  for (const auto &p : prompts) longest = std::max(longest, p.size());
  gcore::cli::Session s;
  if (!s.open(model, dtype == "float32", prompts.size(), max_seq, &err, 0, longest + (size_t)std::max(sp.max_tokens, 1))) return complain(err);
  std::vector<std::vector<int32_t>> out;
  if (prompts.size() == 1) {
    gcore::inference::GenerationStats st;
    out.push_back(s.generator.generate_tokens(prompts[0], sp, &st, &err));
    if (err.empty()) std::fprintf(stderr, "%zu prompt + %zu new ids, first after %.2f ms, decode %.2f ms\n", st.prompt_tokens, st.generated_tokens, st.time_to_first_token_ms, st.decode_time_ms);
  } else {
    out = s.generator.generate_batch(prompts, sp, &err);
  }
  if (!err.empty()) return complain(err);
  for (const auto &ids : out) {
    for (size_t i = 0; i < ids.size(); ++i) std::printf(i ? ",%d" : "%d", ids[i]);
    std::printf("\n");
  }
  return 0;
}
