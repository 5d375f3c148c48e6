// A model opened from a folder or a GGUF file, ready to run: shared by the command-line programs.
#pragma once
#include <algorithm>
#include <memory>
#include <string>

#include "gcore/greta_b200.hpp"

namespace gcore::cli {

struct Session {
  inference::ModelConfig config;
  inference::BlockScheduler scheduler;
  inference::Generator generator;

  // fp32: run an unquantised design in true 32-bit.  max_seq: positions of a sequence; 0: as many as the model has or, where
  // nothing bounds them, `needed`.  A model with no more than `roomy` positions gets them all.
  bool open(const std::string &path, bool fp32, size_t batch, size_t max_seq, std::string *err, size_t roomy = 0, size_t needed = 0) {
    std::unique_ptr<inference::WeightLoader> loader = inference::create_weight_loader(path, err);
    if (!loader) return false;
    config = loader->get_config();
    if (config.arch == inference::ModelArch::HYBRID) {
      config.weight_type = config.lm_head_type = fp32 ? rt::GretaDataType::FP32 : rt::GretaDataType::BF16;
    } else if (fp32) {
      *err = "32-bit computation: only unquantised model folders run in it";
      return false;
    }
    if (!max_seq && config.default_seq_len) max_seq = needed ? needed : config.default_seq_len;
    const size_t seq = max_seq && config.max_seq_len > roomy ? std::min<size_t>(max_seq, config.max_seq_len) : config.max_seq_len;
    return scheduler.init(config, err) && scheduler.allocate_weights(err) && scheduler.load_weights(*loader, err) &&
           scheduler.allocate_activations(batch, seq, err) && generator.init(config, &scheduler, err);
  }
};

}  // namespace gcore::cli
