// Pieces of a decoder design's description: members of its config.json, and the entry of the design registry.
#pragma once

#include <cmath>
#include <string>
#include <vector>

#include "../common.cuh"
#include "json.hpp"
#include "weights.hpp"

namespace evob {

inline int size_member(const Json &object, const char *key, const std::string &where, const std::size_t minimum,
                       std::size_t *out) {
  const Json *value = object.get(key);
  if (value == nullptr || value->kind != Json::kNumber || !(value->number >= static_cast<double>(minimum)) ||
      value->number > 2147483647.0 || value->number != std::floor(value->number))
    return fail(kModelFormat, "config.json: " + where + "." + key + " must be an integer of at least " +
                                  std::to_string(minimum));
  *out = static_cast<std::size_t>(value->number);
  return kOk;
}

inline int real_member(const Json &object, const char *key, const std::string &where, const bool positive, float *out) {
  const Json *value = object.get(key);
  if (value == nullptr || value->kind != Json::kNumber || !std::isfinite(value->number) ||
      (positive && !(value->number > 0.0)))
    return fail(kModelFormat, "config.json: " + where + "." + key + " must be a " +
                                  (positive ? "positive " : "") + "number");
  *out = static_cast<float>(value->number);
  return kOk;
}

inline int object_member(const Json &object, const char *key, const std::string &where, const Json **out) {
  const Json *value = object.get(key);
  if (value == nullptr || value->kind != Json::kObject)
    return fail(kModelFormat, "config.json: " + where + "." + key + " must be an object");
  *out = value;
  return kOk;
}

// A design that a config.json describes, by the architecture it names: its reader, its tensors and their place
// in a stage's slab.  The forward pass is the decoder graph's (decoder.cu).
struct DecoderDesign {
  const char *architecture;
  int (*read)(const ModelFile &file, ModelConfig *config);
  std::vector<ExpectedTensor> (*model_tensors)(const ModelConfig &config);
  std::vector<ExpectedTensor> (*block_tensors)(const ModelConfig &config, std::size_t layer);
  int (*upload_model)(const ModelFile &file, const ModelConfig &config, WeightUploader *up, StageWeights *stage);
  int (*upload_block)(const ModelFile &file, const ModelConfig &config, std::size_t layer, WeightUploader *up,
                      LayerWeights *weights);
};
extern const DecoderDesign kGigusunDesign;  // gigusun.cpp
extern const DecoderDesign kKikepelDesign;  // kikepel.cpp

}  // namespace evob
