// The Gigusun design: a decoder whose blocks mix tokens by softmax attention in a sliding window, by gated
// linear attention or by the gated delta rule, each followed by an optional feed-forward with a normalised
// polynomial activation.  This file reads its config.json, names its tensors and lays them out for the
// decoder graph (decoder.cu); it holds no arithmetic of the forward pass.
//
// config.json: {"architecture": "Gigusun", "vocab", "width", "max_positions", "norm": {"eps"},
//   "layers": [{"type": "attention" | "gla" | "delta", "mixer": {...}, "mlp": {"kind": "dense", "ff"} | null}]}
//   attention: heads, kv_heads, dim, vdim, scale, softcap, mask {size, keep_first}
//   gla:       heads, dim, vdim, tau
//   delta:     heads, kv_heads, dim, vdim, conv
#include <algorithm>
#include <cmath>

#include "../decoder_ops.hpp"
#include "decoder_config.hpp"

namespace evob {
namespace {

#define EVOB_TRY(expr)              \
  do {                              \
    const int status__ = (expr);    \
    if (status__ != kOk) return status__; \
  } while (0)

int read_block(const ModelFile &file, const Json &entry, const std::size_t index, DecoderBlock *block) {
  const std::string where = "layers[" + std::to_string(index) + "]";
  const Json *type = entry.get("type"), *mixer = entry.get("mixer"), *mlp = entry.get("mlp");
  if (type == nullptr || type->kind != Json::kString || mixer == nullptr || mixer->kind != Json::kObject)
    return fail(kModelFormat, "config.json: " + where + " needs a type and a mixer");
  DecoderBlock b;
  const std::string in = where + ".mixer";
  EVOB_TRY(size_member(*mixer, "heads", in, 1, &b.heads));
  EVOB_TRY(size_member(*mixer, "dim", in, 1, &b.dim));
  EVOB_TRY(size_member(*mixer, "vdim", in, 1, &b.value_dim));
  b.kv_heads = b.heads;
  if (type->text == "attention" || type->text == "delta") {
    EVOB_TRY(size_member(*mixer, "kv_heads", in, 1, &b.kv_heads));
    if (b.heads % b.kv_heads != 0)
      return fail(kModelFormat, "config.json: " + in + ".heads is not a multiple of kv_heads");
  }
  if (type->text == "attention") {
    b.mixer = MixerType::kWindowAttention;
    EVOB_TRY(real_member(*mixer, "scale", in, false, &b.scale));
    EVOB_TRY(real_member(*mixer, "softcap", in, true, &b.softcap));
    const Json *mask = mixer->get("mask");
    if (mask == nullptr || mask->kind != Json::kObject)
      return fail(kModelFormat, "config.json: " + in + " needs a mask");
    EVOB_TRY(size_member(*mask, "size", in + ".mask", 1, &b.window));
    EVOB_TRY(size_member(*mask, "keep_first", in + ".mask", 0, &b.keep_first));
  } else if (type->text == "gla") {
    b.mixer = MixerType::kGatedLinear;
    EVOB_TRY(real_member(*mixer, "tau", in, true, &b.tau));
    const TensorView *bottleneck = file.find("l" + std::to_string(index) + ".mix.a1");
    if (bottleneck == nullptr || bottleneck->shape.size() != 2)
      return fail(kModelFormat, "required tensor is missing: l" + std::to_string(index) + ".mix.a1");
    b.decay_rank = bottleneck->shape[0];
  } else if (type->text == "delta") {
    b.mixer = MixerType::kGatedDelta;
    EVOB_TRY(size_member(*mixer, "conv", in, 1, &b.conv_taps));
  } else {
    return fail(kUnsupported, "config.json: " + where + " has an unknown mixer type: " + type->text);
  }
  if (b.dim > kDecoderMaxHeadDim || (b.mixer == MixerType::kWindowAttention && b.value_dim > kDecoderMaxHeadDim))
    return fail(kUnsupported, "config.json: " + in + " head sizes above " + std::to_string(kDecoderMaxHeadDim) +
                                  " are not supported");
  if (mlp != nullptr && mlp->kind != Json::kNull) {
    const Json *kind = mlp->get("kind");
    if (mlp->kind != Json::kObject || kind == nullptr || kind->kind != Json::kString || kind->text != "dense")
      return fail(kUnsupported, "config.json: " + where + ".mlp is not a dense feed-forward");
    b.feed_forward = FeedForward::kPolyNorm;
    EVOB_TRY(size_member(*mlp, "ff", where + ".mlp", 1, &b.inner_width));
  }
  *block = b;
  return kOk;
}

std::vector<float> one_plus(std::vector<float> values) {
  for (float &v : values) v = 1.0F + v;
  return values;
}

int read_gigusun_config(const ModelFile &file, ModelConfig *config) {
  const Json *const root = file.configuration();
  if (root == nullptr) return fail(kModelFormat, "the model directory has no config.json");
  ModelConfig c;
  c.graph = BlockGraph::kDecoder;
  c.design = &kGigusunDesign;
  c.learned_positions = true;
  c.architecture = "Gigusun";
  c.artifact_profile = "decoder-config-v1";
  EVOB_TRY(size_member(*root, "vocab", "model", 1, &c.vocab));
  EVOB_TRY(size_member(*root, "width", "model", 1, &c.width));
  EVOB_TRY(size_member(*root, "max_positions", "model", 1, &c.max_seqlen));
  const Json *norm = root->get("norm"), *layers = root->get("layers");
  if (norm == nullptr || norm->kind != Json::kObject) return fail(kModelFormat, "config.json: norm is missing");
  EVOB_TRY(real_member(*norm, "eps", "norm", true, &c.epsilon));
  if (layers == nullptr || layers->kind != Json::kArray || layers->items.empty())
    return fail(kModelFormat, "config.json: layers must be a non-empty list");
  c.layers = layers->items.size();
  for (std::size_t i = 0; i < c.layers; ++i) {
    DecoderBlock block;
    EVOB_TRY(read_block(file, layers->items[i], i, &block));
    c.blocks.push_back(block);
    c.mixers.push_back(block.mixer);
    c.heads = std::max(c.heads, block.heads);
    c.inner_width = std::max(c.inner_width, block.inner_width);
    c.state_size = std::max(c.state_size, block.mixer == MixerType::kWindowAttention ? 0 : block.dim);
    c.short_taps = std::max(c.short_taps, block.conv_taps);
  }
  *config = std::move(c);
  return kOk;
}

std::vector<ExpectedTensor> gigusun_model_tensors(const ModelConfig &c) {
  return {{"embed", TensorType::kBF16, {c.vocab, c.width}},
          {"pos", TensorType::kBF16, {c.max_seqlen, c.width}},
          {"embed.norm", TensorType::kBF16, {c.width}},
          {"final.norm", TensorType::kBF16, {c.width}},
          {"head", TensorType::kBF16, {c.vocab, c.width}}};
}

std::vector<ExpectedTensor> gigusun_block_tensors(const ModelConfig &c, const std::size_t layer) {
  const DecoderBlock &b = c.blocks[layer];
  const std::string l = "l" + std::to_string(layer) + ".", p = l + "mix.";
  const std::size_t D = c.width;
  std::vector<ExpectedTensor> list;
  const auto add = [&list](const std::string &name, std::vector<std::size_t> shape) {
    list.push_back({name, TensorType::kBF16, std::move(shape)});
  };
  add(l + "norm1", {D});
  add(p + "q", {b.query_width(), D});
  add(p + "k", {b.key_width(), D});
  add(p + "v", {b.value_width(), D});
  add(p + "g", {b.gate_width(), D});
  add(p + "o", {D, b.output_width()});
  switch (b.mixer) {
    case MixerType::kWindowAttention:
      add(p + "q.norm", {b.dim});
      add(p + "k.norm", {b.dim});
      add(p + "r1", {b.heads});
      add(p + "r2", {b.heads});
      break;
    case MixerType::kGatedLinear:
      add(p + "a1", {b.decay_rank, D});
      add(p + "a2", {b.heads * b.dim, b.decay_rank});
      add(p + "a2.b", {b.heads * b.dim});
      add(p + "norm", {b.value_dim});
      break;
    default:
      add(p + "q.conv", {b.query_width(), b.conv_taps});
      add(p + "k.conv", {b.key_width(), b.conv_taps});
      add(p + "v.conv", {b.value_width(), b.conv_taps});
      add(p + "b", {b.heads, D});
      add(p + "a", {b.heads, D});
      add(p + "A_log", {b.heads});
      add(p + "dt_bias", {b.heads});
      add(p + "norm", {b.value_dim});
      break;
  }
  if (b.inner_width != 0) {
    add(l + "norm2", {D});
    add(l + "mlp.up", {b.inner_width, D});
    add(l + "mlp.down", {D, b.inner_width});
    add(l + "mlp.act", {4});
  }
  return list;
}

int upload_gigusun_model(const ModelFile &file, const ModelConfig &, WeightUploader *up, StageWeights *stage) {
  EVOB_TRY(up->tensor(*file.find("embed"), &stage->embedding));
  EVOB_TRY(up->tensor(*file.find("pos"), &stage->positions));
  EVOB_TRY(up->tensor(*file.find("head"), &stage->head));
  EVOB_TRY(up->floats(one_plus(widened(*file.find("embed.norm"))), &stage->embedding_norm));
  return up->floats(one_plus(widened(*file.find("final.norm"))), &stage->final_norm);
}

int upload_gigusun_block(const ModelFile &file, const ModelConfig &c, const std::size_t layer, WeightUploader *up,
                         LayerWeights *w) {
  const DecoderBlock &b = c.blocks[layer];
  for (const ExpectedTensor &e : gigusun_block_tensors(c, layer)) {
    const TensorView *view = nullptr;
    EVOB_TRY(lookup_tensor(file, e, &view));
    w->payload_bytes += view->bytes;
  }
  const std::string l = "l" + std::to_string(layer) + ".", p = l + "mix.";
  const auto view = [&file](const std::string &name) -> const TensorView & { return *file.find(name); };
  w->type = b.mixer;
  EVOB_TRY(up->floats(one_plus(widened(view(l + "norm1"))), &w->pre_norm));
  // fused input projection: the segments' rows one after another, zeros between them
  {
    const std::size_t row_bytes = c.width * 2, bytes = b.projection_width() * row_bytes;
    unsigned char *const dst = static_cast<unsigned char *>(up->place(bytes));
    w->projection = dst;
    if (!up->dry_run && cudaMemsetAsync(dst, 0, bytes, up->stream) != cudaSuccess)
      return fail(kCuda, "weight upload failed");
    const auto segment = [&](const char *name, const std::size_t column) {
      const TensorView &t = view(p + name);
      return up->copy(up->dry_run ? nullptr : dst + column * row_bytes, t.data, t.bytes);
    };
    EVOB_TRY(segment("q", 0));
    EVOB_TRY(segment("k", b.key_column()));
    EVOB_TRY(segment("v", b.value_column()));
    EVOB_TRY(segment("g", b.gate_column()));
    if (b.mixer == MixerType::kGatedLinear) EVOB_TRY(segment("a1", b.beta_column()));
    if (b.mixer == MixerType::kGatedDelta) {
      EVOB_TRY(segment("b", b.beta_column()));
      EVOB_TRY(segment("a", b.decay_column()));
    }
  }
  EVOB_TRY(up->tensor(view(p + "o"), &w->out_weight));
  switch (b.mixer) {
    case MixerType::kWindowAttention: {
      EVOB_TRY(up->floats(widened(view(p + "q.norm")), &w->query_norm));
      EVOB_TRY(up->floats(widened(view(p + "k.norm")), &w->key_norm));
      // r1 ln(1 + r2 d) for every head and distance: the score kernels read it from this table
      const std::vector<float> r1 = widened(view(p + "r1")), r2 = widened(view(p + "r2"));
      const float *rates = nullptr;
      std::vector<float> both(r1);
      both.insert(both.end(), r2.begin(), r2.end());
      EVOB_TRY(up->floats(std::move(both), &rates));
      float *const table = static_cast<float *>(up->place(b.heads * c.max_seqlen * sizeof(float)));
      w->distance_bias = table;
      if (!up->dry_run)
        EVOB_TRY(distance_bias_table(rates, rates + b.heads, b.heads, c.max_seqlen, table, up->stream));
      break;
    }
    case MixerType::kGatedLinear: {
      // [channels, rank] -> [rank, channels]: neighbouring threads read neighbouring channels
      const std::vector<float> a2 = widened(view(p + "a2"));
      const std::size_t channels = b.heads * b.dim;
      std::vector<float> transposed(a2.size());
      for (std::size_t channel = 0; channel < channels; ++channel)
        for (std::size_t r = 0; r < b.decay_rank; ++r)
          transposed[r * channels + channel] = a2[channel * b.decay_rank + r];
      EVOB_TRY(up->floats(std::move(transposed), &w->decay_weight));
      EVOB_TRY(up->floats(widened(view(p + "a2.b")), &w->decay_bias));
      EVOB_TRY(up->floats(widened(view(p + "norm")), &w->output_norm));
      break;
    }
    default: {
      std::vector<float> taps(b.gate_column() * b.conv_taps, 0.0F);
      const auto place = [&](const char *name, const std::size_t column) {
        const std::vector<float> values = widened(view(p + name));
        std::copy(values.begin(), values.end(), taps.begin() + static_cast<std::ptrdiff_t>(column * b.conv_taps));
      };
      place("q.conv", 0);
      place("k.conv", b.key_column());
      place("v.conv", b.value_column());
      EVOB_TRY(up->floats(std::move(taps), &w->conv));
      std::vector<float> rate = widened(view(p + "A_log"));
      for (float &v : rate) v = -std::exp(v);
      EVOB_TRY(up->floats(std::move(rate), &w->decay_rate));
      EVOB_TRY(up->floats(widened(view(p + "dt_bias")), &w->decay_shift));
      EVOB_TRY(up->floats(widened(view(p + "norm")), &w->output_norm));
      break;
    }
  }
  if (b.inner_width != 0) {
    EVOB_TRY(up->floats(one_plus(widened(view(l + "norm2"))), &w->post_norm));
    EVOB_TRY(up->tensor(view(l + "mlp.up"), &w->l1));
    EVOB_TRY(up->tensor(view(l + "mlp.down"), &w->l3));
    EVOB_TRY(up->floats(widened(view(l + "mlp.act")), &w->activation));
  }
  return kOk;
}

}  // namespace

const DecoderDesign kGigusunDesign = {"Gigusun",          read_gigusun_config,  gigusun_model_tensors, gigusun_block_tensors,
                                      upload_gigusun_model, upload_gigusun_block};

}  // namespace evob
