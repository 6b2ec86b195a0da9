// The Kikepel design: a decoder whose blocks attend through low-rank latents in a sliding window, with or without
// a learned sink per head, and whose feed-forwards are dense ReLU-gated ones or mixtures of clamped-gate experts.
// Sublayers read the residual stream itself; a layer norm sits on what each of them adds to it.  This file reads
// its config.json, names its tensors and lays them out for the decoder graph (decoder.cu); it holds no arithmetic
// of the forward pass.
//
// config.json: {"architecture": "Kikepel", "vocab", "width", "norm": {"eps"}, "logit_scale", "logit_softcap",
//   "layers": [{"type": "latent_attention" (with sinks) | "latent_attention_2" (without), "mixer": {"heads", "dim",
//     "vdim", "q_rank", "kv_rank", "scale", "mask": {"size"}}, "mlp": {"kind": "dense", "ff"} |
//     {"kind": "moe", "expert": {"ff", "limit"}, "router": {"experts", "top"}} | null}]}
#include <algorithm>
#include <cstring>

#include "../decoder_ops.hpp"
#include "decoder_config.hpp"

namespace evob {
namespace {

#define EVOB_TRY(expr)              \
  do {                              \
    const int status__ = (expr);    \
    if (status__ != kOk) return status__; \
  } while (0)

// There are no positions to run out of; what bounds a context is that its rows are counted in 32 bits.
constexpr std::size_t kLongestContext = std::size_t{1} << 30;

int read_feed_forward(const Json &mlp, const std::string &where, DecoderBlock *b) {
  const Json *kind = mlp.get("kind");
  if (mlp.kind != Json::kObject || kind == nullptr || kind->kind != Json::kString)
    return fail(kModelFormat, "config.json: " + where + " needs a kind");
  if (kind->text == "dense") {
    b->feed_forward = FeedForward::kReluGated;
    return size_member(mlp, "ff", where, 1, &b->inner_width);
  }
  if (kind->text != "moe")
    return fail(kUnsupported, "config.json: " + where + " has an unknown kind of feed-forward: " + kind->text);
  b->feed_forward = FeedForward::kExperts;
  const Json *expert = nullptr, *router = nullptr;
  EVOB_TRY(object_member(mlp, "expert", where, &expert));
  EVOB_TRY(object_member(mlp, "router", where, &router));
  EVOB_TRY(size_member(*expert, "ff", where + ".expert", 1, &b->inner_width));
  EVOB_TRY(real_member(*expert, "limit", where + ".expert", true, &b->gate_limit));
  EVOB_TRY(size_member(*router, "experts", where + ".router", 1, &b->experts));
  EVOB_TRY(size_member(*router, "top", where + ".router", 1, &b->top));
  if (b->top > b->experts) return fail(kModelFormat, "config.json: " + where + ".router.top is above the number of experts");
  if (b->experts > kDecoderMaxExperts)
    return fail(kUnsupported, "config.json: " + where + ".router has more than " + std::to_string(kDecoderMaxExperts) +
                                  " experts");
  return kOk;
}

int read_block(const Json &entry, const std::size_t index, DecoderBlock *block) {
  const std::string where = "layers[" + std::to_string(index) + "]", in = where + ".mixer";
  const Json *type = entry.get("type"), *mlp = entry.get("mlp"), *mixer = nullptr, *mask = nullptr;
  if (type == nullptr || type->kind != Json::kString) return fail(kModelFormat, "config.json: " + where + " needs a type");
  if (type->text != "latent_attention" && type->text != "latent_attention_2")
    return fail(kUnsupported, "config.json: " + where + " has an unknown mixer type: " + type->text);
  EVOB_TRY(object_member(entry, "mixer", where, &mixer));
  EVOB_TRY(object_member(*mixer, "mask", in, &mask));
  DecoderBlock b;
  b.mixer = MixerType::kLatentAttention;
  b.sink = type->text == "latent_attention";
  EVOB_TRY(size_member(*mixer, "heads", in, 1, &b.heads));
  EVOB_TRY(size_member(*mixer, "dim", in, 1, &b.dim));
  EVOB_TRY(size_member(*mixer, "vdim", in, 1, &b.value_dim));
  EVOB_TRY(size_member(*mixer, "q_rank", in, 1, &b.query_rank));
  EVOB_TRY(size_member(*mixer, "kv_rank", in, 1, &b.latent_rank));
  EVOB_TRY(real_member(*mixer, "scale", in, false, &b.scale));
  EVOB_TRY(size_member(*mask, "size", in + ".mask", 1, &b.window));
  b.kv_heads = b.heads;
  if (b.dim > kDecoderMaxHeadDim || b.value_dim > kDecoderMaxHeadDim)
    return fail(kUnsupported, "config.json: " + in + " head sizes above " + std::to_string(kDecoderMaxHeadDim) +
                                  " are not supported");
  if (b.latent_rank > kDecoderMaxLatent)
    return fail(kUnsupported, "config.json: " + in + ".kv_rank above " + std::to_string(kDecoderMaxLatent) +
                                  " is not supported");
  if (mlp != nullptr && mlp->kind != Json::kNull) EVOB_TRY(read_feed_forward(*mlp, where + ".mlp", &b));
  *block = b;
  return kOk;
}

int read_kikepel_config(const ModelFile &file, ModelConfig *config) {
  const Json *const root = file.configuration();
  if (root == nullptr) return fail(kModelFormat, "the model directory has no config.json");
  ModelConfig c;
  c.graph = BlockGraph::kDecoder;
  c.design = &kKikepelDesign;
  c.architecture = kKikepelDesign.architecture;
  c.artifact_profile = "decoder-config-v1";
  c.output_norms = true;
  c.max_seqlen = kLongestContext;
  EVOB_TRY(size_member(*root, "vocab", "model", 1, &c.vocab));
  EVOB_TRY(size_member(*root, "width", "model", 1, &c.width));
  EVOB_TRY(real_member(*root, "logit_scale", "model", false, &c.logit_scale));
  EVOB_TRY(real_member(*root, "logit_softcap", "model", true, &c.logit_softcap));
  const Json *norm = nullptr, *layers = root->get("layers");
  EVOB_TRY(object_member(*root, "norm", "model", &norm));
  EVOB_TRY(real_member(*norm, "eps", "norm", true, &c.epsilon));
  if (layers == nullptr || layers->kind != Json::kArray || layers->items.empty())
    return fail(kModelFormat, "config.json: layers must be a non-empty list");
  c.layers = layers->items.size();
  for (std::size_t i = 0; i < c.layers; ++i) {
    DecoderBlock block;
    EVOB_TRY(read_block(layers->items[i], i, &block));
    c.blocks.push_back(block);
    c.mixers.push_back(block.mixer);
    c.heads = std::max(c.heads, block.heads);
    c.inner_width = std::max(c.inner_width, block.inner_width);
  }
  *config = std::move(c);
  return kOk;
}

std::vector<ExpectedTensor> kikepel_model_tensors(const ModelConfig &c) {
  return {{"embed", TensorType::kBF16, {c.vocab, c.width}},
          {"final.norm", TensorType::kBF16, {c.width}},
          {"head", TensorType::kBF16, {c.vocab, c.width}}};
}

std::vector<ExpectedTensor> kikepel_block_tensors(const ModelConfig &c, const std::size_t layer) {
  const DecoderBlock &b = c.blocks[layer];
  const std::string l = "l" + std::to_string(layer) + ".", p = l + "mix.", m = l + "mlp.";
  const std::size_t D = c.width, I = b.inner_width;
  std::vector<ExpectedTensor> list;
  const auto add = [&list](const std::string &name, std::vector<std::size_t> shape) {
    list.push_back({name, TensorType::kBF16, std::move(shape)});
  };
  add(l + "norm1", {D});
  add(p + "dq", {b.query_rank, D});
  add(p + "dq.norm", {b.query_rank});
  add(p + "uq", {b.heads * b.dim, b.query_rank});
  add(p + "dkv", {b.latent_rank, D});
  add(p + "dkv.norm", {b.latent_rank});
  add(p + "uk", {b.heads * b.dim, b.latent_rank});
  add(p + "uv", {b.heads * b.value_dim, b.latent_rank});
  add(p + "o", {D, b.heads * b.value_dim});
  if (b.sink) add(p + "sink", {b.heads});
  if (b.feed_forward == FeedForward::kNone) return list;
  add(l + "norm2", {D});
  if (b.feed_forward == FeedForward::kReluGated) {
    for (const char *name : {"gate", "up"}) {
      add(m + name, {I, D});
      add(m + name + ".b", {I});
    }
    add(m + "down", {D, I});
    add(m + "down.b", {D});
    return list;
  }
  add(m + "router", {b.experts, D});
  for (std::size_t e = 0; e < b.experts; ++e) {
    const std::string x = m + "e" + std::to_string(e) + ".";
    add(x + "gate", {I, D});
    add(x + "up", {I, D});
    add(x + "down", {D, I});
  }
  return list;
}

int upload_kikepel_model(const ModelFile &file, const ModelConfig &, WeightUploader *up, StageWeights *stage) {
  EVOB_TRY(up->tensor(*file.find("embed"), &stage->embedding));
  EVOB_TRY(up->tensor(*file.find("head"), &stage->head));
  return up->floats(widened(*file.find("final.norm")), &stage->final_norm);
}

// Gate and up rows in alternating blocks of 128 at `gated`, the down matrix with padded rows at `down`.
int place_gated(WeightUploader *up, const DecoderBlock &b, const std::size_t width, const TensorView &gate,
                const TensorView &raise, const TensorView &lower, unsigned char *gated, unsigned char *down) {
  if (up->dry_run) return kOk;
  const std::size_t row_bytes = width * 2, inner_bytes = b.inner_width * 2;
  for (std::size_t row = 0; row < b.inner_width; row += 128) {
    const std::size_t bytes = std::min<std::size_t>(128, b.inner_width - row) * row_bytes;
    EVOB_TRY(up->copy(gated + 2 * row * row_bytes, gate.data + row * row_bytes, bytes));
    EVOB_TRY(up->copy(gated + (2 * row + 128) * row_bytes, raise.data + row * row_bytes, bytes));
  }
  return up->copy_rows(down, b.inner_columns() * 2, lower.data, inner_bytes, inner_bytes, width);
}

int upload_kikepel_block(const ModelFile &file, const ModelConfig &c, const std::size_t layer, WeightUploader *up,
                         LayerWeights *w) {
  const DecoderBlock &b = c.blocks[layer];
  for (const ExpectedTensor &e : kikepel_block_tensors(c, layer)) {
    const TensorView *view = nullptr;
    EVOB_TRY(lookup_tensor(file, e, &view));
    w->payload_bytes += view->bytes;
  }
  const std::string l = "l" + std::to_string(layer) + ".", p = l + "mix.", m = l + "mlp.";
  const auto view = [&file](const std::string &name) -> const TensorView & { return *file.find(name); };
  const std::size_t D = c.width;
  w->type = b.mixer;
  EVOB_TRY(up->floats(widened(view(l + "norm1")), &w->pre_norm));
  unsigned char *fused = nullptr;
  EVOB_TRY(up->zeros(b.projection_width() * D * 2, &fused));
  w->projection = fused;
  EVOB_TRY(up->copy(fused, view(p + "dq").data, view(p + "dq").bytes));
  EVOB_TRY(up->copy(up->dry_run ? nullptr : fused + b.latent_column() * D * 2, view(p + "dkv").data, view(p + "dkv").bytes));
  EVOB_TRY(up->floats(widened(view(p + "dq.norm")), &w->query_norm));
  EVOB_TRY(up->floats(widened(view(p + "dkv.norm")), &w->key_norm));
  EVOB_TRY(up->tensor(view(p + "uq"), &w->query_up));
  EVOB_TRY(up->tensor(view(p + "uk"), &w->key_up));
  EVOB_TRY(up->tensor(view(p + "uv"), &w->value_up));
  EVOB_TRY(up->tensor(view(p + "o"), &w->out_weight));
  if (b.sink) EVOB_TRY(up->floats(widened(view(p + "sink")), &w->sink_logit));
  if (b.feed_forward == FeedForward::kNone) return kOk;
  EVOB_TRY(up->floats(widened(view(l + "norm2")), &w->post_norm));
  const std::size_t columns = b.inner_columns(), gated_bytes = 2 * columns * D * 2, down_bytes = D * columns * 2;
  const std::size_t copies = b.feed_forward == FeedForward::kExperts ? b.experts : 1;
  unsigned char *gated = nullptr, *down = nullptr;
  EVOB_TRY(up->zeros(copies * gated_bytes, &gated));
  EVOB_TRY(up->zeros(copies * down_bytes, &down));
  w->l12 = gated;
  w->l3 = down;
  if (b.feed_forward == FeedForward::kReluGated) {
    EVOB_TRY(place_gated(up, b, D, view(m + "gate"), view(m + "up"), view(m + "down"), gated, down));
    const std::vector<float> gate_bias = widened(view(m + "gate.b")), up_bias = widened(view(m + "up.b"));
    std::vector<float> both(2 * columns, 0.0F);
    for (std::size_t i = 0; i < b.inner_width; ++i) {
      both[i / 128 * 256 + i % 128] = gate_bias[i];
      both[i / 128 * 256 + 128 + i % 128] = up_bias[i];
    }
    EVOB_TRY(up->floats(std::move(both), &w->l12_bias));
    return up->floats(widened(view(m + "down.b")), &w->l3_bias);
  }
  unsigned char *router = nullptr;
  EVOB_TRY(up->zeros(b.router_rows() * D * 2, &router));
  w->router = router;
  EVOB_TRY(up->copy(router, view(m + "router").data, view(m + "router").bytes));
  for (std::size_t e = 0; e < b.experts; ++e) {
    const std::string x = m + "e" + std::to_string(e) + ".";
    EVOB_TRY(place_gated(up, b, D, view(x + "gate"), view(x + "up"), view(x + "down"),
                         up->dry_run ? nullptr : gated + e * gated_bytes, up->dry_run ? nullptr : down + e * down_bytes));
  }
  return kOk;
}

}  // namespace

const DecoderDesign kKikepelDesign = {"Kikepel",          read_kikepel_config,  kikepel_model_tensors, kikepel_block_tensors,
                                      upload_kikepel_model, upload_kikepel_block};

}  // namespace evob
