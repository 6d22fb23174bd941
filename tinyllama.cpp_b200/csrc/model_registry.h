// Model registry: which architectures the engine serves, and the description of a block model (a stack of layers that
// differ in mixer and feed-forward) as its config.json gives it. Host code only.
//
//   llama    GGUF file, packed Q8_0 / Q4_K / Q6_K weights (b200_engine_load_gguf)
//   Nezolix  folder with config.json + model.safetensors: layers with a latent-attention or a WKV mixer, normalised
//            before and after each sublayer, optionally with a stretch of layers that runs several times
//   Pizilix  the same kind of folder: layers with an attention mixer whose values are its keys (chunked mask, capped scores,
//            sink) or a gated linear recurrence (RG-LRU) with a short convolution, normalised before each sublayer; a
//            looped stretch gets the embedding added again before every further pass; tied, capped head
//
// A new block architecture adds a row to the table in model_registry.cpp with the function that reads its config.json
// into a BlockSpec; the mixers, feed-forwards and norms below take every constant from that description.
#pragma once
#include <string>
#include <vector>

#include "json.h"
#include "safetensors.h"

namespace b200 {

// Rotary positions over the first `dims` dimensions of a vector, pairs (2i, 2i+1), frequency base^(-2i/dims); with
// `yarn`, the frequencies are interpolated between f and f / factor and cos / sin are multiplied by 0.1 ln(factor) + 1.
struct RotSpec {
  int dims = 0;
  double base = 10000.0;
  bool yarn = false;
  double factor = 1.0, original = 0.0, fast = 32.0, slow = 1.0;
  bool operator==(const RotSpec& o) const {
    return dims == o.dims && base == o.base && yarn == o.yarn && factor == o.factor && original == o.original && fast == o.fast && slow == o.slow;
  }
};
// Frequencies [dims / 2] and the factor on cos and sin.
std::vector<double> rot_frequencies(const RotSpec& r, double* amplitude);

enum class MixerKind { LatentAttention, Wkv, SharedKvAttention, RgLru };

// Which earlier keys a query at position p sees (besides its own): all of them (size 0), those of the last `size` positions,
// or, chunked, those of its own block of `size` positions counted from position 0.
struct MaskSpec {
  int size = 0;
  bool chunked = false;
  bool operator==(const MaskSpec& o) const { return size == o.size && chunked == o.chunked; }
};

struct MixerSpec {
  MixerKind kind = MixerKind::LatentAttention;
  int heads = 0, dim = 0;                         // wkv: state dim x dim per head; latent attention: unrotated dimensions
  int rot_dim = 0, vdim = 0, q_rank = 0, kv_rank = 0;  // latent attention
  int kv_heads = 0;                               // shared-kv attention: key / value heads
  MaskSpec mask;
  double scale = 1.0;
  double softcap = 0.0;                           // shared-kv attention: scores become cap * tanh(score / cap); 0 = left as they are
  bool sink = false;                              // shared-kv attention: one more term exp(0) in the softmax denominator
  RotSpec rot;
  int decay_rank = 0;                             // wkv: inner size of the decay's two-matrix product
  int width = 0, blocks = 0, conv = 0;            // rg-lru: channels, blocks of the gate matrices, taps of the convolution
};

enum class GluKind { Relu, Silu };

struct LayerSpec {
  MixerSpec mix;
  int ff = 0;  // inner size of the gated feed-forward, 0 = the layer has none
  GluKind glu = GluKind::Relu;
};

struct BlockSpec {
  std::string arch;
  int vocab = 0, width = 0;
  double eps = 1e-6, embed_scale = 1.0;
  std::vector<LayerSpec> layers;
  int loop_start = 0, loop_stop = 0, loop_times = 1;
  bool loop_adds_embedding = false;  // the embedding output is added to the stream before every pass but the first
  bool post_norm = true;             // sublayer outputs are normalised before they are added
  double norm_offset = 0.0;          // added to every stored norm weight
  bool tied_head = false;            // the embedding table is the head
  double logit_softcap = 0.0;        // logits become cap * tanh(logit / cap); 0 = left as they are
  std::vector<int> runs() const;  // layer index of every layer run, in order
  bool begins_further_pass(int run) const;  // run opens a pass of the loop that is not the first
};

struct TensorNeed {
  std::string name;
  std::vector<int64_t> shape;
};
// Every tensor the model needs, with its shape.
std::vector<TensorNeed> block_tensor_needs(const BlockSpec& s);

struct ArchEntry {
  const char* name;
  bool gguf;                                            // weights and configuration come from a GGUF file
  BlockSpec (*read)(const Json& config, const StFile& weights);  // block models; nullptr for GGUF
};
const ArchEntry* find_arch(const std::string& name);
std::string known_archs();

// Reads folder/config.json and opens folder/model.safetensors; checks that every needed tensor is there in bfloat16 with
// the right shape. Throws std::runtime_error with the reason otherwise.
BlockSpec read_model_folder(const std::string& folder, StFile& weights);

}  // namespace b200
