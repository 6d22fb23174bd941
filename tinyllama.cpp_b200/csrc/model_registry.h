// Model registry: which architectures the engine serves, and the description of a block model (a stack of layers that
// differ in mixer and feed-forward) as its config.json gives it. Host code only.
//
//   llama    GGUF file, packed Q8_0 / Q4_K / Q6_K weights (b200_engine_load_gguf)
//   Nezolix  folder with config.json + model.safetensors: layers with a latent-attention or a WKV mixer, normalised
//            before and after each sublayer, optionally with a stretch of layers that runs several times
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

enum class MixerKind { LatentAttention, Wkv };

struct MixerSpec {
  MixerKind kind = MixerKind::LatentAttention;
  int heads = 0, dim = 0;                         // wkv: state dim x dim per head; latent attention: unrotated dimensions
  int rot_dim = 0, vdim = 0, q_rank = 0, kv_rank = 0;  // latent attention
  int window = 0;                                 // keys a query sees (itself included); 0 = all earlier ones
  double scale = 1.0;
  RotSpec rot;
  int decay_rank = 0;                             // wkv: inner size of the decay's two-matrix product
};

struct LayerSpec {
  MixerSpec mix;
  int ff = 0;  // inner size of the gated feed-forward, 0 = the layer has none
};

struct BlockSpec {
  std::string arch;
  int vocab = 0, width = 0;
  double eps = 1e-6, embed_scale = 1.0;
  std::vector<LayerSpec> layers;
  int loop_start = 0, loop_stop = 0, loop_times = 1;
  std::vector<int> runs() const;  // layer index of every layer run, in order
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
