#include "model_registry.h"

#include <algorithm>
#include <cmath>
#include <fstream>
#include <sstream>
#include <stdexcept>

namespace b200 {

std::vector<double> rot_frequencies(const RotSpec& r, double* amplitude) {
  const int n = r.dims / 2;
  std::vector<double> f(n);
  for (int i = 0; i < n; ++i) f[i] = std::pow(r.base, -2.0 * i / r.dims);
  *amplitude = 1.0;
  if (r.yarn) {
    const double pi = 3.14159265358979323846;
    // the (fractional) pair index whose wavelength fits `turns` turns into the original context
    auto where = [&](double turns) { return r.dims * std::log(r.original / (2.0 * pi * turns)) / (2.0 * std::log(r.base)); };
    const double lo = std::max(std::floor(where(r.fast)), 0.0), hi = std::min(std::ceil(where(r.slow)), (double)r.dims - 1.0);
    const double span = std::max(hi - lo, 0.001);
    for (int i = 0; i < n; ++i) {
      const double ramp = std::min(std::max((i - lo) / span, 0.0), 1.0);
      f[i] = f[i] / r.factor * ramp + f[i] * (1.0 - ramp);
    }
    *amplitude = 0.1 * std::log(r.factor) + 1.0;
  }
  return f;
}

std::vector<int> BlockSpec::runs() const {
  std::vector<int> out;
  for (int i = 0; i < loop_start; ++i) out.push_back(i);
  for (int t = 0; t < loop_times; ++t)
    for (int i = loop_start; i < loop_stop; ++i) out.push_back(i);
  for (int i = loop_stop; i < (int)layers.size(); ++i) out.push_back(i);
  return out;
}

bool BlockSpec::begins_further_pass(int run) const {
  const int n = loop_stop - loop_start, at = run - loop_start;
  return n > 0 && at > 0 && at < n * loop_times && at % n == 0;
}

std::vector<TensorNeed> block_tensor_needs(const BlockSpec& s) {
  std::vector<TensorNeed> out;
  const int64_t W = s.width;
  out.push_back({"embed", {s.vocab, W}});
  for (size_t l = 0; l < s.layers.size(); ++l) {
    const LayerSpec& y = s.layers[l];
    const MixerSpec& m = y.mix;
    const std::string L = "l" + std::to_string(l) + ".";
    out.push_back({L + "norm1", {W}});
    if (s.post_norm) out.push_back({L + "norm1b", {W}});
    const int64_t H = m.heads, D = m.dim;
    if (m.kind == MixerKind::LatentAttention) {
      out.push_back({L + "mix.dq", {m.q_rank, W}});
      out.push_back({L + "mix.dq.norm", {m.q_rank}});
      out.push_back({L + "mix.uq", {H * (D + m.rot_dim), m.q_rank}});
      out.push_back({L + "mix.dkv", {(int64_t)m.kv_rank + m.rot_dim, W}});
      out.push_back({L + "mix.dkv.norm", {m.kv_rank}});
      out.push_back({L + "mix.uk", {H * D, m.kv_rank}});
      out.push_back({L + "mix.uv", {H * m.vdim, m.kv_rank}});
      out.push_back({L + "mix.g", {H * m.vdim, W}});
      out.push_back({L + "mix.o", {W, H * m.vdim}});
    } else if (m.kind == MixerKind::SharedKvAttention) {
      out.push_back({L + "mix.q", {H * D, W}});
      out.push_back({L + "mix.k", {m.kv_heads * D, W}});
      out.push_back({L + "mix.o", {W, H * D}});
    } else if (m.kind == MixerKind::RgLru) {
      const int64_t N = m.width, B = m.blocks, S = N / B;
      for (const char* k : {"y", "x"}) {
        out.push_back({L + "mix." + k, {N, W}});
        out.push_back({L + "mix." + k + ".b", {N}});
      }
      out.push_back({L + "mix.conv", {N, m.conv}});
      out.push_back({L + "mix.conv.b", {N}});
      for (const char* k : {"ra", "ri"}) {
        out.push_back({L + "mix." + k, {B, S, S}});
        out.push_back({L + "mix." + k + ".b", {B, S}});
      }
      out.push_back({L + "mix.lam", {N}});
      out.push_back({L + "mix.o", {W, N}});
    } else {
      for (const char* k : {"r", "k", "v", "g", "w"}) out.push_back({L + "mix.mu." + k, {W}});
      for (const char* k : {"r", "k", "v", "g"}) out.push_back({L + "mix." + k, {H * D, W}});
      out.push_back({L + "mix.w1", {m.decay_rank, W}});
      out.push_back({L + "mix.w2", {H * D, m.decay_rank}});
      out.push_back({L + "mix.w0", {H * D}});
      out.push_back({L + "mix.u", {H, D}});
      out.push_back({L + "mix.norm", {H * D}});
      out.push_back({L + "mix.o", {W, H * D}});
    }
    if (y.ff) {
      out.push_back({L + "norm2", {W}});
      if (s.post_norm) out.push_back({L + "norm2b", {W}});
      out.push_back({L + "mlp.gate", {y.ff, W}});
      out.push_back({L + "mlp.up", {y.ff, W}});
      out.push_back({L + "mlp.down", {W, y.ff}});
    }
  }
  out.push_back({"final.norm", {W}});
  if (!s.tied_head) out.push_back({"head", {s.vocab, W}});
  return out;
}

static int positive(const Json& j, const char* key) {
  const int v = j.integer(key);
  if (v <= 0) throw std::runtime_error(std::string("field '") + key + "' must be positive");
  return v;
}

static RotSpec read_rot(const Json& j) {
  RotSpec r;
  r.dims = j.integer("dims");
  r.base = j.number("base");
  if (r.dims < 0 || r.dims % 2) throw std::runtime_error("rot.dims must be even");
  if (const Json* s = j.find("scaling")) {
    r.yarn = true;
    r.factor = s->number("factor");
    r.original = s->number("original");
    r.fast = s->number("fast");
    r.slow = s->number("slow");
  }
  return r;
}

static MixerSpec read_latent_attention(const Json& j) {
  MixerSpec m;
  m.kind = MixerKind::LatentAttention;
  m.heads = positive(j, "heads");
  m.dim = positive(j, "dim");
  m.rot_dim = positive(j, "rot_dim");
  m.vdim = positive(j, "vdim");
  m.q_rank = positive(j, "q_rank");
  m.kv_rank = positive(j, "kv_rank");
  m.scale = j.number("scale");
  if (const Json* r = j.find("rot")) m.rot = read_rot(*r);
  if (m.rot.dims > m.rot_dim) throw std::runtime_error("rot.dims exceeds rot_dim");
  if (const Json* k = j.find("mask"))
    if (k->find("size")) m.mask.size = positive(*k, "size");
  return m;
}

static MixerSpec read_shared_kv_attention(const Json& j) {
  MixerSpec m;
  m.kind = MixerKind::SharedKvAttention;
  m.heads = positive(j, "heads");
  m.kv_heads = positive(j, "kv_heads");
  m.dim = m.vdim = positive(j, "dim");
  m.sink = true;
  m.scale = j.number("scale");
  if (j.find("softcap")) m.softcap = j.number("softcap");
  if (m.heads % m.kv_heads) throw std::runtime_error("heads must be a multiple of kv_heads");
  if (j.find("vdim") && j.integer("vdim") != m.dim) throw std::runtime_error("vdim must equal dim: the values are the keys");
  if (m.softcap < 0) throw std::runtime_error("softcap must be positive");
  if (const Json* r = j.find("rot")) m.rot = read_rot(*r);
  if (m.rot.dims > m.dim) throw std::runtime_error("rot.dims exceeds dim");
  if (const Json* k = j.find("mask"))
    if (k->find("size")) m.mask = {positive(*k, "size"), true};
  return m;
}

static MixerSpec read_rglru(const Json& j) {
  MixerSpec m;
  m.kind = MixerKind::RgLru;
  m.width = positive(j, "width");
  m.blocks = positive(j, "blocks");
  m.conv = positive(j, "conv");
  if (m.width % m.blocks) throw std::runtime_error("width must be a multiple of blocks");
  return m;
}

// What the block architectures' config.json files share: sizes, the layer list (mixer: type, entry, layer index -> its
// description) and the loop.
template <typename Mixer>
static BlockSpec read_stack(const Json& c, GluKind glu, Mixer mixer) {
  BlockSpec s;
  s.arch = c.text("architecture");
  s.vocab = positive(c, "vocab");
  s.width = positive(c, "width");
  s.eps = c.at("norm").number("eps");
  const Json& layers = c.at("layers");
  if (layers.kind != Json::Array || layers.items.empty()) throw std::runtime_error("'layers' must be a non-empty list");
  for (size_t l = 0; l < layers.items.size(); ++l) {
    const Json& e = layers.items[l];
    const std::string where = "layer " + std::to_string(l) + ": ";
    LayerSpec y;
    if (!mixer(e.text("type"), e.at("mixer"), l, y.mix)) throw std::runtime_error(where + "unknown mixer '" + e.text("type") + "'");
    if (const Json* f = e.find("mlp")) {
      if (f->text("kind") != "dense") throw std::runtime_error(where + "unknown feed-forward '" + f->text("kind") + "'");
      y.ff = positive(*f, "ff");
      y.glu = glu;
    }
    s.layers.push_back(y);
  }
  s.loop_stop = (int)s.layers.size();
  if (const Json* lp = c.find("loop")) {
    s.loop_start = lp->integer("start");
    s.loop_stop = lp->integer("stop");
    s.loop_times = positive(*lp, "times");
    if (s.loop_start < 0 || s.loop_stop < s.loop_start || s.loop_stop > (int)s.layers.size()) throw std::runtime_error("'loop' lies outside the layers");
  }
  return s;
}

static BlockSpec read_nezolix(const Json& c, const StFile& weights) {
  BlockSpec s = read_stack(c, GluKind::Relu, [&](const std::string& type, const Json& j, size_t l, MixerSpec& m) {
    if (type == "latent_attention") {
      m = read_latent_attention(j);
    } else if (type == "wkv") {
      m.kind = MixerKind::Wkv;
      m.heads = positive(j, "heads");
      m.dim = positive(j, "dim");
      const auto it = weights.tensors.find("l" + std::to_string(l) + ".mix.w1");
      if (it == weights.tensors.end() || it->second.shape.size() != 2 || it->second.shape[0] < 1)
        throw std::runtime_error("layer " + std::to_string(l) + ": decay matrix w1 is missing");
      m.decay_rank = (int)it->second.shape[0];
    } else {
      return false;
    }
    return true;
  });
  if (const Json* e = c.find("embedding"))
    if (e->find("scale")) s.embed_scale = e->number("scale");
  return s;
}

static BlockSpec read_pizilix(const Json& c, const StFile&) {
  BlockSpec s = read_stack(c, GluKind::Silu, [](const std::string& type, const Json& j, size_t, MixerSpec& m) {
    if (type == "attention") m = read_shared_kv_attention(j);
    else if (type == "rglru") m = read_rglru(j);
    else return false;
    return true;
  });
  s.post_norm = false;
  s.norm_offset = 1.0;
  s.tied_head = true;
  s.loop_adds_embedding = true;
  if (c.find("logit_softcap")) s.logit_softcap = c.number("logit_softcap");
  if (s.logit_softcap < 0) throw std::runtime_error("logit_softcap must be positive");
  return s;
}

static const ArchEntry ARCHS[] = {
    {"llama", true, nullptr},
    {"Nezolix", false, read_nezolix},
    {"Pizilix", false, read_pizilix},
};

const ArchEntry* find_arch(const std::string& name) {
  for (const ArchEntry& a : ARCHS)
    if (name == a.name) return &a;
  return nullptr;
}

std::string known_archs() {
  std::string s;
  for (const ArchEntry& a : ARCHS) s += (s.empty() ? "" : ", ") + std::string(a.name);
  return s;
}

BlockSpec read_model_folder(const std::string& folder, StFile& weights) {
  std::ifstream f(folder + "/config.json", std::ios::binary);
  if (!f) throw std::runtime_error("cannot open " + folder + "/config.json");
  std::stringstream ss;
  ss << f.rdbuf();
  const std::string text = ss.str();
  const Json config = json_parse(text.data(), text.size());
  const std::string& arch = config.text("architecture");
  const ArchEntry* a = find_arch(arch);
  if (!a || !a->read) throw std::runtime_error("unknown architecture '" + arch + "' (known: " + known_archs() + ")");
  safetensors_open(folder + "/model.safetensors", weights);
  BlockSpec s = a->read(config, weights);
  for (const TensorNeed& n : block_tensor_needs(s)) {
    const auto it = weights.tensors.find(n.name);
    if (it == weights.tensors.end()) throw std::runtime_error("tensor " + n.name + " is missing");
    if (it->second.dtype != "BF16") throw std::runtime_error("tensor " + n.name + " must be BF16");
    if (it->second.shape != n.shape) throw std::runtime_error("tensor " + n.name + " has an unexpected shape");
  }
  return s;
}

}  // namespace b200
