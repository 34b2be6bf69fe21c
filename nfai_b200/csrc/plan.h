// Layer plans (internal): models whose layers are listed in a configuration file, each layer with a mixer of its own
// kind and size and an optional feed-forward. The plan says what to compute and which tensors belong to it; it knows
// nothing about devices.
#pragma once
#include <stdint.h>

#include <string>
#include <vector>

namespace nfai {

// Attention over latents: per position one latent c (RMS-normed, `rank` wide) and one rotated key part shared by all
// heads are kept; per-head keys and values are linear maps of c. Sliding window over the last `window` positions.
struct LatentSpec {
  uint32_t heads = 0, dim = 0, rot = 0, vdim = 0, rank = 0;
  uint32_t rope_dims = 0;  // rotated prefix of the `rot` part
  uint32_t window = 0;     // 0: all earlier positions
  float scale = 0.f, rope_base = 0.f;
  constexpr uint32_t q_rows() const { return heads * (dim + rot); }
  constexpr uint32_t kv_rows() const { return rank + rot; }
  constexpr uint32_t gate_rows() const { return heads * vdim; }
  constexpr uint32_t in_rows() const { return q_rows() + kv_rows() + gate_rows(); }
};

// Selective state space layer with a scalar decay per head (Mamba-2): [z | x | B | C | dt] projection, short causal
// convolution over [x | B | C], state [vdim][state] per head in float32.
struct SsmSpec {
  uint32_t heads = 0, vdim = 0, state = 0, groups = 1, taps = 1, norm_groups = 1;
  constexpr uint32_t inner() const { return heads * vdim; }
  constexpr uint32_t channels() const { return inner() + 2 * groups * state; }
  constexpr uint32_t in_rows() const { return inner() + channels() + heads; }
};

enum MixerKind { MIXER_LATENT = 0, MIXER_SSM = 1 };

struct PlanLayer {
  MixerKind mixer = MIXER_LATENT;
  LatentSpec latent;
  SsmSpec ssm;
  bool has_mlp = false;
  uint32_t ff = 0;
  uint32_t in_rows() const { return mixer == MIXER_LATENT ? latent.in_rows() : ssm.in_rows(); }
  uint32_t out_cols() const { return mixer == MIXER_LATENT ? latent.gate_rows() : ssm.inner(); }
};

struct LayerPlan {
  std::string architecture;
  uint32_t width = 0, vocab = 0, streams = 1;
  float eps = 0.f;
  int act = 0;  // Activation of the gated feed-forward
  std::vector<PlanLayer> layers;
  uint32_t sublayers() const {
    uint32_t n = 0;
    for (const PlanLayer& l : layers) n += l.has_mlp ? 2 : 1;
    return n;
  }
};

// One tensor the plan needs: shape outermost first (as the file lists it).
struct PlanTensor {
  std::string name;
  std::vector<uint64_t> shape;
};

// Architectures that are described by a configuration with a layer list: name in "architecture" -> reader.
bool plan_architecture_known(const std::string& name);
// Read config.json. False: *err says why (unknown architecture, missing key, size that does not fit).
bool plan_parse(const char* json, size_t len, LayerPlan* out, std::string* err);
std::vector<PlanTensor> plan_tensors(const LayerPlan& plan);

}  // namespace nfai
