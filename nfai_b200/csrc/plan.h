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

// Grouped-query attention over cached keys and values. Projected row [q | k | v | gate]; a layer that borrows (kv_from)
// has [q | gate] and reads the cache rows of an earlier layer.
struct GqaSpec {
  uint32_t heads = 0, kv_heads = 0, dim = 0, vdim = 0;
  int kv_from = -1;             // layer whose keys and values are used; -1: its own
  float scale = 0.f;
  bool qk_norm = false;         // every query and key head over its root mean square before the score
  bool v_norm = false;          // every value head over its root mean square before it is cached
  bool distance_bias = false;   // score -= 2^(-8 (h+1) / heads) * (distance to the key)
  bool head_gate = false;       // head h's output times the sigmoid of its gate row
  constexpr bool own_kv() const { return kv_from < 0; }
  constexpr uint32_t q_rows() const { return heads * dim; }
  constexpr uint32_t k_cols() const { return kv_heads * dim; }
  constexpr uint32_t v_cols() const { return kv_heads * vdim; }
  constexpr uint32_t kv_rows() const { return own_kv() ? k_cols() + v_cols() : 0; }
  constexpr uint32_t gate_row0() const { return q_rows() + kv_rows(); }
  constexpr uint32_t in_rows() const { return gate_row0() + (head_gate ? heads : 0); }
  constexpr uint32_t out_cols() const { return heads * vdim; }
};

// Routed feed-forward: `top` of `experts` small gated feed-forwards per token, chosen among the best `keep` of `groups`
// equal groups by sigmoid scores plus a correction, weighted by the scores alone; optionally a shared one for every token,
// times the sigmoid of one number.
struct MoeSpec {
  uint32_t experts = 0, top = 0, ff = 0, groups = 1, keep = 1;
  float limit = 0.f, scale = 1.f;
  uint32_t shared_ff = 0;  // 0: no shared feed-forward
  float shared_limit = 0.f;
  // The first product of a routed layer: [shared gate, up interleaved | router | shared's own gate | padding to even]
  constexpr uint32_t gated_rows() const { return 2 * shared_ff; }
  constexpr uint32_t tail_rows() const { return experts + (shared_ff ? 1u : 0u); }
  constexpr uint32_t first_rows() const { return (gated_rows() + tail_rows() + 1u) & ~1u; }
  // hidden values of one token: those of the chosen experts in the order of choice, then the shared ones
  constexpr uint32_t hidden() const { return top * ff + shared_ff; }
};
constexpr uint32_t kMaxExperts = 1024, kMaxChosen = 32, kMaxGroups = 64;

enum MixerKind { MIXER_LATENT = 0, MIXER_SSM = 1, MIXER_GQA = 2 };
enum FeedForwardKind { FF_NONE = 0, FF_DENSE = 1, FF_MOE = 2 };
// How a sublayer's output meets the residual: written into several streams (hyper-connections, the sublayer reads a normed
// combination of them), or x += mult * norm(y) with the sublayer reading x itself.
enum ResidualKind { RESIDUAL_STREAMS = 0, RESIDUAL_POST_NORM = 1 };

struct PlanLayer {
  MixerKind mixer = MIXER_LATENT;
  LatentSpec latent;
  SsmSpec ssm;
  GqaSpec gqa;
  FeedForwardKind mlp = FF_NONE;
  uint32_t ff = 0;    // FF_DENSE
  float limit = 0.f;  // FF_DENSE with a clamped activation
  MoeSpec moe;        // FF_MOE
  bool has_mlp() const { return mlp != FF_NONE; }
  uint32_t in_rows() const { return mixer == MIXER_LATENT ? latent.in_rows() : mixer == MIXER_SSM ? ssm.in_rows() : gqa.in_rows(); }
  uint32_t out_cols() const { return mixer == MIXER_LATENT ? latent.gate_rows() : mixer == MIXER_SSM ? ssm.inner() : gqa.out_cols(); }
};

struct LayerPlan {
  std::string architecture;
  uint32_t width = 0, vocab = 0, streams = 1;
  float eps = 0.f;
  int act = 0;  // Activation of the gated feed-forwards
  bool mixer_bias = false;  // biases of the q, k, v and output projections (GQA)
  bool ff_bias = false;     // biases of dense feed-forwards
  ResidualKind residual = RESIDUAL_STREAMS;
  float residual_mult = 1.f;  // RESIDUAL_POST_NORM
  bool scalar_norms = false;  // norms have one gain for all coordinates
  float sinusoid_base = 0.f;  // > 0: a sinusoidal position vector is added to the embedding
  std::vector<PlanLayer> layers;
  uint32_t sublayers() const {
    uint32_t n = 0;
    for (const PlanLayer& l : layers) n += l.has_mlp() ? 2 : 1;
    return n;
  }
};

// One tensor the plan needs: shape outermost first (as the file lists it), empty for a single number.
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
