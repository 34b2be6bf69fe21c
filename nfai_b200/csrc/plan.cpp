// config.json -> LayerPlan, and the tensors a plan needs. Host code only; every number of the file is checked before it
// is used as a size.
#include "plan.h"

#include <math.h>
#include <stdio.h>

#include <algorithm>

#include "json.h"

namespace nfai {

namespace {

struct Fail {
  std::string* err;
  bool operator()(const std::string& m) const {
    if (err && err->empty()) *err = m;
    return false;
  }
};

// A positive integer below 2^24 (products of two stay far inside 64 bits; sizes of rows are checked again below).
bool size_of(const Json* obj, const char* key, const std::string& where, uint32_t* out, const Fail& fail) {
  const Json* v = obj ? obj->get(key) : nullptr;
  if (!v || v->kind != Json::Number) return fail(where + ": missing number '" + key + "'");
  if (!(v->num >= 1 && v->num < 16777216.0) || v->num != floor(v->num))
    return fail(where + ": '" + key + "' must be a positive integer");
  *out = (uint32_t)v->num;
  return true;
}

bool real_of(const Json* obj, const char* key, const std::string& where, float* out, const Fail& fail) {
  const Json* v = obj ? obj->get(key) : nullptr;
  if (!v || v->kind != Json::Number) return fail(where + ": missing number '" + key + "'");
  *out = (float)v->num;
  return true;
}

bool read_latent(const Json* m, const std::string& w, LatentSpec* s, const Fail& fail) {
  if (!size_of(m, "heads", w, &s->heads, fail) || !size_of(m, "dim", w, &s->dim, fail) || !size_of(m, "rot_dim", w, &s->rot, fail) ||
      !size_of(m, "vdim", w, &s->vdim, fail) || !size_of(m, "kv_rank", w, &s->rank, fail) || !real_of(m, "scale", w, &s->scale, fail))
    return false;
  const Json* rot = m->get("rot");
  if (!size_of(rot, "dims", w + ".rot", &s->rope_dims, fail) || !real_of(rot, "base", w + ".rot", &s->rope_base, fail)) return false;
  if (s->rope_dims > s->rot || (s->rope_dims & 1)) return fail(w + ": rot.dims must be even and at most rot_dim");
  if (!(s->rope_base > 0.f)) return fail(w + ": rot.base must be positive");
  const Json* mask = m->get("mask");
  if (mask && !mask->is_null() && !size_of(mask, "size", w + ".mask", &s->window, fail)) return false;
  return true;
}

bool read_ssm(const Json* m, const std::string& w, SsmSpec* s, const Fail& fail) {
  if (!size_of(m, "heads", w, &s->heads, fail) || !size_of(m, "vdim", w, &s->vdim, fail) || !size_of(m, "state", w, &s->state, fail) ||
      !size_of(m, "groups", w, &s->groups, fail) || !size_of(m, "conv", w, &s->taps, fail) ||
      !size_of(m, "norm_groups", w, &s->norm_groups, fail))
    return false;
  if (s->heads % s->groups) return fail(w + ": heads must be a multiple of groups");
  if ((uint64_t)s->heads * s->vdim % s->norm_groups) return fail(w + ": heads * vdim must be a multiple of norm_groups");
  return true;
}

// Tometar: hyper-connected streams, latent attention and Mamba-2 layers in any order, relu-gated feed-forwards with
// biases, untied output matrix.
bool read_tometar(const Json& root, LayerPlan* p, const Fail& fail) {
  if (!size_of(&root, "width", "config", &p->width, fail) || !size_of(&root, "vocab", "config", &p->vocab, fail) ||
      !size_of(&root, "streams", "config", &p->streams, fail) || !real_of(root.get("norm"), "eps", "config.norm", &p->eps, fail))
    return false;
  if (p->streams > 16) return fail("config: at most 16 streams");
  if (!(p->eps >= 0.f)) return fail("config.norm: eps must not be negative");
  p->act = 1;  // relu
  p->ff_bias = true;
  const Json* layers = root.get("layers");
  if (!layers || layers->kind != Json::Array || layers->items.empty()) return fail("config: 'layers' must be a non-empty list");
  if (layers->items.size() > 4096) return fail("config: too many layers");
  for (size_t i = 0; i < layers->items.size(); ++i) {
    const Json& l = layers->items[i];
    const std::string w = "config.layers[" + std::to_string(i) + "]";
    const Json* type = l.get("type");
    const Json* mixer = l.get("mixer");
    if (!type || type->kind != Json::String || !mixer || mixer->kind != Json::Object) return fail(w + ": 'type' and 'mixer' are needed");
    PlanLayer pl;
    if (type->str == "latent_attention") {
      pl.mixer = MIXER_LATENT;
      if (!read_latent(mixer, w + ".mixer", &pl.latent, fail)) return false;
    } else if (type->str == "mamba2") {
      pl.mixer = MIXER_SSM;
      if (!read_ssm(mixer, w + ".mixer", &pl.ssm, fail)) return false;
    } else {
      return fail(w + ": unknown layer type '" + type->str + "'");
    }
    const Json* mlp = l.get("mlp");
    if (mlp && !mlp->is_null()) {
      const Json* kind = mlp->get("kind");
      if (!kind || kind->kind != Json::String || kind->str != "dense") return fail(w + ".mlp: unknown kind of feed-forward");
      if (!size_of(mlp, "ff", w + ".mlp", &pl.ff, fail)) return false;
      pl.mlp = FF_DENSE;
    }
    p->layers.push_back(pl);
  }
  return true;
}

bool read_gqa(const Json* m, const std::string& w, size_t layer, const LayerPlan& p, GqaSpec* s, const Fail& fail) {
  if (!size_of(m, "heads", w, &s->heads, fail) || !size_of(m, "kv_heads", w, &s->kv_heads, fail) || !size_of(m, "dim", w, &s->dim, fail) ||
      !size_of(m, "vdim", w, &s->vdim, fail) || !real_of(m, "scale", w, &s->scale, fail))
    return false;
  if (s->heads % s->kv_heads) return fail(w + ": heads must be a multiple of kv_heads");
  const Json* from = m->get("kv_from");
  if (from && !from->is_null()) {
    if (from->kind != Json::Number || !(from->num >= 0 && from->num < (double)layer) || from->num != floor(from->num))
      return fail(w + ": 'kv_from' must name an earlier layer");
    s->kv_from = (int)from->num;
    const PlanLayer& src = p.layers[(size_t)s->kv_from];
    if (src.mixer != MIXER_GQA || !src.gqa.own_kv()) return fail(w + ": 'kv_from' must name a layer with keys and values of its own");
    if (src.gqa.kv_heads != s->kv_heads || src.gqa.dim != s->dim || src.gqa.vdim != s->vdim)
      return fail(w + ": the key and value heads of layer " + std::to_string(s->kv_from) + " differ");
  }
  return true;
}

bool read_moe(const Json* m, const std::string& w, MoeSpec* s, const Fail& fail) {
  const Json *expert = m->get("expert"), *router = m->get("router"), *shared = m->get("shared");
  if (!size_of(expert, "ff", w + ".expert", &s->ff, fail) || !real_of(expert, "limit", w + ".expert", &s->limit, fail) ||
      !size_of(router, "experts", w + ".router", &s->experts, fail) || !size_of(router, "top", w + ".router", &s->top, fail) ||
      !real_of(router, "scale", w + ".router", &s->scale, fail))
    return false;
  const Json* groups = router->get("groups");
  if (groups && !groups->is_null() &&
      (!size_of(groups, "count", w + ".router.groups", &s->groups, fail) || !size_of(groups, "keep", w + ".router.groups", &s->keep, fail)))
    return false;
  if (s->experts > kMaxExperts || s->top > kMaxChosen || s->groups > kMaxGroups)
    return fail(w + ": at most " + std::to_string(kMaxExperts) + " experts, " + std::to_string(kMaxChosen) + " of them chosen, in " +
                std::to_string(kMaxGroups) + " groups");
  if (s->experts % s->groups || s->keep > s->groups) return fail(w + ".router: groups must be equal parts, and no more kept than there are");
  if (s->top > s->keep * (s->experts / s->groups)) return fail(w + ".router: the kept groups hold fewer than 'top' experts");
  if (shared && !shared->is_null() &&
      (!size_of(shared, "ff", w + ".shared", &s->shared_ff, fail) || !real_of(shared, "limit", w + ".shared", &s->shared_limit, fail)))
    return false;
  return true;
}

// Tutizen: sinusoidal positions, x += m * norm(sublayer(x)) with one gain per norm, grouped-query attention with head norms,
// distance bias, head gates and keys and values borrowed from earlier layers, clamped gated feed-forwards, dense or routed.
bool read_tutizen(const Json& root, LayerPlan* p, const Fail& fail) {
  if (!size_of(&root, "width", "config", &p->width, fail) || !size_of(&root, "vocab", "config", &p->vocab, fail) ||
      !real_of(&root, "residual_mult", "config", &p->residual_mult, fail) || !real_of(root.get("norm"), "eps", "config.norm", &p->eps, fail))
    return false;
  if (!(p->eps >= 0.f)) return fail("config.norm: eps must not be negative");
  p->act = 2;  // clamped sigmoid-gated
  p->mixer_bias = true;
  p->residual = RESIDUAL_POST_NORM;
  p->scalar_norms = true;
  p->sinusoid_base = 10000.f;
  const Json* layers = root.get("layers");
  if (!layers || layers->kind != Json::Array || layers->items.empty()) return fail("config: 'layers' must be a non-empty list");
  if (layers->items.size() > 4096) return fail("config: too many layers");
  for (size_t i = 0; i < layers->items.size(); ++i) {
    const Json& l = layers->items[i];
    const std::string w = "config.layers[" + std::to_string(i) + "]";
    const Json* type = l.get("type");
    const Json* mixer = l.get("mixer");
    if (!type || type->kind != Json::String || !mixer || mixer->kind != Json::Object) return fail(w + ": 'type' and 'mixer' are needed");
    if (type->str != "attention") return fail(w + ": unknown layer type '" + type->str + "'");
    PlanLayer pl;
    pl.mixer = MIXER_GQA;
    if (!read_gqa(mixer, w + ".mixer", i, *p, &pl.gqa, fail)) return false;
    pl.gqa.qk_norm = pl.gqa.v_norm = pl.gqa.distance_bias = pl.gqa.head_gate = true;
    const Json* mlp = l.get("mlp");
    if (mlp && !mlp->is_null()) {
      const Json* kind = mlp->get("kind");
      if (!kind || kind->kind != Json::String) return fail(w + ".mlp: missing 'kind'");
      if (kind->str == "dense") {
        pl.mlp = FF_DENSE;
        if (!size_of(mlp, "ff", w + ".mlp", &pl.ff, fail) || !real_of(mlp, "limit", w + ".mlp", &pl.limit, fail)) return false;
      } else if (kind->str == "moe") {
        pl.mlp = FF_MOE;
        if (!read_moe(mlp, w + ".mlp", &pl.moe, fail)) return false;
      } else {
        return fail(w + ".mlp: unknown kind of feed-forward");
      }
    }
    p->layers.push_back(pl);
  }
  return true;
}

struct Architecture {
  const char* name;
  bool (*read)(const Json& root, LayerPlan* plan, const Fail& fail);
};
const Architecture kArchitectures[] = {{"Tometar", read_tometar}, {"Tutizen", read_tutizen}};

}  // namespace

bool plan_architecture_known(const std::string& name) {
  for (const Architecture& a : kArchitectures)
    if (name == a.name) return true;
  return false;
}

bool plan_parse(const char* json, size_t len, LayerPlan* out, std::string* err) {
  std::string why;
  const Fail fail{&why};
  Json root;
  bool ok = JsonReader(json, len).parse(&root, &why);
  if (ok) {
    const Json* a = root.get("architecture");
    if (!a || a->kind != Json::String) ok = fail("config: missing 'architecture'");
    else {
      bool found = false;
      for (const Architecture& arch : kArchitectures)
        if (a->str == arch.name) {
          found = true;
          *out = LayerPlan();
          out->architecture = a->str;
          ok = arch.read(root, out, fail);
        }
      if (!found) ok = fail("config: unknown architecture '" + a->str + "'");
    }
  }
  if (ok) {
    // rows of a projection stay below 2^31 and one matrix below 2^40 elements, so that no later product can wrap
    for (const PlanLayer& l : out->layers) {
      const uint64_t rows = l.mixer == MIXER_LATENT
                                ? (uint64_t)l.latent.heads * ((uint64_t)l.latent.dim + l.latent.rot + l.latent.vdim) + l.latent.rank + l.latent.rot
                            : l.mixer == MIXER_SSM
                                ? 2ull * l.ssm.heads * l.ssm.vdim + 2ull * l.ssm.groups * l.ssm.state + l.ssm.heads
                                : (uint64_t)l.gqa.heads * ((uint64_t)l.gqa.dim + l.gqa.vdim + 1) + (uint64_t)l.gqa.kv_heads * ((uint64_t)l.gqa.dim + l.gqa.vdim);
      const uint64_t ff = std::max<uint64_t>({2ull * l.ff, 2ull * l.moe.experts * l.moe.ff, 2ull * l.moe.shared_ff + l.moe.experts});
      for (const uint64_t r : {rows, ff})
        if (r >= (1ull << 28) || r * out->width >= (1ull << 40)) ok = fail("config: a layer is too large");
    }
  }
  if (!ok && err) *err = why;
  return ok;
}

std::vector<PlanTensor> plan_tensors(const LayerPlan& p) {
  std::vector<PlanTensor> t;
  const uint64_t H = p.width, S = p.streams;
  const std::vector<uint64_t> norm = p.scalar_norms ? std::vector<uint64_t>{} : std::vector<uint64_t>{H};
  t.push_back({"embed", {p.vocab, H}});
  for (size_t i = 0; i < p.layers.size(); ++i) {
    const PlanLayer& l = p.layers[i];
    const std::string n = "l" + std::to_string(i) + ".";
    auto add = [&](const std::string& name, std::vector<uint64_t> shape) { t.push_back({n + name, std::move(shape)}); };
    add("norm1", norm);
    if (l.has_mlp()) add("norm2", norm);
    if (l.mixer == MIXER_LATENT) {
      const LatentSpec& a = l.latent;
      add("mix.q", {a.q_rows(), H});
      add("mix.dkv", {a.kv_rows(), H});
      add("mix.dkv.norm", {a.rank});
      add("mix.uk", {(uint64_t)a.heads * a.dim, a.rank});
      add("mix.uv", {(uint64_t)a.heads * a.vdim, a.rank});
      add("mix.g", {a.gate_rows(), H});
      add("mix.o", {H, a.gate_rows()});
    } else if (l.mixer == MIXER_SSM) {
      const SsmSpec& s = l.ssm;
      add("mix.in", {s.in_rows(), H});
      add("mix.conv", {s.channels(), s.taps});
      add("mix.conv.b", {s.channels()});
      add("mix.dt_bias", {s.heads});
      add("mix.A_log", {s.heads});
      add("mix.D", {s.heads});
      add("mix.norm", {s.inner()});
      add("mix.o", {H, s.inner()});
    } else {
      const GqaSpec& a = l.gqa;
      auto linear = [&](const char* name, uint64_t rows, uint64_t cols) {
        add(std::string("mix.") + name, {rows, cols});
        if (p.mixer_bias) add(std::string("mix.") + name + ".b", {rows});
      };
      linear("q", a.q_rows(), H);
      if (a.own_kv()) {
        linear("k", a.k_cols(), H);
        linear("v", a.v_cols(), H);
      }
      if (a.head_gate) add("mix.g", {a.heads, H});
      linear("o", H, a.out_cols());
    }
    auto ff = [&](const std::string& pre, uint64_t rows, bool bias) {
      add(pre + "gate", {rows, H});
      if (bias) add(pre + "gate.b", {rows});
      add(pre + "up", {rows, H});
      if (bias) add(pre + "up.b", {rows});
      add(pre + "down", {H, rows});
      if (bias) add(pre + "down.b", {H});
    };
    if (l.mlp == FF_DENSE) ff("mlp.", l.ff, p.ff_bias);
    if (l.mlp == FF_MOE) {
      for (uint32_t e = 0; e < l.moe.experts; ++e) ff("mlp.e" + std::to_string(e) + ".", l.moe.ff, false);
      add("mlp.router", {l.moe.experts, H});
      add("mlp.correction", {l.moe.experts});
      if (l.moe.shared_ff) {
        ff("mlp.shared.", l.moe.shared_ff, false);
        add("mlp.shared.sg", {1, H});
      }
    }
    if (p.residual == RESIDUAL_STREAMS)
      for (int q = 1; q <= (l.has_mlp() ? 2 : 1); ++q) {
        const std::string hc = "hc" + std::to_string(q) + ".";
        add(hc + "in", {S});
        add(hc + "out", {S});
        add(hc + "mix", {S, S});
      }
  }
  t.push_back({"final.norm", norm});
  t.push_back({"head", {p.vocab, H}});
  return t;
}

}  // namespace nfai
