// config.json -> LayerPlan, and the tensors a plan needs. Host code only; every number of the file is checked before it
// is used as a size.
#include "plan.h"

#include <math.h>
#include <stdio.h>

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
      pl.has_mlp = true;
    }
    p->layers.push_back(pl);
  }
  return true;
}

struct Architecture {
  const char* name;
  bool (*read)(const Json& root, LayerPlan* plan, const Fail& fail);
};
const Architecture kArchitectures[] = {{"Tometar", read_tometar}};

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
                                : 2ull * l.ssm.heads * l.ssm.vdim + 2ull * l.ssm.groups * l.ssm.state + l.ssm.heads;
      if (rows >= (1ull << 28) || rows * out->width >= (1ull << 40)) ok = fail("config: a layer is too large");
    }
  }
  if (!ok && err) *err = why;
  return ok;
}

std::vector<PlanTensor> plan_tensors(const LayerPlan& p) {
  std::vector<PlanTensor> t;
  const uint64_t H = p.width, S = p.streams;
  t.push_back({"embed", {p.vocab, H}});
  for (size_t i = 0; i < p.layers.size(); ++i) {
    const PlanLayer& l = p.layers[i];
    const std::string n = "l" + std::to_string(i) + ".";
    auto add = [&](const char* name, std::vector<uint64_t> shape) { t.push_back({n + name, std::move(shape)}); };
    add("norm1", {H});
    if (l.has_mlp) add("norm2", {H});
    if (l.mixer == MIXER_LATENT) {
      const LatentSpec& a = l.latent;
      add("mix.q", {a.q_rows(), H});
      add("mix.dkv", {a.kv_rows(), H});
      add("mix.dkv.norm", {a.rank});
      add("mix.uk", {(uint64_t)a.heads * a.dim, a.rank});
      add("mix.uv", {(uint64_t)a.heads * a.vdim, a.rank});
      add("mix.g", {a.gate_rows(), H});
      add("mix.o", {H, a.gate_rows()});
    } else {
      const SsmSpec& s = l.ssm;
      add("mix.in", {s.in_rows(), H});
      add("mix.conv", {s.channels(), s.taps});
      add("mix.conv.b", {s.channels()});
      add("mix.dt_bias", {s.heads});
      add("mix.A_log", {s.heads});
      add("mix.D", {s.heads});
      add("mix.norm", {s.inner()});
      add("mix.o", {H, s.inner()});
    }
    if (l.has_mlp) {
      add("mlp.gate", {l.ff, H});
      add("mlp.gate.b", {l.ff});
      add("mlp.up", {l.ff, H});
      add("mlp.up.b", {l.ff});
      add("mlp.down", {H, l.ff});
      add("mlp.down.b", {H});
    }
    for (int q = 1; q <= (l.has_mlp ? 2 : 1); ++q) {
      const std::string hc = "hc" + std::to_string(q) + ".";
      add((hc + "in").c_str(), {S});
      add((hc + "out").c_str(), {S});
      add((hc + "mix").c_str(), {S, S});
    }
  }
  t.push_back({"final.norm", {H}});
  t.push_back({"head", {p.vocab, H}});
  return t;
}

}  // namespace nfai
