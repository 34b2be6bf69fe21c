// Model folders: config.json + model.safetensors -> nfai_model, through the public upload entry points. The weight file is
// memory-mapped; its header is untrusted, every offset is checked against the file before it is used.
#include <fcntl.h>
#include <stdio.h>
#include <string.h>
#include <sys/mman.h>
#include <sys/stat.h>
#include <unistd.h>

#include <string>
#include <unordered_map>
#include <vector>

#include "../../include/nfai_cuda.h"
#include "json.h"
#include "plan.h"

namespace nfai {
int ctx_fail(nfai_ctx* c, int code, const char* message);
}

namespace {

using namespace nfai;

struct Mapped {
  const char* p = nullptr;
  size_t n = 0;
  ~Mapped() {
    if (p) munmap((void*)p, n);
  }
  bool open(const std::string& path, std::string* err) {
    const int fd = ::open(path.c_str(), O_RDONLY | O_CLOEXEC);
    if (fd < 0) return *err = "cannot open " + path, false;
    struct stat st;
    bool ok = fstat(fd, &st) == 0 && S_ISREG(st.st_mode) && st.st_size > 0;
    if (ok) {
      void* a = mmap(nullptr, (size_t)st.st_size, PROT_READ, MAP_PRIVATE, fd, 0);
      ok = a != MAP_FAILED;
      if (ok) {
        p = (const char*)a;
        n = (size_t)st.st_size;
      }
    }
    close(fd);
    if (!ok) *err = "cannot map " + path;
    return ok;
  }
};

struct Entry {
  int dtype = 0;
  std::vector<uint64_t> shape;
  const char* data = nullptr;
  size_t bytes = 0;
};

bool whole(const Json& j, uint64_t* out) {
  if (j.kind != Json::Number || !(j.num >= 0 && j.num < 9007199254740992.0) || j.num != floor(j.num)) return false;
  *out = (uint64_t)j.num;
  return true;
}

// The entry `name` of a parsed header (indexed once: routed models have tens of thousands); data sits behind `base`.
using Directory = std::unordered_map<std::string, const Json*>;
bool find(const Directory& header, const char* base, size_t avail, const std::string& name, Entry* e, std::string* err) {
  const auto it = header.find(name);
  const Json* t = it == header.end() ? nullptr : it->second;
  if (!t) return *err = "model.safetensors has no tensor " + name, false;
  const Json *dt = t->get("dtype"), *sh = t->get("shape"), *of = t->get("data_offsets");
  const std::string bad = "model.safetensors: malformed entry of " + name;
  if (!dt || dt->kind != Json::String || !sh || sh->kind != Json::Array || !of || of->kind != Json::Array || of->items.size() != 2)
    return *err = bad, false;
  size_t es = 0;
  if (dt->str == "BF16") { e->dtype = NFAI_BF16; es = 2; }
  else if (dt->str == "F16") { e->dtype = NFAI_F16; es = 2; }
  else if (dt->str == "F32") { e->dtype = NFAI_F32; es = 4; }
  else return *err = "tensor " + name + ": element type " + dt->str + " is not supported", false;
  uint64_t count = 1, lo = 0, hi = 0;
  for (const Json& d : sh->items) {
    uint64_t v = 0;
    if (!whole(d, &v) || v == 0 || count > avail / v) return *err = bad, false;
    e->shape.push_back(v);
    count *= v;
  }
  if (!whole(of->items[0], &lo) || !whole(of->items[1], &hi) || hi < lo || hi > avail || hi - lo != count * es) return *err = bad, false;
  e->data = base + lo;
  e->bytes = (size_t)(hi - lo);
  return true;
}

}  // namespace

extern "C" int nfai_model_load_dir(nfai_ctx* c, const char* dir, uint32_t kv_cache_size, int weight_dtype, nfai_model** out) {
  if (!c) return ctx_fail(nullptr, NFAI_ERR_ARG, "ctx is null");
  if (!dir || !out) return ctx_fail(c, NFAI_ERR_ARG, "null argument");
  *out = nullptr;
  std::string err;
  Mapped cfg, st;
  LayerPlan plan;
  if (!cfg.open(std::string(dir) + "/config.json", &err) || !st.open(std::string(dir) + "/model.safetensors", &err) ||
      !plan_parse(cfg.p, cfg.n, &plan, &err))
    return ctx_fail(c, NFAI_ERR_ARG, err.c_str());
  uint64_t hlen = 0;
  if (st.n < 8) return ctx_fail(c, NFAI_ERR_ARG, "model.safetensors is truncated");
  memcpy(&hlen, st.p, 8);
  if (hlen > st.n - 8) return ctx_fail(c, NFAI_ERR_ARG, "model.safetensors is truncated");
  Json header;
  if (!JsonReader(st.p + 8, (size_t)hlen).parse(&header, &err)) return ctx_fail(c, NFAI_ERR_ARG, err.c_str());
  Directory directory;
  for (const auto& m : header.members) directory.emplace(m.first, &m.second);
  const char* base = st.p + 8 + hlen;
  const size_t avail = st.n - 8 - (size_t)hlen;
  // everything is looked up before a byte of device memory is taken
  const std::vector<PlanTensor> need = plan_tensors(plan);
  std::vector<Entry> entries(need.size());
  for (size_t i = 0; i < need.size(); ++i) {
    if (!find(directory, base, avail, need[i].name, &entries[i], &err)) return ctx_fail(c, NFAI_ERR_ARG, err.c_str());
    if (entries[i].shape != need[i].shape) return ctx_fail(c, NFAI_ERR_ARG, ("tensor " + need[i].name + ": shape does not match config.json").c_str());
  }
  nfai_model* m = nullptr;
  int rc = nfai_model_create_from_config(c, cfg.p, cfg.n, kv_cache_size, weight_dtype, &m);
  for (size_t i = 0; rc == NFAI_OK && i < need.size(); ++i) {
    std::vector<uint64_t> ne(entries[i].shape.rbegin(), entries[i].shape.rend());  // innermost first
    if (ne.empty()) ne.push_back(1);  // a single number
    rc = nfai_model_tensor_begin(m, need[i].name.c_str(), entries[i].dtype, ne.data(), (int)ne.size());
    if (rc == NFAI_OK) rc = nfai_model_tensor_chunk(m, entries[i].data, entries[i].bytes);
    if (rc == NFAI_OK) rc = nfai_model_tensor_end(m);
  }
  if (rc == NFAI_OK) rc = nfai_model_finalize(m);
  if (rc != NFAI_OK) {
    nfai_model_destroy(m);
    return rc;
  }
  *out = m;
  return NFAI_OK;
}
