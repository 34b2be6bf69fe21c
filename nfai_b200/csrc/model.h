// The objects behind the opaque handles of include/nfai_cuda.h (internal): device context, model, upload target; shared
// by the translation units that implement the C ABI.
#pragma once
#include <cuda_fp16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include <memory>
#include <string>
#include <vector>

#include "../../include/nfai_cuda.h"
#include "gemm_tc.h"
#include "kernels.h"
#include "tp.h"

namespace nfai {
constexpr size_t kStageBytes = 16u << 20;
constexpr int kStageSlots = 2;

inline size_t align_up(size_t v, size_t a) { return (v + a - 1) / a * a; }
inline size_t dtype_size(int dt) { return dt == NFAI_F32 ? 4 : 2; }
// Record the text of a failure on the context (may be null) and return `code`.
int fail(nfai_ctx* c, int code, const char* fmt, ...);
}  // namespace nfai

using namespace nfai;  // an internal header: every includer implements the C ABI

struct nfai_ctx {
  int device = 0;
  int rank = 0, world = 1;
  cudaStream_t stream = nullptr;
  cudaEvent_t ev0 = nullptr, ev1 = nullptr;
  void* stage[kStageSlots] = {nullptr, nullptr};  // pinned, device-visible
  cudaEvent_t stage_ev[kStageSlots] = {nullptr, nullptr};
  int stage_next = 0;
  uint32_t* pin_small = nullptr;  // pinned scratch for tokens / state read-back (256 bytes)
  uint32_t* dev_err = nullptr;    // device word for error bits of kernels that run outside a model step
  TpComm* tp = nullptr;
  bool pdl = true;
  bool use_graph = true;
  unsigned long long wait_ns = 1000000000ull;  // budget of every bounded device-side wait on peers (NFAI_WAIT_NS)
  std::string err;
};

#define CU(c, call)                                                                                    \
  do {                                                                                                 \
    cudaError_t e__ = (call);                                                                          \
    if (e__ != cudaSuccess)                                                                            \
      return fail((c), e__ == cudaErrorMemoryAllocation ? NFAI_ERR_OOM : NFAI_ERR_CUDA, "%s: %s (%s:%d)", #call, \
                  cudaGetErrorString(e__), __FILE__, __LINE__);                                        \
  } while (0)

namespace nfai {

struct Matrix {
  void* ptr = nullptr;
  uint64_t rows = 0, cols = 0;  // local (this rank's) shape
  size_t bytes = 0;
};

struct Gain {
  float* ptr = nullptr;
  bool done = false;
};

struct LayerW {
  Matrix qkv, o, gateup, down;
  Gain attn_norm, ffn_norm;
  bool got_q = false, got_k = false, got_v = false, got_o = false, got_gate = false, got_up = false, got_down = false;
};

// Where the tensor being uploaded goes.
struct UploadTarget {
  bool active = false;
  bool skip = false;  // accepted and ignored (output.weight on a tied model)
  std::string name;
  int src_dtype = 0, dst_dtype = 0;
  uint64_t K = 0, N = 0;  // source shape: N rows of K
  uint64_t received = 0;  // source elements so far
  IngestParams ip;
  bool* done_flag = nullptr;
};


// What a model described by a layer plan holds beyond the common part (plan_model.cu).
struct PlanModel;
struct PlanModelDeleter {
  void operator()(PlanModel* p) const;
};

}  // namespace nfai

struct nfai_model {
  nfai_ctx* ctx = nullptr;
  nfai_hparams hp{};
  // local (per-rank) geometry
  uint32_t qHl = 0, kvHl = 0, qDimL = 0, kvDimL = 0, Fl = 0, Vl = 0, v_lo = 0;
  bool finalized = false;
  char* warena = nullptr;
  size_t warena_bytes = 0;
  Matrix embd, head;
  bool got_embd = false, got_head = false;
  Gain out_norm;
  std::vector<LayerW> layers;
  UploadTarget up;
  // run-time buffers (one allocation)
  char* rarena = nullptr;
  void* kc = nullptr;
  void* vc = nullptr;  // [L][ctx][kvDimL]
  float2* rope_cs = nullptr;
  float* xbuf = nullptr;  // [(2L+1)][H]: x_in(0), then per layer (after attention, after FFN)
  float* q = nullptr;
  float* attn_out = nullptr;
  float* hbuf = nullptr;
  float* logits = nullptr;
  float* part_val = nullptr;
  uint32_t* part_idx = nullptr;
  uint32_t nparts = 0, nparts_alloc = 0;
  float* attn_part = nullptr;
  uint32_t* tickets = nullptr;
  uint32_t S_max = 1;
  uint32_t attn_heads = 4;  // query heads per attention CTA in the decode step
  std::vector<AttnTileMaps> attn_maps;  // per layer, when the decode step uses the tile-staged attention kernel
  bool attn_mma = false;                // long float16 caches: the tensor-core attention kernel (default over the tile-staged one)
  StepState* state = nullptr;
  uint32_t* history = nullptr;
  uint32_t* prompt = nullptr;
  float* pin_logits = nullptr;  // pinned V floats
  float* tp_buf = nullptr;      // [H] partial sums exchanged between ranks
  void* sample_scratch = nullptr;  // per-slice sums and candidates of the on-device sampler
  cudaGraphExec_t g_full = nullptr, g_nohead = nullptr;
  int launches_full = 0;
  uint32_t pos = 0;  // host mirror of state->pos
  GemvTune tune_qkv, tune_o, tune_gateup, tune_down, tune_head;
  // batched prompt path (float16 weights, one GPU): chunk workspace
  bool prefill_gemm = false;
  uint32_t pf_chunk = 0;
  float* pfX0 = nullptr;      // [chunk][H] residual stream
  float* pfX1 = nullptr;      // [chunk][H]
  __half* pfA = nullptr;      // [chunk][max(H, qDim)] normalised activations
  float* pfQ = nullptr;       // [chunk][qDim] rotated queries
  __half* pfAO = nullptr;     // [chunk][qDim] attention output
  __half* pfH = nullptr;      // [chunk][F] SiLU(gate)*up
  float* pfPart = nullptr;    // split-K partial tiles of the prompt GEMMs
  size_t pfPartFloats = 0;
  uint32_t* pfTok = nullptr;  // [chunk]
  // L2 look-ahead: how far beyond the weights a kernel consumes the step's weight sequence is requested
  uint64_t pf_look = 0, pf_extra = 0;
  int pf_mode = 1;
  // layer-plan models: their layers' weights, caches, states and workspaces (the Llama-block members above stay empty)
  std::unique_ptr<PlanModel, PlanModelDeleter> plan;
};

namespace nfai {

// ---- shared by api.cu and plan_model.cu ------------------------------------------------------------------------------------
// Hands out 256-byte aligned pieces of one allocation.
struct Arena {
  size_t off = 0;
  size_t take(size_t bytes) {
    const size_t at = off;
    off = align_up(off + bytes, 256);
    return at;
  }
};
// The run-time buffers every model has: logits, arg-max partials, step state, history, prompt, sampler scratch.
struct CommonOffsets {
  size_t logits, part_val, part_idx, state, history, prompt, sample;
};
CommonOffsets place_common(nfai_model* m, Arena& a);
void bind_common(nfai_model* m, const CommonOffsets& o);
int capture_graphs(nfai_model* m);
int ready(nfai_model* m);
int check_state(nfai_model* m, StepState* host_copy);
int set_state_word(nfai_model* m, size_t offset, uint32_t value, int slot);
void read_tune(const char* name, GemvTune& t, int r_default, int u_default);

// ---- hooks of layer-plan models (plan_model.cu), called where the Llama path would run its own code --------------------------
int plan_resolve(nfai_model* m, const char* name, const uint64_t* shape, int ndim, UploadTarget* t);
int plan_finalize(nfai_model* m);
cudaError_t plan_record_step(nfai_model* m, bool with_head, bool from_prompt, int* launches);
// n tokens at the current position in batched passes; logits of the places `want` (ascending) if given, and the last token's
// logits and arg-max where a decode step leaves them. Position in *state advanced; m->pos is the caller's.
int plan_prefill(nfai_model* m, const uint32_t* tokens, int n, const uint32_t* want, int n_want, float* logits_out);
bool plan_batched(const nfai_model* m);
int plan_step_launches(const nfai_model* m);
bool plan_rewinds(const nfai_model* m);  // every layer keeps rows per position: any earlier position can be returned to
// settled: the residual behind the last layer is already in place (a prompt pass leaves it there)
GemvParams plan_head_params(nfai_model* m, bool settled = false);
size_t plan_snapshot_bytes(const nfai_model* m, uint32_t pos);
cudaError_t plan_snapshot_copy(nfai_model* m, uint32_t pos, char* buf, bool save);
int plan_read_kv(nfai_model* m, uint32_t layer, uint32_t pos, float* k, float* v);
int plan_read_hidden(nfai_model* m, uint32_t layer, float* out);
// One launch of the decode-step kernel `which` for profiling, and the bytes it must move; null pointer when the model has none.
cudaError_t plan_profile_launch(nfai_model* m, int which, int iter);
uint64_t plan_profile_bytes(nfai_model* m, int which);

}  // namespace nfai
