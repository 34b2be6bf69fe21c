// Models described by a layer plan (plan.h) behind the same handle, upload calls, decode graphs, samplers and snapshots as
// the Llama models: this file places their weights, caches and recurrent states, and lays out their decode step and prompt
// passes as sequences of kernel launches.
//
// Decode step, per layer (H = width, S = streams):
//   latent attention   GEMV [q | latent, key part | gate] (norm in its prologue)
//                      latent_decode (query to latents, window, values, gate; cache row)
//                      GEMV o, whose epilogue writes all S streams and forms the next sublayer's input
//   state space        GEMV in-projection into the ring row of this position
//                      ssm_step_kernel (convolution, step size, state, skip, gate)
//                      GEMV o with the grouped norm in its prologue, hyper epilogue as above
//   feed-forward       GEMV gate/up (norm prologue, biases, gated), GEMV down (bias, hyper epilogue)
// and with a post-norm residual, where x += mult * norm(y) is formed by whoever reads x next (prologue of its GEMV):
//   grouped-query      GEMV [q | k | v | gate] (bias), gqa_decode (norms, cache row, attention, gate), GEMV o (bias)
//   feed-forward       GEMV gate/up, GEMV down
//   routed             GEMV [shared gate/up | router], GEMV gate/up of the chosen experts (chosen in its prologue, weights in
//                      its epilogue), GEMV down over the chosen and the shared hidden values together
// Prompt pass: the same mathematics on rows of tokens, products on the tensor cores (bfloat16) or, for float32 models, in
// true float32 on the CUDA cores.
#include <string.h>

#include <algorithm>
#include <cmath>
#include <map>

#include "model.h"
#include "plan_kernels.h"

namespace nfai {

namespace {

struct Vector {  // float32 parameters
  float* ptr = nullptr;
};

struct SubW {  // norm of one sublayer, and its hyper-connection if the residual has streams
  Vector norm, in, out, mix;
};

struct LayerWeights {
  Matrix in, out;  // mixer projections
  Matrix kv;       // latent attention: [heads*dim | heads*vdim][rank]
  Vector lat_norm;
  Vector conv, conv_b, dt_bias, A_log, D, ssm_norm;
  Vector in_b, out_b;  // grouped-query attention: biases of the projections (zero for the gate rows)
  Matrix gateup, down;
  Vector gateup_b, down_b;
  // routed feed-forward: [shared gate/up | router | shared's gate], the experts' matrices one after the other, shared down
  Matrix first, exp_gateup, exp_down, shared_down;
  Vector correction;
  SubW sub[2];
};

struct LayerState {
  // latent attention
  char* c = nullptr;
  char* kr = nullptr;
  void* scratch = nullptr;
  float2* rope = nullptr;
  // state space
  float* ring = nullptr;
  float* S = nullptr;
  // grouped-query attention: own or borrowed rows
  char* k = nullptr;
  char* v = nullptr;
};

struct TensorSlot {
  uint64_t K = 0, N = 0;  // source: N rows of K
  int ndim = 0;
  void* dst = nullptr;
  int dst_dtype = 0;
  uint64_t row_mul = 1, row_off = 0;
  bool done = false;
};

}  // namespace

struct PlanModel {
  LayerPlan plan;
  std::map<std::string, TensorSlot> slots;
  std::vector<LayerWeights> w;
  std::vector<LayerState> st;
  Vector ones;  // [S]
  int act_dtype = 0;  // caches and operands of products: the weights' type
  // decode
  float* X = nullptr;    // [sublayers + 1][S][H]: streams before every sublayer and at the end
  float* u = nullptr;    // [H] what the next reader reads
  float* mix = nullptr;  // [max in_rows]
  float* ao = nullptr;   // [max out_cols]
  float* hbuf = nullptr; // [max hidden values of a feed-forward]
  float* y = nullptr;    // [H] output of the last sublayer (post-norm residual)
  float* tail = nullptr; // [max tail rows] router logits and the shared feed-forward's gate
  uint32_t* chosen = nullptr;  // [kMaxChosen]
  double* freq = nullptr;      // [(H+1)/2] angles per position of the position vector
  int step_launches = 0;
  // prompt passes
  bool batched = false;
  uint32_t chunk = 0;
  float* pX = nullptr;   // [chunk][S][H]
  char* pA = nullptr;    // [chunk][max(H, out_cols)] operand
  float* pIn = nullptr;  // [chunk][max in_rows]
  char* pQ = nullptr;    // [chunk][max q_rows] operand
  char* pKV = nullptr;   // [rows][max heads*(dim+vdim)] operand
  float* pY = nullptr;   // [chunk][H]
  char* pF = nullptr;    // [chunk][max ff] operand
  char* pXBC = nullptr;  // [chunk][max channels] operand
  float* pDT = nullptr;  // [chunk][max heads]
  float* pSY = nullptr;  // [chunk][max inner]
  float* pChunk = nullptr;
  size_t pChunkFloats = 0;
  float* pPart = nullptr;
  size_t pPartFloats = 0;
  float* pTail = nullptr;     // [chunk][max tail]
  char* pG = nullptr;         // [chunk*top][H] operand: rows sorted by expert
  char* pFE = nullptr;        // [chunk*top][expert ff] operand
  float* pYE = nullptr;       // [chunk*top][H]
  MoeRows pRoute;             // its lists
  uint32_t* pTok = nullptr;   // [chunk]
  uint32_t* pRows = nullptr;  // [chunk]
  float* pLogits = nullptr;   // [logit_rows][V]
  uint32_t logit_rows = 0;
  float* pin_rows = nullptr;  // pinned [logit_rows][V]
};

void PlanModelDeleter::operator()(PlanModel* p) const {
  if (p && p->pin_rows) cudaFreeHost(p->pin_rows);
  delete p;
}

namespace {

uint32_t max_over(const LayerPlan& p, uint32_t (*f)(const PlanLayer&)) {
  uint32_t m = 0;
  for (const PlanLayer& l : p.layers) m = std::max(m, f(l));
  return m;
}
uint32_t f_in(const PlanLayer& l) { return l.in_rows(); }
uint32_t f_out(const PlanLayer& l) { return l.out_cols(); }
uint32_t f_ff(const PlanLayer& l) { return l.mlp == FF_DENSE ? l.ff : l.mlp == FF_MOE ? l.moe.shared_ff : 0; }
uint32_t f_hidden(const PlanLayer& l) { return l.mlp == FF_DENSE ? l.ff : l.mlp == FF_MOE ? l.moe.hidden() : 0; }
uint32_t f_tail(const PlanLayer& l) { return l.mlp == FF_MOE ? l.moe.first_rows() - l.moe.gated_rows() : 0; }
uint32_t f_experts(const PlanLayer& l) { return l.mlp == FF_MOE ? l.moe.experts : 0; }
uint32_t f_top(const PlanLayer& l) { return l.mlp == FF_MOE ? l.moe.top : 0; }
uint32_t f_sorted_ff(const PlanLayer& l) { return l.mlp == FF_MOE ? l.moe.top * l.moe.ff : 0; }
uint32_t f_q(const PlanLayer& l) { return l.mixer == MIXER_LATENT ? l.latent.q_rows() : l.mixer == MIXER_GQA ? l.gqa.q_rows() : 0; }
uint32_t f_kv(const PlanLayer& l) { return l.mixer == MIXER_LATENT ? l.latent.heads * (l.latent.dim + l.latent.vdim) : 0; }
uint32_t f_ch(const PlanLayer& l) { return l.mixer == MIXER_SSM ? l.ssm.channels() : 0; }
uint32_t f_sh(const PlanLayer& l) { return l.mixer == MIXER_SSM ? l.ssm.heads : 0; }
uint32_t f_inner(const PlanLayer& l) { return l.mixer == MIXER_SSM ? l.ssm.inner() : 0; }
// most rows of expanded keys and values a pass of `chunk` tokens needs
uint32_t kv_rows_needed(const PlanLayer& l, uint32_t chunk, uint32_t ctx) {
  if (l.mixer != MIXER_LATENT) return 0;
  if (!l.latent.window) return ctx;
  return (uint32_t)std::min<uint64_t>(ctx, (uint64_t)l.latent.window - 1 + chunk);
}

float* streams(nfai_model* m, uint32_t sub) { return m->plan->X + (size_t)sub * m->plan->plan.streams * m->hp.H; }

}  // namespace

}  // namespace nfai

// ---- creation -----------------------------------------------------------------------------------------------------------------
static int plan_create(nfai_ctx* c, LayerPlan&& plan_in, uint32_t ctx_size, int weight_dtype, nfai_model** out) {
  if (c->world != 1) return fail(c, NFAI_ERR_ARG, "models with a layer plan run on one GPU");
  if (weight_dtype != NFAI_F32 && weight_dtype != NFAI_BF16) return fail(c, NFAI_ERR_ARG, "weight_dtype must be NFAI_F32 or NFAI_BF16");
  if (!ctx_size) return fail(c, NFAI_ERR_ARG, "the cache capacity must be positive");
  CU(c, cudaSetDevice(c->device));
  std::unique_ptr<nfai_model> m(new nfai_model());
  m->ctx = c;
  m->plan.reset(new PlanModel());
  PlanModel* P = m->plan.get();
  P->plan = std::move(plan_in);
  const LayerPlan& pl = P->plan;
  for (const PlanLayer& l : pl.layers) {
    std::string why;
    if (l.mixer == MIXER_LATENT && !latent_supported(l.latent, weight_dtype, &why)) return fail(c, NFAI_ERR_ARG, "%s", why.c_str());
    if (l.mixer == MIXER_GQA && !gqa_supported(l.gqa, &why)) return fail(c, NFAI_ERR_ARG, "%s", why.c_str());
    if (l.mlp == FF_MOE && (pl.act != ACT_CLAMPED || pl.residual != RESIDUAL_POST_NORM))
      return fail(c, NFAI_ERR_ARG, "routed feed-forwards come with the clamped activation and a post-norm residual");
  }
  P->act_dtype = weight_dtype;
  nfai_hparams& hp = m->hp;
  hp.H = pl.width;
  hp.L = (uint32_t)pl.layers.size();
  hp.V = pl.vocab;
  hp.ctx = ctx_size;
  hp.eps = pl.eps;
  hp.weight_dtype = hp.kv_dtype = weight_dtype;
  m->Vl = hp.V;
  const size_t ws = dtype_size(weight_dtype);
  Arena a;
  auto place = [&](Matrix& M, uint64_t rows, uint64_t cols) {
    M.rows = rows;
    M.cols = cols;
    M.bytes = rows * cols * ws;
    M.ptr = (void*)a.take(M.bytes);
  };
  auto vec = [&](Vector& v, uint64_t n) { v.ptr = (float*)a.take(n * 4); };
  const uint64_t H = hp.H, S = pl.streams;
  place(m->embd, hp.V, H);
  place(m->head, hp.V, H);
  const uint64_t norm_len = pl.scalar_norms ? 1 : H;
  m->out_norm.ptr = (float*)a.take(norm_len * 4);
  vec(P->ones, S);
  P->w.resize(hp.L);
  for (uint32_t i = 0; i < hp.L; ++i) {
    const PlanLayer& l = pl.layers[i];
    LayerWeights& w = P->w[i];
    place(w.in, l.in_rows(), H);
    if (l.mixer == MIXER_LATENT) {
      place(w.kv, (uint64_t)l.latent.heads * (l.latent.dim + l.latent.vdim), l.latent.rank);
      vec(w.lat_norm, l.latent.rank);
    } else if (l.mixer == MIXER_SSM) {
      vec(w.conv, (uint64_t)l.ssm.channels() * l.ssm.taps);
      vec(w.conv_b, l.ssm.channels());
      vec(w.dt_bias, l.ssm.heads);
      vec(w.A_log, l.ssm.heads);
      vec(w.D, l.ssm.heads);
      vec(w.ssm_norm, l.ssm.inner());
    }
    place(w.out, H, l.out_cols());
    if (l.mixer == MIXER_GQA && pl.mixer_bias) {
      vec(w.in_b, l.in_rows());
      vec(w.out_b, H);
    }
    if (l.mlp == FF_DENSE) {
      place(w.gateup, 2 * (uint64_t)l.ff, H);
      place(w.down, H, l.ff);
      if (pl.ff_bias) {
        vec(w.gateup_b, 2 * (uint64_t)l.ff);
        vec(w.down_b, H);
      }
    }
    if (l.mlp == FF_MOE) {
      place(w.first, l.moe.first_rows(), H);
      place(w.exp_gateup, 2 * (uint64_t)l.moe.experts * l.moe.ff, H);
      place(w.exp_down, l.moe.experts * H, l.moe.ff);
      if (l.moe.shared_ff) place(w.shared_down, H, l.moe.shared_ff);
      vec(w.correction, l.moe.experts);
    }
    for (int q = 0; q < (l.has_mlp() ? 2 : 1); ++q) {
      vec(w.sub[q].norm, norm_len);
      if (pl.residual != RESIDUAL_STREAMS) continue;
      vec(w.sub[q].in, S);
      vec(w.sub[q].out, S);
      vec(w.sub[q].mix, S * S);
    }
  }
  m->warena_bytes = a.off;
  cudaError_t e = cudaMalloc((void**)&m->warena, a.off);
  if (e != cudaSuccess) return fail(c, NFAI_ERR_OOM, "cudaMalloc of %zu weight bytes: %s", a.off, cudaGetErrorString(e));
  if ((e = cudaMemset(m->warena, 0, a.off)) != cudaSuccess) {  // rows and biases no tensor fills stay zero
    cudaFree(m->warena);
    return fail(c, NFAI_ERR_CUDA, "cudaMemset: %s", cudaGetErrorString(e));
  }
  auto fix = [&](Matrix& M) { M.ptr = m->warena + (size_t)M.ptr; };
  auto fixv = [&](Vector& v) { v.ptr = (float*)(m->warena + (size_t)v.ptr); };
  fix(m->embd);
  fix(m->head);
  m->out_norm.ptr = (float*)(m->warena + (size_t)m->out_norm.ptr);
  fixv(P->ones);
  // where every tensor of the plan goes
  auto mat = [&](const std::string& n, const Matrix& M, uint64_t rows, uint64_t off, uint64_t mul = 1) {
    TensorSlot t;
    t.K = M.cols; t.N = rows; t.ndim = 2; t.dst = M.ptr; t.dst_dtype = weight_dtype; t.row_off = off; t.row_mul = mul;
    P->slots[n] = t;
  };
  auto flat = [&](const std::string& n, const Vector& v, uint64_t rows, uint64_t cols = 0) {  // cols = 0: one dimension
    TensorSlot t;
    t.K = cols ? cols : rows; t.N = cols ? rows : 1; t.ndim = cols ? 2 : 1; t.dst = v.ptr; t.dst_dtype = NFAI_F32;
    P->slots[n] = t;
  };
  auto strided = [&](const std::string& n, const Vector& v, uint64_t rows, uint64_t off, uint64_t mul = 2) {  // every mul-th element from off
    TensorSlot t;
    t.K = 1; t.N = rows; t.ndim = 1; t.dst = v.ptr; t.dst_dtype = NFAI_F32; t.row_mul = mul; t.row_off = off;
    P->slots[n] = t;
  };
  mat("embed", m->embd, hp.V, 0);
  mat("head", m->head, hp.V, 0);
  flat("final.norm", Vector{m->out_norm.ptr}, norm_len);
  for (uint32_t i = 0; i < hp.L; ++i) {
    const PlanLayer& l = pl.layers[i];
    LayerWeights& w = P->w[i];
    const std::string n = "l" + std::to_string(i) + ".";
    fix(w.in);
    fix(w.out);
    if (l.mixer == MIXER_LATENT) {
      const LatentSpec& s = l.latent;
      fix(w.kv);
      fixv(w.lat_norm);
      mat(n + "mix.q", w.in, s.q_rows(), 0);
      mat(n + "mix.dkv", w.in, s.kv_rows(), s.q_rows());
      mat(n + "mix.g", w.in, s.gate_rows(), s.q_rows() + s.kv_rows());
      mat(n + "mix.uk", w.kv, (uint64_t)s.heads * s.dim, 0);
      mat(n + "mix.uv", w.kv, (uint64_t)s.heads * s.vdim, (uint64_t)s.heads * s.dim);
      flat(n + "mix.dkv.norm", w.lat_norm, s.rank);
    } else if (l.mixer == MIXER_GQA) {
      const GqaSpec& s = l.gqa;
      if (pl.mixer_bias) {
        fixv(w.in_b);
        fixv(w.out_b);
        flat(n + "mix.o.b", w.out_b, H);
      }
      auto rows = [&](const char* name, uint64_t count, uint64_t off, bool bias) {
        mat(n + "mix." + name, w.in, count, off);
        if (bias) strided(n + "mix." + name + ".b", w.in_b, count, off, 1);
      };
      rows("q", s.q_rows(), 0, pl.mixer_bias);
      if (s.own_kv()) {
        rows("k", s.k_cols(), s.q_rows(), pl.mixer_bias);
        rows("v", s.v_cols(), s.q_rows() + s.k_cols(), pl.mixer_bias);
      }
      if (s.head_gate) rows("g", s.heads, s.gate_row0(), false);
    } else {
      const SsmSpec& s = l.ssm;
      fixv(w.conv); fixv(w.conv_b); fixv(w.dt_bias); fixv(w.A_log); fixv(w.D); fixv(w.ssm_norm);
      mat(n + "mix.in", w.in, s.in_rows(), 0);
      flat(n + "mix.conv", w.conv, s.channels(), s.taps);
      flat(n + "mix.conv.b", w.conv_b, s.channels());
      flat(n + "mix.dt_bias", w.dt_bias, s.heads);
      flat(n + "mix.A_log", w.A_log, s.heads);
      flat(n + "mix.D", w.D, s.heads);
      flat(n + "mix.norm", w.ssm_norm, s.inner());
    }
    mat(n + "mix.o", w.out, H, 0);
    auto feed_forward = [&](const std::string& pre, const Matrix& gateup, const Matrix& down, uint64_t ff, uint64_t index) {
      mat(pre + "gate", gateup, ff, index * 2 * ff, 2);
      mat(pre + "up", gateup, ff, index * 2 * ff + 1, 2);
      mat(pre + "down", down, H, index * H);
    };
    if (l.mlp == FF_DENSE) {
      fix(w.gateup); fix(w.down);
      feed_forward(n + "mlp.", w.gateup, w.down, l.ff, 0);
      if (pl.ff_bias) {
        fixv(w.gateup_b); fixv(w.down_b);
        strided(n + "mlp.gate.b", w.gateup_b, l.ff, 0);
        strided(n + "mlp.up.b", w.gateup_b, l.ff, 1);
        flat(n + "mlp.down.b", w.down_b, H);
      }
    }
    if (l.mlp == FF_MOE) {
      const MoeSpec& s = l.moe;
      fix(w.first); fix(w.exp_gateup); fix(w.exp_down); fixv(w.correction);
      for (uint32_t x = 0; x < s.experts; ++x) feed_forward(n + "mlp.e" + std::to_string(x) + ".", w.exp_gateup, w.exp_down, s.ff, x);
      mat(n + "mlp.router", w.first, s.experts, s.gated_rows());
      flat(n + "mlp.correction", w.correction, s.experts);
      if (s.shared_ff) {
        fix(w.shared_down);
        feed_forward(n + "mlp.shared.", w.first, w.shared_down, s.shared_ff, 0);
        mat(n + "mlp.shared.sg", w.first, 1, s.gated_rows() + s.experts);
      }
    }
    for (int q = 0; q < (l.has_mlp() ? 2 : 1); ++q) {
      SubW& sw = w.sub[q];
      fixv(sw.norm);
      flat(n + "norm" + std::to_string(q + 1), sw.norm, norm_len);
      if (pl.residual != RESIDUAL_STREAMS) continue;
      fixv(sw.in); fixv(sw.out); fixv(sw.mix);
      const std::string hc = n + "hc" + std::to_string(q + 1) + ".";
      flat(hc + "in", sw.in, S);
      flat(hc + "out", sw.out, S);
      flat(hc + "mix", sw.mix, S, S);
    }
  }
  read_tune("QKV", m->tune_qkv, 2, 4);
  read_tune("O", m->tune_o, 2, 4);
  read_tune("GATEUP", m->tune_gateup, 2, 4);
  read_tune("DOWN", m->tune_down, 2, 4);
  read_tune("HEAD", m->tune_head, 2, 4);
  const std::vector<float> one(S, 1.0f);
  e = cudaMemcpy(P->ones.ptr, one.data(), S * 4, cudaMemcpyHostToDevice);
  if (e != cudaSuccess) {
    cudaFree(m->warena);
    return fail(c, NFAI_ERR_CUDA, "cudaMemcpy: %s", cudaGetErrorString(e));
  }
  *out = m.release();
  return NFAI_OK;
}

namespace nfai {

int plan_resolve(nfai_model* m, const char* name, const uint64_t* shape, int ndim, UploadTarget* t) {
  nfai_ctx* c = m->ctx;
  auto it = m->plan->slots.find(name);
  if (it == m->plan->slots.end()) return fail(c, NFAI_ERR_ARG, "unknown tensor name %s", name);
  TensorSlot& s = it->second;
  const uint64_t inner = s.ndim == 1 ? s.K * s.N : s.K;
  if (ndim != s.ndim || shape[0] != inner || (ndim == 2 && shape[1] != s.N))
    return fail(c, NFAI_ERR_ARG, "tensor %s: shape does not match the model", name);
  t->name = name;
  t->received = 0;
  t->skip = false;
  t->K = s.K;
  t->N = s.N;
  t->dst_dtype = s.dst_dtype;
  t->done_flag = &s.done;
  IngestParams& ip = t->ip;
  ip = IngestParams();
  ip.K = s.K;
  ip.row_hi = s.N;
  ip.col_hi = s.K;
  ip.row_mul = s.row_mul;
  ip.row_off = s.row_off;
  ip.ldd = s.K;
  ip.dst = s.dst;
  return NFAI_OK;
}

int plan_finalize(nfai_model* m) {
  nfai_ctx* c = m->ctx;
  PlanModel* P = m->plan.get();
  const LayerPlan& pl = P->plan;
  const nfai_hparams& hp = m->hp;
  for (const auto& s : P->slots)
    if (!s.second.done) return fail(c, NFAI_ERR_STATE, "missing tensor %s", s.first.c_str());
  CU(c, cudaSetDevice(c->device));
  CU(c, cudaStreamSynchronize(c->stream));
  const size_t as = dtype_size(P->act_dtype);
  const uint32_t H = hp.H, S = pl.streams;
  m->nparts = gemv_grid(hp.weight_dtype, EPI_LOGITS, plan_head_params(m), m->tune_head);
  Arena a;
  const CommonOffsets common = place_common(m, a);
  // per layer: caches and states; one (cos, sin) table per distinct rotation
  struct Off { size_t c = 0, kr = 0, scratch = 0, rope = 0, ring = 0, S = 0, k = 0, v = 0; };
  std::vector<Off> off(hp.L);
  std::map<std::pair<uint32_t, float>, size_t> ropes;
  for (uint32_t i = 0; i < hp.L; ++i) {
    const PlanLayer& l = pl.layers[i];
    if (l.mixer == MIXER_LATENT) {
      off[i].c = a.take((size_t)hp.ctx * l.latent.rank * as);
      off[i].kr = a.take((size_t)hp.ctx * l.latent.rot * as);
      off[i].scratch = a.take(latent_decode_scratch(l.latent, P->act_dtype, hp.ctx));
      const std::pair<uint32_t, float> key(l.latent.rope_dims, l.latent.rope_base);
      auto r = ropes.find(key);
      if (r == ropes.end()) r = ropes.emplace(key, a.take((size_t)hp.ctx * (key.first / 2) * sizeof(float2) + 16)).first;
      off[i].rope = r->second;
    } else if (l.mixer == MIXER_GQA) {
      if (l.gqa.own_kv()) {
        off[i].k = a.take((size_t)hp.ctx * l.gqa.k_cols() * as);
        off[i].v = a.take((size_t)hp.ctx * l.gqa.v_cols() * as);
      }
      off[i].scratch = a.take(gqa_decode_scratch(l.gqa, hp.ctx));
    } else {
      off[i].ring = a.take((size_t)l.ssm.taps * l.ssm.in_rows() * 4);
      off[i].S = a.take((size_t)l.ssm.heads * l.ssm.vdim * l.ssm.state * 4);
    }
  }
  const size_t o_X = a.take((size_t)(pl.sublayers() + 1) * S * H * 4);
  const size_t o_u = a.take((size_t)H * 4);
  const size_t o_mix = a.take((size_t)max_over(pl, f_in) * 4);
  const size_t o_ao = a.take((size_t)max_over(pl, f_out) * 4);
  const size_t o_h = a.take((size_t)max_over(pl, f_hidden) * 4 + 16);
  const size_t o_y = a.take((size_t)H * 4);
  const size_t o_tail = a.take((size_t)max_over(pl, f_tail) * 4);
  const size_t o_chosen = a.take((size_t)kMaxChosen * 4);
  const size_t o_freq = a.take((size_t)(H + 1) / 2 * sizeof(double));
  // prompt passes
  P->batched = env_int("NFAI_PREFILL_GEMM", 1) != 0;
  const uint32_t want = (uint32_t)std::min(std::max(env_int("NFAI_PREFILL_CHUNK", 2048), 8), 8192);
  const uint32_t T = P->batched ? std::min(hp.ctx, want) : 0;
  P->chunk = T;
  uint32_t kv_elems_rows = 0;
  size_t kv_bytes = 0, chunk_floats = 0;
  for (const PlanLayer& l : pl.layers) {
    kv_elems_rows = T ? kv_rows_needed(l, T, hp.ctx) : 0;
    kv_bytes = std::max(kv_bytes, (size_t)kv_elems_rows * f_kv(l) * as);
    if (T && l.mixer == MIXER_SSM) chunk_floats = std::max(chunk_floats, ssm_chunk_floats(l.ssm, T));
  }
  const uint32_t amax = std::max(H, max_over(pl, f_out));
  const size_t o_pX = a.take((size_t)T * S * H * 4);
  const size_t o_pA = a.take((size_t)T * amax * as);
  const size_t o_pIn = a.take((size_t)T * max_over(pl, f_in) * 4);
  const size_t o_pQ = a.take((size_t)T * max_over(pl, f_q) * as);
  const size_t o_pKV = a.take(kv_bytes);
  const size_t o_pY = a.take((size_t)T * H * 4);
  const size_t o_pF = a.take((size_t)T * max_over(pl, f_ff) * as);
  const size_t o_pXBC = a.take((size_t)T * max_over(pl, f_ch) * as);
  const size_t o_pDT = a.take((size_t)T * max_over(pl, f_sh) * 4);
  const size_t o_pSY = a.take((size_t)T * max_over(pl, f_inner) * 4);
  const size_t o_pC = a.take(chunk_floats * 4);
  const size_t part = T && P->act_dtype == NFAI_BF16 && env_int("NFAI_GEMM_SPLIT", 1) ? (size_t)sm_count() * 128 * 128 * 2 : 0;
  const size_t o_pp = a.take(part * 4);
  // routed feed-forwards: the widest of each list over the layers
  const uint32_t top = max_over(pl, f_top), experts = max_over(pl, f_experts), pairs = T * top;
  uint32_t max_tiles = 0;
  for (const PlanLayer& l : pl.layers)
    if (l.mlp == FF_MOE && T) max_tiles = std::max(max_tiles, moe_max_tiles(l.moe, T));
  const size_t o_pTail = a.take((size_t)T * max_over(pl, f_tail) * 4);
  const size_t o_pG = a.take((size_t)pairs * H * as);
  const size_t o_pFE = a.take((size_t)T * max_over(pl, f_sorted_ff) * as);
  const size_t o_pYE = a.take((size_t)pairs * H * 4);
  const size_t o_ids = a.take((size_t)pairs * 4), o_rw = a.take((size_t)pairs * 4), o_where = a.take((size_t)pairs * 4), o_src = a.take((size_t)pairs * 4);
  const size_t o_erows = a.take((size_t)(experts + 1) * 4), o_tiles = a.take((size_t)max_tiles * sizeof(uint2)), o_ntiles = a.take(16);
  const size_t o_tok = a.take((size_t)T * 4 + 16);
  const size_t o_rows = a.take((size_t)T * 4 + 16);
  P->logit_rows = T ? std::min<uint32_t>(T, 64) : 0;
  const size_t o_lg = a.take((size_t)P->logit_rows * hp.V * 4);
  cudaError_t e = cudaMalloc((void**)&m->rarena, a.off);
  if (e != cudaSuccess) return fail(c, NFAI_ERR_OOM, "cudaMalloc of %zu run-time bytes (caches, states, workspaces): %s", a.off, cudaGetErrorString(e));
  CU(c, cudaMemsetAsync(m->rarena, 0, a.off, c->stream));
  bind_common(m, common);
  char* base = m->rarena;
  P->st.resize(hp.L);
  for (uint32_t i = 0; i < hp.L; ++i) {
    LayerState& s = P->st[i];
    if (pl.layers[i].mixer == MIXER_LATENT) {
      s.c = base + off[i].c;
      s.kr = base + off[i].kr;
      s.scratch = base + off[i].scratch;
      s.rope = (float2*)(base + off[i].rope);
    } else if (pl.layers[i].mixer == MIXER_GQA) {
      const GqaSpec& g = pl.layers[i].gqa;
      s.k = g.own_kv() ? base + off[i].k : P->st[(size_t)g.kv_from].k;  // (an earlier layer)
      s.v = g.own_kv() ? base + off[i].v : P->st[(size_t)g.kv_from].v;
      s.scratch = base + off[i].scratch;
    } else {
      s.ring = (float*)(base + off[i].ring);
      s.S = (float*)(base + off[i].S);
    }
  }
  P->X = (float*)(base + o_X);
  P->u = (float*)(base + o_u);
  P->mix = (float*)(base + o_mix);
  P->ao = (float*)(base + o_ao);
  P->hbuf = (float*)(base + o_h);
  P->y = (float*)(base + o_y);
  P->tail = (float*)(base + o_tail);
  P->chosen = (uint32_t*)(base + o_chosen);
  P->freq = pl.sinusoid_base > 0.f ? (double*)(base + o_freq) : nullptr;
  P->pTail = (float*)(base + o_pTail);
  P->pG = base + o_pG;
  P->pFE = base + o_pFE;
  P->pYE = (float*)(base + o_pYE);
  P->pRoute.ids = (uint32_t*)(base + o_ids);
  P->pRoute.w = (float*)(base + o_rw);
  P->pRoute.where = (uint32_t*)(base + o_where);
  P->pRoute.src = (uint32_t*)(base + o_src);
  P->pRoute.rows = (uint32_t*)(base + o_erows);
  P->pRoute.tiles = (uint2*)(base + o_tiles);
  P->pRoute.n_tiles = (uint32_t*)(base + o_ntiles);
  P->pX = (float*)(base + o_pX);
  P->pA = base + o_pA;
  P->pIn = (float*)(base + o_pIn);
  P->pQ = base + o_pQ;
  P->pKV = base + o_pKV;
  P->pY = (float*)(base + o_pY);
  P->pF = base + o_pF;
  P->pXBC = base + o_pXBC;
  P->pDT = (float*)(base + o_pDT);
  P->pSY = (float*)(base + o_pSY);
  P->pChunk = chunk_floats ? (float*)(base + o_pC) : nullptr;
  P->pChunkFloats = chunk_floats;
  P->pPart = part ? (float*)(base + o_pp) : nullptr;
  P->pPartFloats = part;
  P->pTok = (uint32_t*)(base + o_tok);
  P->pRows = (uint32_t*)(base + o_rows);
  P->pLogits = (float*)(base + o_lg);
  CU(c, cudaStreamSynchronize(c->stream));
  // angles in float32 (position times frequency), their cosine and sine from the host's double-precision library
  for (const auto& r : ropes) {
    const uint32_t dims = r.first.first, half = dims / 2;
    if (!half) continue;
    std::vector<float> f(half);
    for (uint32_t i = 0; i < half; ++i) f[i] = (float)std::pow((double)r.first.second, -2.0 * i / dims);
    std::vector<float2> tab((size_t)hp.ctx * half);
    for (uint32_t p = 0; p < hp.ctx; ++p)
      for (uint32_t i = 0; i < half; ++i) {
        const float angle = (float)p * f[i];
        tab[(size_t)p * half + i] = make_float2((float)std::cos((double)angle), (float)std::sin((double)angle));
      }
    CU(c, cudaMemcpy(base + r.second, tab.data(), tab.size() * sizeof(float2), cudaMemcpyHostToDevice));
  }
  if (P->freq) {
    std::vector<double> f((H + 1) / 2);
    for (uint32_t i = 0; i < f.size(); ++i) f[i] = std::pow((double)pl.sinusoid_base, -2.0 * i / H);
    CU(c, cudaMemcpy(P->freq, f.data(), f.size() * sizeof(double), cudaMemcpyHostToDevice));
  }
  CU(c, cudaHostAlloc((void**)&m->pin_logits, (size_t)hp.V * 4, cudaHostAllocDefault));
  if (P->logit_rows) CU(c, cudaHostAlloc((void**)&P->pin_rows, (size_t)P->logit_rows * hp.V * 4, cudaHostAllocDefault));
  int rc = capture_graphs(m);
  if (rc) return rc;
  m->pos = 0;
  m->finalized = true;
  return NFAI_OK;
}

// ---- decode step ----------------------------------------------------------------------------------------------------------------
namespace {

// Who reads the streams after sublayer (layer, q): the weights of that read; null = the plain sum (the output).
const float* next_reader(nfai_model* m, uint32_t layer, int q) {
  PlanModel* P = m->plan.get();
  if (q == 0 && P->plan.layers[layer].has_mlp()) return P->w[layer].sub[1].in.ptr;
  if (layer + 1 < m->hp.L) return P->w[layer + 1].sub[0].in.ptr;
  return P->ones.ptr;
}

bool post_norm(const nfai_model* m) { return m->plan->plan.residual == RESIDUAL_POST_NORM; }

// How the sublayer behind sublayer (layer, q), number `sub` of the model, finds its input: the residual before that sublayer
// and what to add to it; it keeps the sum.
void behind(nfai_model* m, GemvParams& p, uint32_t layer, int q, uint32_t sub) {
  PlanModel* P = m->plan.get();
  p.form = FORM_POST_NORM;
  p.x = streams(m, sub);
  p.post.y = P->y;
  p.post.gain = P->w[layer].sub[q].norm.ptr;
  p.post.mult = P->plan.residual_mult;
  p.post.eps = m->hp.eps;
  p.post.store = streams(m, sub + 1);
}

// Input of sublayer (l, q), number `sub`.
void reader(nfai_model* m, GemvParams& p, uint32_t l, int q, uint32_t sub) {
  PlanModel* P = m->plan.get();
  p.K = m->hp.H;
  if (!post_norm(m)) {
    p.x = P->u;
    p.gain = P->w[l].sub[q].norm.ptr;
    p.eps = m->hp.eps;
  } else if (sub == 0) {
    p.form = FORM_POST_NORM;
    p.x = streams(m, 0);
  } else {
    if (q) behind(m, p, l, 0, sub - 1);
    else behind(m, p, l - 1, P->plan.layers[l - 1].has_mlp() ? 1 : 0, sub - 1);
  }
}

GemvParams in_params(nfai_model* m, uint32_t l, uint32_t sub) {
  PlanModel* P = m->plan.get();
  const PlanLayer& pl = P->plan.layers[l];
  GemvParams p;
  p.W = P->w[l].in.ptr;
  p.N = pl.in_rows();
  reader(m, p, l, 0, sub);
  p.state = m->state;
  if (pl.mixer == MIXER_SSM) {
    p.y = P->st[l].ring;
    p.y_ring = pl.ssm.taps;
    p.y_stride = pl.ssm.in_rows();
  } else {
    p.y = P->mix;
    p.bias = P->w[l].in_b.ptr;
  }
  return p;
}

// Where the output of sublayer (l, q) goes.
GemvEpilogue out_epilogue(const nfai_model* m) { return post_norm(m) ? EPI_STORE : EPI_HYPER; }
void writer(nfai_model* m, GemvParams& p, uint32_t l, int q, uint32_t sub) {
  PlanModel* P = m->plan.get();
  p.N = m->hp.H;
  if (post_norm(m)) {
    p.y = P->y;
    return;
  }
  const SubW& w = P->w[l].sub[q];
  p.hyper.S = P->plan.streams;
  p.hyper.x_in = streams(m, sub);
  p.hyper.x_out = streams(m, sub + 1);
  p.hyper.mix = w.mix.ptr;
  p.hyper.out = w.out.ptr;
  p.hyper.next_in = next_reader(m, l, q);
  p.hyper.u = P->u;
}

GemvParams out_params(nfai_model* m, uint32_t l, uint32_t sub) {
  PlanModel* P = m->plan.get();
  const PlanLayer& pl = P->plan.layers[l];
  GemvParams p;
  p.W = P->w[l].out.ptr;
  p.K = pl.out_cols();
  p.x = P->ao;
  p.bias = P->w[l].out_b.ptr;
  if (pl.mixer == MIXER_SSM) {
    p.gain = P->w[l].ssm_norm.ptr;
    p.eps = m->hp.eps;
    p.norm_groups = pl.ssm.norm_groups;
  }
  writer(m, p, l, 0, sub);
  return p;
}

GemvParams gateup_params(nfai_model* m, uint32_t l, uint32_t sub) {
  PlanModel* P = m->plan.get();
  GemvParams p;
  p.W = P->w[l].gateup.ptr;
  p.N = 2 * P->plan.layers[l].ff;
  reader(m, p, l, 1, sub);
  p.bias = P->w[l].gateup_b.ptr;
  p.act = P->plan.act;
  p.act_limit = P->plan.layers[l].limit;
  p.y = P->hbuf;
  return p;
}

GemvParams down_params(nfai_model* m, uint32_t l, uint32_t sub) {
  PlanModel* P = m->plan.get();
  GemvParams p;
  p.W = P->w[l].down.ptr;
  p.K = P->plan.layers[l].ff;
  p.x = P->hbuf;
  p.bias = P->w[l].down_b.ptr;
  writer(m, p, l, 1, sub);
  return p;
}

// Routed feed-forward: the shared hidden values and the router's logits (and the shared feed-forward's gate behind them) ...
GemvEpilogue first_epilogue(const MoeSpec& s) { return s.shared_ff ? EPI_GATED : EPI_STORE; }
GemvParams first_params(nfai_model* m, uint32_t l, uint32_t sub) {
  PlanModel* P = m->plan.get();
  const MoeSpec& s = P->plan.layers[l].moe;
  GemvParams p;
  p.W = P->w[l].first.ptr;
  p.N = s.first_rows();
  reader(m, p, l, 1, sub);
  p.act = P->plan.act;
  p.act_limit = s.shared_limit;
  p.gated_rows = s.gated_rows();
  p.tail = P->tail;
  p.y = s.shared_ff ? P->hbuf + (size_t)s.top * s.ff : P->tail;
  return p;
}
Router router_of(nfai_model* m, uint32_t l) {
  const MoeSpec& s = m->plan->plan.layers[l].moe;
  Router r;
  r.correction = m->plan->w[l].correction.ptr;
  r.experts = s.experts;
  r.top = s.top;
  r.groups = s.groups;
  r.keep = s.keep;
  r.scale = s.scale;
  return r;
}
// ... the hidden values of the chosen experts, times their weights ...
GemvParams expert_params(nfai_model* m, uint32_t l, uint32_t sub) {
  PlanModel* P = m->plan.get();
  const MoeSpec& s = P->plan.layers[l].moe;
  GemvParams p;
  p.W = P->w[l].exp_gateup.ptr;
  p.N = s.top * 2 * s.ff;
  p.K = m->hp.H;
  p.x = streams(m, sub);  // kept by the kernel of first_params
  p.act = P->plan.act;
  p.act_limit = s.limit;
  p.y = P->hbuf;
  p.form = FORM_EXPERT_ROWS;
  p.expert.router = router_of(m, l);
  p.expert.logits = P->tail;
  p.expert.rows = 2 * s.ff;
  p.expert.chosen = P->chosen;
  return p;
}
// ... and one product over all of them.
GemvParams expert_down_params(nfai_model* m, uint32_t l, uint32_t sub) {
  PlanModel* P = m->plan.get();
  const MoeSpec& s = P->plan.layers[l].moe;
  GemvParams p;
  p.W = P->w[l].exp_down.ptr;
  p.K = s.hidden();
  p.x = P->hbuf;
  p.form = FORM_EXPERT_COLUMNS;
  p.expert.chosen = P->chosen;
  p.expert.seg = s.ff;
  p.expert.top = s.top;
  p.expert.W2 = P->w[l].shared_down.ptr;
  p.expert.shared_gate = P->tail + s.experts;
  writer(m, p, l, 1, sub);
  return p;
}

GqaParams gqa_params(nfai_model* m, uint32_t l) {
  PlanModel* P = m->plan.get();
  GqaParams p;
  p.spec = P->plan.layers[l].gqa;
  p.eps = m->hp.eps;
  p.k_cache = P->st[l].k;
  p.v_cache = P->st[l].v;
  p.dtype = P->act_dtype;
  p.ctx = m->hp.ctx;
  p.part = (float*)P->st[l].scratch;
  return p;
}

LatentParams latent_params(nfai_model* m, uint32_t l) {
  PlanModel* P = m->plan.get();
  LatentParams p;
  p.spec = P->plan.layers[l].latent;
  p.lat_gain = P->w[l].lat_norm.ptr;
  p.eps = m->hp.eps;
  p.rope_cs = P->st[l].rope;
  p.Wkv = P->w[l].kv.ptr;
  p.c_cache = P->st[l].c;
  p.kr_cache = P->st[l].kr;
  p.dtype = P->act_dtype;
  p.ctx = m->hp.ctx;
  p.scratch = P->st[l].scratch;
  return p;
}

SsmParams ssm_params(nfai_model* m, uint32_t l) {
  PlanModel* P = m->plan.get();
  const LayerWeights& w = P->w[l];
  SsmParams p;
  p.spec = P->plan.layers[l].ssm;
  p.ring = P->st[l].ring;
  p.conv_w = w.conv.ptr;
  p.conv_b = w.conv_b.ptr;
  p.dt_bias = w.dt_bias.ptr;
  p.A_log = w.A_log.ptr;
  p.D = w.D.ptr;
  p.S = P->st[l].S;
  return p;
}

cudaError_t launch_mixer_step(nfai_model* m, uint32_t l, bool pdl, int* launches) {
  PlanModel* P = m->plan.get();
  if (P->plan.layers[l].mixer == MIXER_LATENT) {
    LatentParams p = latent_params(m, l);
    p.in = P->mix;
    p.state = m->state;
    p.out = P->ao;
    return launch_latent_decode(m->ctx->stream, p, pdl, launches);
  }
  if (P->plan.layers[l].mixer == MIXER_GQA) {
    GqaParams p = gqa_params(m, l);
    p.in = P->mix;
    p.state = m->state;
    p.out = P->ao;
    if (launches) ++*launches;
    return launch_gqa_decode(m->ctx->stream, p, pdl);
  }
  SsmParams p = ssm_params(m, l);
  p.state = m->state;
  p.y = P->ao;
  if (launches) ++*launches;
  return launch_ssm_step(m->ctx->stream, p, pdl);
}

}  // namespace

GemvParams plan_head_params(nfai_model* m, bool settled) {
  const LayerPlan& pl = m->plan->plan;
  GemvParams p;
  p.W = m->head.ptr;
  p.N = m->hp.V;
  p.K = m->hp.H;
  p.x = m->plan->u;
  if (post_norm(m)) {
    const uint32_t last = pl.sublayers();
    p.form = FORM_POST_NORM;
    if (settled) p.x = streams(m, last);
    else behind(m, p, m->hp.L - 1, pl.layers.back().has_mlp() ? 1 : 0, last - 1);
  }
  p.gain = m->out_norm.ptr;
  p.gain_stride = pl.scalar_norms ? 0 : 1;
  p.eps = m->hp.eps;
  p.y = m->logits;
  p.part_val = m->part_val;
  p.part_idx = m->part_idx;
  return p;
}

cudaError_t plan_record_step(nfai_model* m, bool with_head, bool from_prompt, int* launches) {
  nfai_ctx* c = m->ctx;
  PlanModel* P = m->plan.get();
  const nfai_hparams& hp = m->hp;
  cudaStream_t s = c->stream;
  const bool pdl = c->pdl;
  const int wdt = hp.weight_dtype;
  int n = 0;
  cudaError_t e;
#define STEP(call)                 \
  do {                             \
    e = (call);                    \
    if (e != cudaSuccess) return e; \
    ++n;                           \
  } while (0)
  // the first kernel of a step must not overlap the previous step's tail: plain launch
  if (post_norm(m))
    STEP(launch_embed_position(s, wdt, m->embd.ptr, hp.H, hp.V, m->state, from_prompt ? m->prompt : nullptr, P->freq, streams(m, 0), false));
  else
    STEP(launch_embed_streams(s, wdt, m->embd.ptr, hp.H, hp.V, P->plan.streams, m->state, from_prompt ? m->prompt : nullptr,
                              P->w[0].sub[0].in.ptr, streams(m, 0), P->u, false));
  const GemvEpilogue out = out_epilogue(m);
  uint32_t sub = 0;
  for (uint32_t l = 0; l < hp.L; ++l) {
    const PlanLayer& pl = P->plan.layers[l];
    STEP(launch_gemv(s, wdt, 0, EPI_STORE, in_params(m, l, sub), m->tune_qkv, pdl));
    if ((e = launch_mixer_step(m, l, pdl, &n)) != cudaSuccess) return e;
    STEP(launch_gemv(s, wdt, 0, out, out_params(m, l, sub++), m->tune_o, pdl));
    if (pl.mlp == FF_DENSE) {
      STEP(launch_gemv(s, wdt, 0, EPI_GATED, gateup_params(m, l, sub), m->tune_gateup, pdl));
      STEP(launch_gemv(s, wdt, 0, out, down_params(m, l, sub++), m->tune_down, pdl));
    } else if (pl.mlp == FF_MOE) {
      STEP(launch_gemv(s, wdt, 0, first_epilogue(pl.moe), first_params(m, l, sub), m->tune_gateup, pdl));
      STEP(launch_gemv(s, wdt, 0, EPI_GATED, expert_params(m, l, sub), m->tune_gateup, pdl));
      STEP(launch_gemv(s, wdt, 0, out, expert_down_params(m, l, sub++), m->tune_down, pdl));
    }
  }
  if (with_head) {
    STEP(launch_gemv(s, wdt, 0, EPI_LOGITS, plan_head_params(m), m->tune_head, pdl));
    STEP(launch_argmax_final(s, m->part_val, m->part_idx, m->nparts, m->state, nullptr, m->history, hp.ctx, PrefetchPlan(),
                             nullptr, 0, XchgHooks(), pdl));
  } else {
    STEP(launch_advance(s, m->state, nullptr, 0, pdl));
  }
#undef STEP
  if (launches) *launches = n;
  if (with_head) P->step_launches = n;
  return cudaSuccess;
}

// (without graphs: known after the first recorded step)
int plan_step_launches(const nfai_model* m) { return m->plan->step_launches; }

bool plan_rewinds(const nfai_model* m) {
  for (const PlanLayer& l : m->plan->plan.layers)
    if (l.mixer == MIXER_SSM) return false;
  return true;
}

// ---- prompt passes ----------------------------------------------------------------------------------------------------------------
bool plan_batched(const nfai_model* m) { return m->plan->batched && m->plan->chunk >= 2; }

namespace {

cudaError_t product(nfai_model* m, const void* A, const void* W, uint32_t M, uint32_t N, uint32_t K, GemmEpilogue ep) {
  PlanModel* P = m->plan.get();
  cudaStream_t s = m->ctx->stream;
  ep.out_dtype = P->act_dtype;
  if (P->act_dtype == NFAI_BF16 && K % 8 == 0 && (((uintptr_t)A | (uintptr_t)W) & 15) == 0) {
    ep.operands_bf16 = 1;
    ep.scratch = P->pPart;
    ep.scratch_floats = P->pPartFloats;
    return launch_gemm_tc(s, (const __half*)A, (const __half*)W, M, N, K, ep, &m->state->err);
  }
  return launch_gemm_simt(s, P->act_dtype, A, W, M, N, K, ep);
}

cudaError_t mixer_pass(nfai_model* m, uint32_t l, uint32_t pos0, uint32_t T) {
  PlanModel* P = m->plan.get();
  cudaStream_t s = m->ctx->stream;
  const PlanLayer& pl = P->plan.layers[l];
  const LayerWeights& w = P->w[l];
  cudaError_t e;
  GemmEpilogue ei;
  ei.kind = GEMM_EPI_STORE;
  ei.out_f32 = P->pIn;
  ei.bias = w.in_b.ptr;
  if ((e = product(m, P->pA, w.in.ptr, T, pl.in_rows(), m->hp.H, ei)) != cudaSuccess) return e;
  if (pl.mixer == MIXER_LATENT) {
    LatentParams p = latent_params(m, l);
    p.in = P->pIn;
    p.in_ld = pl.in_rows();
    p.pos0 = pos0;
    p.q = P->pQ;
    p.kv = P->pKV;
    p.ao = P->pA;
    p.kv_pos0 = pl.latent.window && pos0 + 1 > pl.latent.window ? pos0 + 1 - pl.latent.window : 0;
    if ((e = launch_latent_prep(s, p, T)) != cudaSuccess) return e;
    // keys and values of every latent the portion's windows reach
    GemmEpilogue ek;
    ek.kind = GEMM_EPI_STORE_ACT;
    ek.out_act = P->pKV;
    const char* rows = P->st[l].c + (size_t)p.kv_pos0 * pl.latent.rank * dtype_size(P->act_dtype);
    if ((e = product(m, rows, w.kv.ptr, pos0 + T - p.kv_pos0, f_kv(pl), pl.latent.rank, ek)) != cudaSuccess) return e;
    return launch_latent_prefill(s, p, T);
  }
  if (pl.mixer == MIXER_GQA) {
    GqaParams p = gqa_params(m, l);
    p.in = P->pIn;
    p.in_ld = pl.in_rows();
    p.pos0 = pos0;
    p.q = P->pQ;
    p.ao = P->pA;
    if ((e = launch_gqa_prep(s, p, T)) != cudaSuccess) return e;
    return launch_gqa_prefill(s, p, T);
  }
  SsmParams p = ssm_params(m, l);
  p.in = P->pIn;
  p.pos0 = pos0;
  p.y = P->pSY;
  p.xbc = P->pXBC;
  p.xbc_dtype = P->act_dtype;
  p.dt = P->pDT;
  p.chunk = P->pChunk;
  p.chunk_floats = P->pChunkFloats;
  if ((e = launch_ssm_prefill(s, p, T)) != cudaSuccess) return e;
  return launch_group_norm_rows(s, P->pSY, w.ssm_norm.ptr, m->hp.eps, pl.ssm.norm_groups, T, pl.ssm.inner(), P->pA, P->act_dtype);
}

cudaError_t grouped_product(nfai_model* m, const void* A, const void* W, uint32_t max_rows, uint32_t N, uint32_t K, const GemmGroups& g, GemmEpilogue ep) {
  PlanModel* P = m->plan.get();
  cudaStream_t s = m->ctx->stream;
  ep.out_dtype = P->act_dtype;
  if (P->act_dtype == NFAI_BF16 && K % 8 == 0 && (((uintptr_t)A | (uintptr_t)W) & 15) == 0) {
    ep.operands_bf16 = 1;
    return launch_gemm_tc_grouped(s, (const __half*)A, (const __half*)W, max_rows, N, K, g, ep, &m->state->err);
  }
  return launch_gemm_simt_grouped(s, P->act_dtype, A, W, N, K, g, ep);
}

// The routed feed-forward of T rows of P->pA up to its expert rows (sorted, P->pYE) and shared rows (P->pY); their weighted
// sum is formed where the residual is written.
cudaError_t moe_pass(nfai_model* m, uint32_t l, uint32_t T) {
  PlanModel* P = m->plan.get();
  cudaStream_t s = m->ctx->stream;
  const MoeSpec& sp = P->plan.layers[l].moe;
  const LayerWeights& w = P->w[l];
  const uint32_t H = m->hp.H;
  cudaError_t e;
  GemmEpilogue ef;
  ef.kind = sp.shared_ff ? GEMM_EPI_GATED_CLAMPED : GEMM_EPI_STORE;
  ef.act_limit = sp.shared_limit;
  ef.gated_cols = sp.gated_rows();
  ef.out_act = P->pF;
  ef.out_f32 = P->pTail;
  if ((e = product(m, P->pA, w.first.ptr, T, sp.first_rows(), H, ef)) != cudaSuccess) return e;
  MoeRows r = P->pRoute;
  r.router = router_of(m, l);
  r.logits = P->pTail;
  r.ld = sp.first_rows() - sp.gated_rows();
  if ((e = launch_moe_route(s, r, T)) != cudaSuccess) return e;
  const uint32_t pairs = T * sp.top;
  if ((e = launch_moe_gather(s, P->pA, r.src, pairs, H, (uint32_t)dtype_size(P->act_dtype), P->pG)) != cudaSuccess) return e;
  GemmGroups g;
  g.count = sp.experts;
  g.rows = r.rows;
  g.tiles = r.tiles;
  g.n_tiles = r.n_tiles;
  g.max_tiles = moe_max_tiles(sp, T);
  GemmEpilogue eg;
  eg.kind = GEMM_EPI_GATED_CLAMPED;
  eg.act_limit = sp.limit;
  eg.out_act = P->pFE;
  if ((e = grouped_product(m, P->pG, w.exp_gateup.ptr, pairs, 2 * sp.ff, H, g, eg)) != cudaSuccess) return e;
  GemmEpilogue ed;
  ed.kind = GEMM_EPI_STORE;
  ed.out_f32 = P->pYE;
  if ((e = grouped_product(m, P->pFE, w.exp_down.ptr, pairs, H, sp.ff, g, ed)) != cudaSuccess) return e;
  if (!sp.shared_ff) return cudaSuccess;
  ed.out_f32 = P->pY;
  return product(m, P->pF, w.shared_down.ptr, T, H, sp.shared_ff, ed);
}

cudaError_t mlp_pass(nfai_model* m, uint32_t l, uint32_t T) {
  PlanModel* P = m->plan.get();
  const PlanLayer& pl = P->plan.layers[l];
  const LayerWeights& w = P->w[l];
  const uint32_t H = m->hp.H;
  if (pl.mlp == FF_MOE) return moe_pass(m, l, T);
  GemmEpilogue eg;
  eg.kind = P->plan.act == ACT_CLAMPED ? GEMM_EPI_GATED_CLAMPED : GEMM_EPI_GATED;
  eg.act = P->plan.act;
  eg.act_limit = pl.limit;
  eg.bias = w.gateup_b.ptr;
  eg.out_act = P->pF;
  cudaError_t e = product(m, P->pA, w.gateup.ptr, T, 2 * pl.ff, H, eg);
  if (e != cudaSuccess) return e;
  GemmEpilogue ed;
  ed.kind = GEMM_EPI_STORE;
  ed.out_f32 = P->pY;
  ed.bias = w.down_b.ptr;
  return product(m, P->pF, w.down.ptr, T, H, pl.ff, ed);
}

HyperRows hyper_rows(nfai_model* m) {
  PlanModel* P = m->plan.get();
  HyperRows h;
  h.S = P->plan.streams;
  h.H = m->hp.H;
  h.eps = m->hp.eps;
  h.normed = P->pA;
  h.normed_dtype = P->act_dtype;
  return h;
}
PostRows post_rows(nfai_model* m) {
  PlanModel* P = m->plan.get();
  PostRows r;
  r.H = m->hp.H;
  r.eps = m->hp.eps;
  r.operand = P->pA;
  r.operand_dtype = P->act_dtype;
  return r;
}

// Rows of the residual for the tokens in P->pTok, and the first sublayer's operand.
cudaError_t begin_rows(nfai_model* m, uint32_t pos0, uint32_t T) {
  PlanModel* P = m->plan.get();
  if (post_norm(m)) {
    PostRows r = post_rows(m);
    r.tokens = P->pTok;
    r.embed = m->embd.ptr;
    r.embed_dtype = m->hp.weight_dtype;
    r.freq = P->freq;
    r.pos0 = pos0;
    r.X_out = P->pX;
    return launch_post_rows(m->ctx->stream, r, T);
  }
  HyperRows h = hyper_rows(m);
  h.X_out = P->pX;
  h.tokens = P->pTok;
  h.embed = m->embd.ptr;
  h.embed_dtype = m->hp.weight_dtype;
  h.next_in = P->w[0].sub[0].in.ptr;
  h.gain = P->w[0].sub[0].norm.ptr;
  return launch_hyper_rows(m->ctx->stream, h, T);
}

// Write the output of sublayer (l, q), number `sub`, into the rows and form the next sublayer's operand. `tap`: keep the last
// token's residual where a decode step would.
cudaError_t close_rows(nfai_model* m, uint32_t l, int q, uint32_t sub, uint32_t T, bool tap) {
  PlanModel* P = m->plan.get();
  cudaStream_t s = m->ctx->stream;
  const SubW& w = P->w[l].sub[q];
  const PlanLayer& pl = P->plan.layers[l];
  const bool end = l + 1 == m->hp.L && (q == 1 || !pl.has_mlp());  // only the wanted rows go on from here
  if (post_norm(m)) {
    PostRows r = post_rows(m);
    r.X = r.X_out = P->pX;
    r.y = P->pY;
    r.gain = w.norm.ptr;
    r.mult = P->plan.residual_mult;
    if (q == 1 && pl.mlp == FF_MOE) {
      const MoeSpec& sp = pl.moe;
      if (!sp.shared_ff) r.y = nullptr;
      r.moe_top = sp.top;
      r.ye = P->pYE;
      r.where = P->pRoute.where;
      r.w = P->pRoute.w;
      r.shared_gate = P->pTail + sp.experts;
      r.shared_ld = sp.first_rows() - sp.gated_rows();
    }
    if (end) r.operand = nullptr;
    if (tap) {
      r.tap = streams(m, sub + 1);
      r.tap_row = T - 1;
    }
    return launch_post_rows(s, r, T);
  }
  const uint32_t S = P->plan.streams, H = m->hp.H;
  HyperRows h = hyper_rows(m);
  h.X = h.X_out = P->pX;
  h.y = P->pY;
  h.mix = w.mix.ptr;
  h.out = w.out.ptr;
  h.next_in = next_reader(m, l, q);
  if (end) h.normed = nullptr;
  else h.gain = q == 0 && pl.has_mlp() ? P->w[l].sub[1].norm.ptr : P->w[l + 1].sub[0].norm.ptr;
  cudaError_t e = launch_hyper_rows(s, h, T);
  if (e == cudaSuccess && tap)
    e = cudaMemcpyAsync(streams(m, sub + 1), P->pX + (size_t)(T - 1) * S * H, (size_t)S * H * 4, cudaMemcpyDeviceToDevice, s);
  return e;
}

// Operand of the output matrix for R rows of the residual (P->pRows).
cudaError_t head_rows(nfai_model* m, uint32_t R) {
  PlanModel* P = m->plan.get();
  if (post_norm(m)) {
    PostRows r = post_rows(m);
    r.X = P->pX;
    r.rows = P->pRows;
    r.norm_gain = m->out_norm.ptr;
    return launch_post_rows(m->ctx->stream, r, R);
  }
  HyperRows h = hyper_rows(m);
  h.X = P->pX;
  h.rows = P->pRows;
  h.next_in = P->ones.ptr;
  h.gain = m->out_norm.ptr;
  return launch_hyper_rows(m->ctx->stream, h, R);
}

}  // namespace

int plan_prefill(nfai_model* m, const uint32_t* tokens, int n, const uint32_t* want, int n_want, float* logits_out) {
  nfai_ctx* c = m->ctx;
  PlanModel* P = m->plan.get();
  const nfai_hparams& hp = m->hp;
  const uint32_t S = P->plan.streams, H = hp.H;
  cudaStream_t s = c->stream;
  uint32_t pos0 = m->pos;
  int done = 0, w_next = 0;
  while (done < n) {
    const uint32_t T = std::min<uint32_t>((uint32_t)(n - done), P->chunk);
    const bool last = done + (int)T == n;
    CU(c, cudaMemcpyAsync(P->pTok, tokens + done, (size_t)T * 4, cudaMemcpyHostToDevice, s));
    CU(c, begin_rows(m, pos0, T));
    uint32_t sub = 0;
    for (uint32_t l = 0; l < hp.L; ++l) {
      const PlanLayer& pl = P->plan.layers[l];
      CU(c, mixer_pass(m, l, pos0, T));
      GemmEpilogue eo;
      eo.kind = GEMM_EPI_STORE;
      eo.out_f32 = P->pY;
      eo.bias = P->w[l].out_b.ptr;
      CU(c, product(m, P->pA, P->w[l].out.ptr, T, H, pl.out_cols(), eo));
      CU(c, close_rows(m, l, 0, sub++, T, last));
      if (!pl.has_mlp()) continue;
      CU(c, mlp_pass(m, l, T));
      CU(c, close_rows(m, l, 1, sub++, T, last));
    }
    // logits of the wanted places of this pass
    while (w_next < n_want && (int)want[w_next] < done + (int)T) {
      std::vector<uint32_t> rows;
      const int w0 = w_next;
      while (w_next < n_want && (int)want[w_next] < done + (int)T && rows.size() < P->logit_rows) rows.push_back(want[w_next++] - (uint32_t)done);
      const uint32_t R = (uint32_t)rows.size();
      CU(c, cudaMemcpyAsync(P->pRows, rows.data(), (size_t)R * 4, cudaMemcpyHostToDevice, s));
      CU(c, head_rows(m, R));
      GemmEpilogue eh;
      eh.kind = GEMM_EPI_STORE;
      eh.out_f32 = P->pLogits;
      CU(c, product(m, P->pA, m->head.ptr, R, hp.V, H, eh));
      CU(c, cudaMemcpyAsync(P->pin_rows, P->pLogits, (size_t)R * hp.V * 4, cudaMemcpyDeviceToHost, s));
      CU(c, cudaStreamSynchronize(s));
      memcpy(logits_out + (size_t)w0 * hp.V, P->pin_rows, (size_t)R * hp.V * 4);
    }
    if (last && !post_norm(m)) {  // what a decode step would read: the sum of the last token's streams
      HyperRows h;
      h.S = S;
      h.H = H;
      h.X = P->pX + (size_t)(T - 1) * S * H;
      h.next_in = P->ones.ptr;
      h.u_out = P->u;
      CU(c, launch_hyper_rows(s, h, 1));
    }
    pos0 += T;
    done += (int)T;
  }
  int rc = set_state_word(m, offsetof(StepState, pos), pos0 - 1, 3);
  if (rc) return rc;
  CU(c, launch_gemv(s, hp.weight_dtype, 0, EPI_LOGITS, plan_head_params(m, true), m->tune_head, false));
  CU(c, launch_argmax_final(s, m->part_val, m->part_idx, m->nparts, m->state, nullptr, m->history, hp.ctx, PrefetchPlan(), nullptr,
                            0, XchgHooks(), false));
  return NFAI_OK;
}

// ---- snapshots and taps ---------------------------------------------------------------------------------------------------------
namespace {
// Visit every piece of state a later turn needs: (address, bytes).
template <typename F>
void each_state(const nfai_model* m, uint32_t pos, F&& f) {
  const PlanModel* P = m->plan.get();
  const size_t as = dtype_size(P->act_dtype);
  for (uint32_t i = 0; i < m->hp.L; ++i) {
    const PlanLayer& l = P->plan.layers[i];
    const LayerState& s = P->st[i];
    if (l.mixer == MIXER_LATENT) {
      f(s.c, (size_t)pos * l.latent.rank * as);
      f(s.kr, (size_t)pos * l.latent.rot * as);
    } else if (l.mixer == MIXER_GQA) {
      if (!l.gqa.own_kv()) continue;
      f(s.k, (size_t)pos * l.gqa.k_cols() * as);
      f(s.v, (size_t)pos * l.gqa.v_cols() * as);
    } else {
      f((char*)s.ring, (size_t)l.ssm.taps * l.ssm.in_rows() * 4);
      f((char*)s.S, (size_t)l.ssm.heads * l.ssm.vdim * l.ssm.state * 4);
    }
  }
}
}  // namespace

size_t plan_snapshot_bytes(const nfai_model* m, uint32_t pos) {
  size_t n = 0;
  each_state(m, pos, [&](char*, size_t b) { n += align_up(b, 16); });
  return n;
}

cudaError_t plan_snapshot_copy(nfai_model* m, uint32_t pos, char* buf, bool save) {
  cudaError_t e = cudaSuccess;
  each_state(m, pos, [&](char* p, size_t b) {
    if (b && e == cudaSuccess) e = cudaMemcpyAsync(save ? buf : p, save ? p : buf, b, cudaMemcpyDeviceToDevice, m->ctx->stream);
    buf += align_up(b, 16);
  });
  return e;
}

int plan_read_kv(nfai_model* m, uint32_t layer, uint32_t pos, float* k, float* v) {
  nfai_ctx* c = m->ctx;
  PlanModel* P = m->plan.get();
  if (layer >= m->hp.L || pos >= m->hp.ctx) return fail(c, NFAI_ERR_ARG, "layer or position out of range");
  const PlanLayer& l = P->plan.layers[layer];
  if (l.mixer == MIXER_SSM) return fail(c, NFAI_ERR_ARG, "layer %u has no key/value cache", layer);
  CU(c, cudaStreamSynchronize(c->stream));
  auto read = [&](const char* src, uint32_t n, float* out) -> int {
    if (!out) return NFAI_OK;
    if (P->act_dtype == NFAI_F32) {
      CU(c, cudaMemcpy(out, src + (size_t)pos * n * 4, (size_t)n * 4, cudaMemcpyDeviceToHost));
      return NFAI_OK;
    }
    std::vector<uint16_t> h(n);
    CU(c, cudaMemcpy(h.data(), src + (size_t)pos * n * 2, (size_t)n * 2, cudaMemcpyDeviceToHost));
    for (uint32_t i = 0; i < n; ++i) {
      const uint32_t bits = (uint32_t)h[i] << 16;
      memcpy(out + i, &bits, 4);
    }
    return NFAI_OK;
  };
  if (l.mixer == MIXER_GQA) {
    const int rk = read(P->st[layer].k, l.gqa.k_cols(), k);
    return rk ? rk : read(P->st[layer].v, l.gqa.v_cols(), v);
  }
  const int rc = read(P->st[layer].c, l.latent.rank, k);
  return rc ? rc : read(P->st[layer].kr, l.latent.rot, v);
}

int plan_read_hidden(nfai_model* m, uint32_t layer, float* out) {
  nfai_ctx* c = m->ctx;
  PlanModel* P = m->plan.get();
  const uint32_t S = P->plan.streams, H = m->hp.H;
  uint32_t sub = 0;
  for (uint32_t l = 0; l <= layer; ++l) sub += P->plan.layers[l].has_mlp() ? 2 : 1;
  std::vector<float> x((size_t)S * H);
  CU(c, cudaStreamSynchronize(c->stream));
  CU(c, cudaMemcpy(x.data(), streams(m, sub), x.size() * 4, cudaMemcpyDeviceToHost));
  for (uint32_t i = 0; i < H; ++i) {
    float a = 0.f;
    for (uint32_t t = 0; t < S; ++t) a += x[(size_t)t * H + i];
    out[i] = a;
  }
  return NFAI_OK;
}

// ---- profiling --------------------------------------------------------------------------------------------------------------------
namespace {
// Selectors of nfai_profile_kernel: 0 gate/up and 1 down of dense feed-forwards, 2 in-projection, 3 out-projection and
// 5 attention of attention layers, 4 LM head, 6 in-projection, 7 step and 8 out-projection of state space layers, 9 shared
// gate/up with router, 10 gate/up of the chosen experts and 11 down of routed feed-forwards. Launch i takes the i-th such layer.
bool profile_layer(nfai_model* m, int which, int iter, uint32_t* layer, uint32_t* sub_out) {
  PlanModel* P = m->plan.get();
  std::vector<std::pair<uint32_t, uint32_t>> hits;  // (layer, index of its mixer's sublayer)
  uint32_t sub = 0;
  for (uint32_t l = 0; l < m->hp.L; ++l) {
    const PlanLayer& pl = P->plan.layers[l];
    const bool ok = which <= 1 ? pl.mlp == FF_DENSE : which <= 5 ? pl.mixer != MIXER_SSM : which <= 8 ? pl.mixer == MIXER_SSM : pl.mlp == FF_MOE;
    if (ok) hits.emplace_back(l, sub);
    sub += pl.has_mlp() ? 2 : 1;
  }
  if (hits.empty()) return false;
  const auto& h = hits[(size_t)iter % hits.size()];
  *layer = h.first;
  *sub_out = h.second;
  return true;
}
}  // namespace

cudaError_t plan_profile_launch(nfai_model* m, int which, int iter) {
  cudaStream_t s = m->ctx->stream;
  const int wdt = m->hp.weight_dtype;
  if (which == 4) return launch_gemv(s, wdt, 0, EPI_LOGITS, plan_head_params(m), m->tune_head, false);
  uint32_t l = 0, sub = 0;
  if (!profile_layer(m, which, iter, &l, &sub)) return cudaErrorInvalidValue;
  const GemvEpilogue out = out_epilogue(m);
  switch (which) {
    case 0: return launch_gemv(s, wdt, 0, EPI_GATED, gateup_params(m, l, sub + 1), m->tune_gateup, false);
    case 1: return launch_gemv(s, wdt, 0, out, down_params(m, l, sub + 1), m->tune_down, false);
    case 2: case 6: return launch_gemv(s, wdt, 0, EPI_STORE, in_params(m, l, sub), m->tune_qkv, false);
    case 3: case 8: return launch_gemv(s, wdt, 0, out, out_params(m, l, sub), m->tune_o, false);
    case 9: return launch_gemv(s, wdt, 0, first_epilogue(m->plan->plan.layers[l].moe), first_params(m, l, sub + 1), m->tune_gateup, false);
    case 10: return launch_gemv(s, wdt, 0, EPI_GATED, expert_params(m, l, sub + 1), m->tune_gateup, false);
    case 11: return launch_gemv(s, wdt, 0, out, expert_down_params(m, l, sub + 1), m->tune_down, false);
    default: return launch_mixer_step(m, l, false, nullptr);
  }
}

uint64_t plan_profile_bytes(nfai_model* m, int which) {
  PlanModel* P = m->plan.get();
  const uint64_t ws = dtype_size(m->hp.weight_dtype), H = m->hp.H, S = P->plan.streams;
  if (which == 4) return (uint64_t)m->hp.V * H * ws + H * 4;
  uint32_t l = 0, sub = 0;
  if (!profile_layer(m, which, 0, &l, &sub)) return 0;
  const PlanLayer& pl = P->plan.layers[l];
  switch (which) {
    case 0: return 2ull * pl.ff * H * ws + H * 4;
    case 1: return H * pl.ff * ws + 2 * S * H * 4;
    case 2: case 6: return (uint64_t)pl.in_rows() * H * ws + H * 4;
    case 3: case 8: return H * pl.out_cols() * ws + 2 * S * H * 4;
    case 5: {
      if (pl.mixer == MIXER_GQA) return gqa_rows_read(pl.gqa, m->pos) * (pl.gqa.dim + pl.gqa.vdim) * ws;
      const uint64_t seen = pl.latent.window ? std::min<uint64_t>(pl.latent.window, (uint64_t)m->pos) : m->pos;
      return (uint64_t)pl.latent.heads * (pl.latent.dim + pl.latent.vdim) * pl.latent.rank * ws + seen * (pl.latent.rank + pl.latent.rot) * ws;
    }
    case 9: return (uint64_t)pl.moe.first_rows() * H * ws + 2 * H * 4;
    case 10: return 2ull * pl.moe.top * pl.moe.ff * H * ws + H * 4;
    case 11: return (uint64_t)pl.moe.hidden() * H * ws + H * 4;
    default: return 2ull * pl.ssm.heads * pl.ssm.vdim * pl.ssm.state * 4 + (uint64_t)pl.ssm.taps * pl.ssm.in_rows() * 4;
  }
}

}  // namespace nfai

// ---- C ABI ------------------------------------------------------------------------------------------------------------------------
extern "C" {

int nfai_config_probe(const char* config_json, size_t len, nfai_hparams* out, char* tensors_out, size_t cap, size_t* n_out,
                      char* err_out, size_t err_bytes) {
  if (err_out && err_bytes) err_out[0] = 0;
  LayerPlan plan;
  std::string err;
  if (!config_json || !plan_parse(config_json, len, &plan, &err)) {
    if (!config_json) err = "config is null";
    if (err_out && err_bytes) snprintf(err_out, err_bytes, "%s", err.c_str());
    return fail(nullptr, NFAI_ERR_ARG, "%s", err.c_str());
  }
  if (out) {
    *out = nfai_hparams();
    out->H = plan.width;
    out->L = (uint32_t)plan.layers.size();
    out->V = plan.vocab;
    out->eps = plan.eps;
    out->weight_dtype = out->kv_dtype = NFAI_BF16;
  }
  std::string list;
  for (const PlanTensor& t : plan_tensors(plan)) {
    list += t.name;
    for (uint64_t d : t.shape) list += " " + std::to_string(d);
    list += "\n";
  }
  if (n_out) *n_out = list.size();
  if (tensors_out) {
    if (cap <= list.size()) return fail(nullptr, NFAI_ERR_ARG, "the listing needs %zu bytes", list.size() + 1);
    memcpy(tensors_out, list.c_str(), list.size() + 1);
  }
  return NFAI_OK;
}

int nfai_model_create_from_config(nfai_ctx* c, const char* config_json, size_t len, uint32_t kv_cache_size, int weight_dtype,
                                  nfai_model** out) {
  if (!c) return fail(nullptr, NFAI_ERR_ARG, "ctx is null");
  if (!config_json || !out) return fail(c, NFAI_ERR_ARG, "null argument");
  *out = nullptr;
  LayerPlan plan;
  std::string err;
  if (!plan_parse(config_json, len, &plan, &err)) return fail(c, NFAI_ERR_ARG, "%s", err.c_str());
  return plan_create(c, std::move(plan), kv_cache_size, weight_dtype, out);
}

}  // extern "C"
