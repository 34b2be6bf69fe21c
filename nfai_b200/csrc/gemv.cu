// Batch-1 decode GEMV family: y = W * f(x) with fused prologue (RMSNorm) and epilogues (residual add,
// RoPE + KV-cache write, SiLU*up, logits + arg-max partials).
//
// The work is HBM-bound (one FMA per 2 or 4 weight bytes), so the kernel is a weight streamer:
//  * the grid is persistent: at most a few CTAs per SM, and every warp walks row blocks gw, gw + TW, gw + 2 TW ...
//    (R consecutive rows each) as ONE continuous stream, so the prologue is paid once per CTA and the loads of
//    the next row block are already in flight while the current one is reduced and stored;
//  * the lanes walk a row in 16-byte vectors (8 halves / 4 floats), 512 contiguous bytes per warp per row per
//    step; U steps are issued back to back and the next batch is requested before the current one is consumed,
//    so every lane keeps 2*U*R 16-byte loads in flight;
//  * the first batch is requested BEFORE the programmatic-dependency wait: the weights do not depend on the
//    previous kernel, so they stream while it drains and while this CTA normalises x;
//  * x (float32) sits in shared memory and is reused by all R rows of all warps; accumulation is float32;
//  * the row sum is finished with warp shuffles; lane 0 applies the epilogue.
// No tensor cores: with one right-hand side there is nothing for them to reuse.
//
// Reference arithmetic this replaces: NFAI.Vulkan.Shaders/MatrixMultiplyShader.cs:266-288 (one thread per
// output, serial k loop), RMSNormShader.cs:129-150, RoPEShader.cs:238-271, SiLUShader.cs:112-127,
// ElementWiseMultiplicationShader.cs:127-138, host residual adds at TransformerBlock.cs:151-161,174-181.
#include "gemv_kernel.cuh"

namespace nfai {

using namespace gemv_detail;

// gemv_bf16.cu
cudaError_t launch_gemv_more(int wdtype, GemvEpilogue epi, bool vec, int R, int U, dim3 grid, size_t smem, cudaStream_t s,
                             bool pdl, const GemvParams& p);
// gemv_post.cu, gemv_moe.cu
cudaError_t launch_gemv_post(int wdtype, GemvEpilogue epi, bool vec, int R, int U, dim3 grid, size_t smem, cudaStream_t s,
                             bool pdl, const GemvParams& p);
cudaError_t launch_gemv_experts(int wdtype, GemvEpilogue epi, bool vec, int R, int U, dim3 grid, size_t smem, cudaStream_t s,
                                bool pdl, const GemvParams& p);

namespace {

template <typename WT, typename KVT>
cudaError_t launch_e(GemvEpilogue epi, bool vec, int R, int U, dim3 grid, size_t smem, cudaStream_t s, bool pdl,
                     const GemvParams& p) {
  if (!vec) {
    switch (epi) {
      case EPI_STORE: return launch_k(gemv_scalar_kernel<WT, float, EPI_STORE>, grid, smem, s, pdl, p);
      case EPI_QKV_ROPE: return launch_k(gemv_scalar_kernel<WT, KVT, EPI_QKV_ROPE>, grid, smem, s, pdl, p);
      case EPI_GATED: return launch_k(gemv_scalar_kernel<WT, float, EPI_GATED>, grid, smem, s, pdl, p);
      case EPI_LOGITS: return launch_k(gemv_scalar_kernel<WT, float, EPI_LOGITS>, grid, smem, s, pdl, p);
      default: break;
    }
    return cudaErrorInvalidValue;
  }
  switch (epi) {
    case EPI_STORE: return launch_r<WT, float, EPI_STORE>(R, U, grid, smem, s, pdl, p);
    case EPI_QKV_ROPE: return launch_r<WT, KVT, EPI_QKV_ROPE>(R, U, grid, smem, s, pdl, p);
    case EPI_GATED: return launch_r<WT, float, EPI_GATED>(R, U, grid, smem, s, pdl, p);
    case EPI_LOGITS: return launch_r<WT, float, EPI_LOGITS>(R, U, grid, smem, s, pdl, p);
    default: break;
  }
  return cudaErrorInvalidValue;
}

bool vector_ok(int wdtype, const GemvParams& p) {
  const uint32_t ve = wdtype == 0 ? 4 : 8;
  if (p.form == FORM_EXPERT_COLUMNS && (p.expert.seg % ve != 0 || (reinterpret_cast<uintptr_t>(p.expert.W2) & 15) != 0)) return false;
  return p.K % ve == 0 && (reinterpret_cast<uintptr_t>(p.W) & 15) == 0;
}

int rows_per_warp(GemvEpilogue epi, bool vec, const GemvTune& t) {
  if (!vec) return 2;
  int R = t.rows_per_warp;
  if ((epi == EPI_QKV_ROPE || epi == EPI_GATED) && R < 2) R = 2;
  return R;
}

}  // namespace

static bool use_ring(int wdtype, GemvEpilogue epi, const GemvParams& p, const GemvTune& t) {
  if (t.mode != 1 || !vector_ok(wdtype, p)) return false;
  if (wdtype == 2 || epi == EPI_HYPER || p.norm_groups > 1 || p.y_ring || p.form) return false;
  return t.unroll >= 1 && t.unroll <= 4 && gemv_ring_smem(p, t.unroll) <= 227 * 1024;
}

// How many warps share one row block (1, 2, 4 or 8; returned as log2). A matrix with fewer row blocks than the
// persistent grid has warps (the down projections: 2 048-4 096 rows of 16-28 KB) leaves warps without work and the
// others with long serial rows; splitting K gives every warp the same amount and puts the whole matrix in flight at
// once. It is used only where it measured faster (the 1B model's down projection: 10.3 -> 9.0 us): rows of at least
// four batches, chunks of whole batches, at most half of the warps busy without it, and no more chunks than needed to
// cover the grid. Short rows and matrices with more rows stream best unsplit (3B down projection: 12.2 vs 13.4 us).
static uint32_t gemv_split_log2(int wdtype, bool vec, int R, const GemvParams& p, const GemvTune& t) {
  if (!vec) return 0;
  if (t.split == 1 || t.split == 2 || t.split == 4 || t.split == 8) return t.split == 1 ? 0 : t.split == 2 ? 1 : t.split == 4 ? 2 : 3;
  const uint32_t ve = wdtype == 0 ? 4 : 8;
  const uint32_t U = (uint32_t)t.unroll;
  const uint32_t per_lane = p.K / ve / 32;  // 16-byte vectors per lane per row
  const uint32_t nrb = (p.N + R - 1) / R;
  const uint32_t warps = (t.grid > 0 ? (uint32_t)t.grid : sm_count() * (uint32_t)(t.ctas_per_sm < 1 ? 1 : t.ctas_per_sm)) * kWarps;
  if (p.K % (ve * 32) != 0) return 0;
  if (2 * nrb > warps) {
    // Plenty of rows: a split does not add parallelism, but it can even out the last round. 8 192 row pairs on 2 368
    // warps are 3.46 rounds, i.e. four with 13.5 % of the warp slots idle; as 16 384 half rows they are 6.9 rounds
    // (1.4 % idle): 14.1 -> 13.8 us for the gate/up product of the 1B model, 605 -> 597 us per step.
    auto idle = [&](uint32_t tasks) {
      const uint32_t rounds = (tasks + warps - 1) / warps;
      return (float)(rounds * warps - tasks) / (float)(rounds * warps);
    };
    if (per_lane % (2 * U) == 0 && idle(nrb) > 0.08f && idle(2 * nrb) + 0.04f < idle(nrb)) return 1;  // halves of whole batches
    return 0;
  }
  if (per_lane < 4 * U) return 0;
  for (uint32_t sl = 1; sl <= 3; ++sl) {
    if ((per_lane % (U << sl)) != 0) break;  // chunks must stay whole batches
    if ((nrb << sl) >= warps) return sl;
  }
  return 0;
}

uint32_t gemv_grid(int wdtype, GemvEpilogue epi, const GemvParams& p, const GemvTune& t) {
  if (use_ring(wdtype, epi, p, t)) return gemv_ring_grid(p, t.ctas_per_sm);
  const bool vec = vector_ok(wdtype, p);
  const int R = rows_per_warp(epi, vec, t);
  const uint32_t nitems = ((p.N + R - 1) / R) << gemv_split_log2(wdtype, vec, R, p, t);
  const uint32_t want = (nitems + kWarps - 1) / kWarps;
  uint32_t cap = sm_count() * (uint32_t)(t.ctas_per_sm < 1 ? 1 : t.ctas_per_sm);  // persistent: warps loop over items
  if (t.grid > 0) cap = (uint32_t)t.grid;
  return want < cap ? want : cap;
}

cudaError_t launch_gemv(cudaStream_t s, int wdtype, int kvdtype, GemvEpilogue epi, const GemvParams& p_in,
                        const GemvTune& t, bool pdl) {
  GemvParams p = p_in;
  if (p.N == 0 || p.K == 0) return cudaErrorInvalidValue;
  if ((epi == EPI_QKV_ROPE || epi == EPI_GATED) && (p.N % 2) != 0) return cudaErrorInvalidValue;
  if (use_ring(wdtype, epi, p, t)) {
    p.l2_ahead = (uint32_t)(t.l2_ahead < 0 ? 0 : t.l2_ahead);
    return launch_gemv_ring(s, wdtype, kvdtype, epi, p, t.unroll, t.ctas_per_sm, pdl);
  }
  const bool vec = vector_ok(wdtype, p);
  const int R = rows_per_warp(epi, vec, t);
  dim3 grid(gemv_grid(wdtype, epi, p, t));
  p.split_log2 = gemv_split_log2(wdtype, vec, R, p, t);
  if (p.norm_groups > 1 && (!p.gain || p.K % p.norm_groups)) return cudaErrorInvalidValue;
  if (p.form != FORM_POST_NORM && (p.post.y || p.gated_rows || p.gain_stride != 1)) return cudaErrorInvalidValue;
  if (p.form == FORM_PLAIN && p.act == ACT_CLAMPED) return cudaErrorInvalidValue;
  if (p.gated_rows && (epi != EPI_GATED || !p.tail || (p.gated_rows & 1u))) return cudaErrorInvalidValue;
  if (p.post.y && (!p.post.gain || p.tp.pull || p.norm_groups > 1)) return cudaErrorInvalidValue;
  size_t smem = (kSmemHeader + (size_t)gemv_x_floats(p) + gemv_form_floats(p, wdtype == 0 ? 4 : 8)) * sizeof(float);
  if (smem > 227 * 1024) return cudaErrorInvalidValue;
  if (p.form == FORM_POST_NORM) return launch_gemv_post(wdtype, epi, vec, R, t.unroll, grid, smem, s, pdl, p);
  if (p.form) {
    const ExpertMap& x = p.expert;
    if (p.form == FORM_EXPERT_ROWS && (epi != EPI_GATED || !x.rows || (x.rows & 1u) || p.N != x.router.top * x.rows || !x.logits || !x.chosen ||
                                     x.router.top > 32 || x.router.experts > kMaxExperts || x.router.groups > kMaxGroups))
      return cudaErrorInvalidValue;
    if (p.form == FORM_EXPERT_COLUMNS && (epi != EPI_STORE || !x.seg || !x.chosen || p.K < x.top * x.seg || (p.K > x.top * x.seg && (!x.W2 || !x.shared_gate))))
      return cudaErrorInvalidValue;
    return launch_gemv_experts(wdtype, epi, vec, R, t.unroll, grid, smem, s, pdl, p);
  }
  if (wdtype == 2 || epi == EPI_HYPER) {
    if (epi == EPI_QKV_ROPE || (epi == EPI_HYPER && (!p.hyper.S || p.hyper.S > kMaxStreams))) return cudaErrorInvalidValue;
    return launch_gemv_more(wdtype, epi, vec, R, t.unroll, grid, smem, s, pdl, p);
  }
  if (wdtype == 1) {
    if (kvdtype == 1) return launch_e<__half, __half>(epi, vec, R, t.unroll, grid, smem, s, pdl, p);
    return launch_e<__half, float>(epi, vec, R, t.unroll, grid, smem, s, pdl, p);
  }
  if (kvdtype == 1) return launch_e<float, __half>(epi, vec, R, t.unroll, grid, smem, s, pdl, p);
  return launch_e<float, float>(epi, vec, R, t.unroll, grid, smem, s, pdl, p);
}

}  // namespace nfai
