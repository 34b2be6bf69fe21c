// The register-streaming GEMV kernel (see gemv.cu for its design) and its launch helpers, as templates.
#pragma once
#include "gemv_common.cuh"
#include "moe_route.cuh"

namespace nfai {

using namespace gemv_detail;

namespace {  // every including translation unit instantiates its own combinations

constexpr int kSmemHeader = 96;  // floats ahead of x in shared memory: reduction scratch and split-row partials

// ---- weights found through the chosen experts (GemvForm) ----------------------------------------------------------
// Shared memory behind x, the gain and the base of a post-norm residual.
__host__ __device__ inline uint32_t gemv_x_floats(const GemvParams& p) {
  return (p.K * (1u + (p.gain ? 1u : 0u) + (p.post.y ? 1u : 0u)) + 3u) & ~3u;
}
__host__ __device__ inline uint32_t gemv_form_floats(const GemvParams& p, uint32_t vec_elems) {
  if (p.form == FORM_EXPERT_ROWS) return 2 * kMaxChosen + route_floats(p.expert.router.experts);
  if (p.form == FORM_EXPERT_COLUMNS) return 2 * (p.K / vec_elems);  // one pointer per vector of a row
  return 0;
}
struct ChosenRows {  // FORM_EXPERT_ROWS
  const uint32_t* ids;
  const float* w;
  __device__ __forceinline__ ChosenRows(const GemvParams& p, float* area) : ids(reinterpret_cast<uint32_t*>(area)), w(area + kMaxChosen) {}
  // warp 0 chooses, CTA 0 keeps the choice for the product that follows
  __device__ __forceinline__ static void choose(const GemvParams& p, float* area) {
    if (threadIdx.x < 32) {
      uint32_t* const ids = reinterpret_cast<uint32_t*>(area);
      route_warp(p.expert.router, p.expert.logits, area + 2 * kMaxChosen, ids, area + kMaxChosen);
      if (blockIdx.x == 0 && threadIdx.x < p.expert.router.top) p.expert.chosen[threadIdx.x] = ids[threadIdx.x];
    }
    __syncthreads();
  }
  __device__ __forceinline__ size_t row(const GemvParams& p, uint32_t n) const {  // row of W
    const uint32_t k = n / p.expert.rows;
    return (size_t)ids[k] * p.expert.rows + (n - k * p.expert.rows);
  }
};
// FORM_EXPERT_COLUMNS: element k of row 0 of the matrix it belongs to; the rows of that matrix are *ld elements apart. `mine` is
// the lane's entry of the chosen experts (chosen_lane). Every lane of the warp takes part.
__device__ __forceinline__ uint32_t chosen_lane(const GemvParams& p) {
  const uint32_t lane = threadIdx.x & 31;
  return lane < p.expert.top ? __ldcg(p.expert.chosen + lane) : 0u;
}
template <typename WT>
__device__ __forceinline__ const WT* chosen_column(const GemvParams& p, uint32_t k, uint32_t mine, uint32_t* ld) {
  const ExpertMap& m = p.expert;
  const uint32_t split = m.top * m.seg, i = min(k / m.seg, 31u);
  const uint32_t e = __shfl_sync(0xffffffffu, mine, (int)i);
  if (k >= split) {
    *ld = p.K - split;
    return reinterpret_cast<const WT*>(m.W2) + (k - split);
  }
  *ld = m.seg;
  return reinterpret_cast<const WT*>(p.W) + (size_t)e * p.N * m.seg + (k - i * m.seg);
}
// x behind the experts' parts belongs to the shared feed-forward
__device__ __forceinline__ void scale_shared(const GemvParams& p, float* xs) {
  const uint32_t split = p.expert.top * p.expert.seg;
  if (split >= p.K) return;
  const float g = route_sigmoid(__ldcg(p.expert.shared_gate));
  for (uint32_t i = split + threadIdx.x; i < p.K; i += kThreads) xs[i] *= g;
  __syncthreads();
}

// ---- the streamer ---------------------------------------------------------------------------------------------
template <typename WT, typename KVT, int R, int U, int EPI, int FORM = FORM_PLAIN>
__global__ void __launch_bounds__(kThreads, 2) gemv_kernel(const GemvParams p) {
  extern __shared__ __align__(16) float smem[];
  float* red = smem;                  // 2*kWarps words of reduction scratch
  float* part = smem + 32;            // [2][kWarps][R] partial row sums of a split row block (two parities)
  float* xs = smem + kSmemHeader;     // K floats of x, then K floats of gain
  constexpr int VE = WeightVec<WT>::kElems;
  constexpr bool kPlainWeights = FORM == FORM_PLAIN || FORM == FORM_POST_NORM;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const uint32_t nvec = p.K / VE;  // host guarantees K % VE == 0 and 16-byte aligned rows
  // A work item is (row block, K chunk): R rows x cv vectors. With split = 1 the chunk is the whole row.
  const uint32_t sl = p.split_log2, S = 1u << sl;
  const uint32_t cv = (((nvec + S - 1) >> sl) + 31u) & ~31u;  // vectors per chunk, a whole number of warp strides
  const uint32_t nkb = (cv + 32 * U - 1) / (32 * U);          // batches per item
  const uint32_t nrb = (p.N + R - 1) / R;                     // row blocks
  const uint32_t nitems = nrb << sl;
  const uint32_t TW = gridDim.x * kWarps;
  const uint32_t nrounds = (nitems + TW - 1) / TW;  // the same for every warp of the grid: barriers stay uniform
  const WT* const Wbase = reinterpret_cast<const WT*>(p.W);
  const uint4 zero = make_uint4(0, 0, 0, 0);
  float* const area = xs + gemv_x_floats(p);
  const ChosenRows rows(p, area);                           // FORM_EXPERT_ROWS
  const WT** const cols = reinterpret_cast<const WT**>(area);  // FORM_EXPERT_COLUMNS: vector v of row 0
  const uint32_t cols_split = FORM == FORM_EXPERT_COLUMNS ? p.expert.top * p.expert.seg / VE : 0u;

  uint32_t mine = 0;  // FORM_EXPERT_COLUMNS, until the table of columns is there
  auto load_batch = [&](uint4(&buf)[U][R], uint32_t t, uint32_t kb, bool first = false) {
    if (t >= nitems) return;
    const uint32_t rb = t >> sl, c = t & (S - 1);
    const uint32_t v0 = c * cv + kb * (32 * U) + lane;
    const uint32_t vend = min((c + 1) * cv, nvec);
    if constexpr (FORM == FORM_EXPERT_COLUMNS) {
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const uint32_t v = v0 + 32 * u;
        uint32_t ld_first;
        const WT* col = nullptr;
        if (first) col = chosen_column<WT>(p, v * VE, mine, &ld_first);
        else if (v < vend) col = cols[v];
        const uint32_t ld = v < cols_split ? p.expert.seg : p.K - p.expert.top * p.expert.seg;
#pragma unroll
        for (int r = 0; r < R; ++r) {
          uint32_t n = rb * R + r;
          n = n < p.N ? n : p.N - 1;
          buf[u][r] = v < vend ? ld_stream16(col + (size_t)n * ld) : zero;
        }
      }
    } else {
#pragma unroll
      for (int r = 0; r < R; ++r) {
        uint32_t n = rb * R + r;
        n = n < p.N ? n : p.N - 1;  // a ragged last block re-reads the last row, never out of bounds
        const uint4* wrow = reinterpret_cast<const uint4*>(Wbase + (FORM == FORM_EXPERT_ROWS ? rows.row(p, n) : (size_t)n) * p.K);
#pragma unroll
        for (int u = 0; u < U; ++u) {
          const uint32_t v = v0 + 32 * u;
          buf[u][r] = v < vend ? ld_stream16(wrow + v) : zero;
        }
      }
    }
  };

  uint32_t t = blockIdx.x * kWarps + warp;
  uint32_t lt = t, lkb = 0;  // load cursor: the batch the next request asks for
  auto advance = [&]() {
    if (++lkb == nkb) {
      lkb = 0;
      lt += TW;
    }
  };
  // Weights do not depend on the previous kernel: the first batch is requested before the dependency wait.
  // (Requesting the first two there, in either loop order, measured 10-30% slower in the steady state.)
  uint4 cur[U][R], nxt[U][R];
  if constexpr (kPlainWeights) {
    load_batch(cur, lt, lkb);
    advance();
  }
  load_gain<FORM == FORM_POST_NORM>(p, xs);
  prefetch_plan(p.pf, kPrefetchChunk);
  pdl_launch_dependents();
  pdl_wait();
  if constexpr (!kPlainWeights) {  // which weights are needed is part of the previous kernel's result
    if constexpr (FORM == FORM_EXPERT_ROWS) ChosenRows::choose(p, area);
    else mine = chosen_lane(p);
    load_batch(cur, lt, lkb, true);
    advance();
    if constexpr (FORM == FORM_EXPERT_COLUMNS) {  // read after the barriers of load_x
      for (uint32_t v = threadIdx.x; v < ((nvec + 31u) & ~31u); v += kThreads) {
        uint32_t ld;
        const WT* col = chosen_column<WT>(p, v * VE, mine, &ld);
        if (v < nvec) cols[v] = col;
      }
    }
  }
  // what the epilogue of the first item reads (residual / cos, sin of this position) travels with x
  uint32_t pos = 0;
  if (EPI == EPI_QKV_ROPE || (EPI == EPI_STORE && p.y_ring)) pos = p.state ? p.state->pos : p.pos_imm;
  float pre[R];
  epi_preload<R, EPI>(p, (min(t, nitems - 1) >> sl) * R, pos, pre);
  load_x<false, FORM == FORM_POST_NORM>(p, xs, red);
  if constexpr (FORM == FORM_EXPERT_COLUMNS) scale_shared(p, xs);

  float best_v = -INFINITY;
  uint32_t best_i = 0xffffffffu;
  float acc[R];
#pragma unroll
  for (int r = 0; r < R; ++r) acc[r] = 0.f;
  for (uint32_t round = 0; round < nrounds; ++round, t += TW) {
    const uint32_t c = t & (S - 1);
    float pre_next[R];
    epi_preload<R, EPI>(p, (min(t + TW, nitems - 1) >> sl) * R, pos, pre_next);
    const uint32_t vend = min((c + 1) * cv, nvec);
    for (uint32_t kb = 0; kb < nkb; ++kb) {
      load_batch(nxt, lt, lkb);
      advance();
      if (t < nitems) {
        const uint32_t v0 = c * cv + kb * (32 * U) + lane;
#pragma unroll
        for (int u = 0; u < U; ++u) {
          const uint32_t v = v0 + 32 * u;
          if (v < vend) {
            float xv[VE];
            const float4* xp = reinterpret_cast<const float4*>(xs + (size_t)v * VE);
#pragma unroll
            for (int i = 0; i < VE / 4; ++i) {
              float4 q = xp[i];
              xv[4 * i] = q.x;
              xv[4 * i + 1] = q.y;
              xv[4 * i + 2] = q.z;
              xv[4 * i + 3] = q.w;
            }
#pragma unroll
            for (int r = 0; r < R; ++r) {
              float wf[VE];
              WeightVec<WT>::unpack(cur[u][r], wf);
#pragma unroll
              for (int i = 0; i < VE; ++i) acc[r] = fmaf(wf[i], xv[i], acc[r]);
            }
          }
        }
      }
#pragma unroll
      for (int u = 0; u < U; ++u)
#pragma unroll
        for (int r = 0; r < R; ++r) cur[u][r] = nxt[u][r];
    }
    if constexpr (FORM == FORM_EXPERT_ROWS) {  // the weight of the pair's expert takes the place of what an epilogue preloads
#pragma unroll
      for (int r = 0; r < R; ++r) pre[r] = rows.w[min((t >> sl) * R + r, p.N - 1) / p.expert.rows];
    }
    // the item is complete
#pragma unroll
    for (int r = 0; r < R; ++r) acc[r] = warp_sum(acc[r]);
    if (S == 1) {
      if (t < nitems) row_epilogue_pre<KVT, R, EPI, FORM>(p, t * R, acc, pre, pos, best_v, best_i);
    } else {
      // the S chunks of a row block sit in S consecutive warps of this CTA: add them up in warp order
      float* pr = part + (round & 1) * (kWarps * R);
      if (lane == 0) {
#pragma unroll
        for (int r = 0; r < R; ++r) pr[warp * R + r] = acc[r];
      }
      __syncthreads();
      if (c == 0 && t < nitems) {
#pragma unroll
        for (int r = 0; r < R; ++r) {
          float a = pr[warp * R + r];
          for (uint32_t j = 1; j < S; ++j) a += pr[(warp + j) * R + r];
          acc[r] = a;
        }
        row_epilogue_pre<KVT, R, EPI, FORM>(p, (t >> sl) * R, acc, pre, pos, best_v, best_i);
      }
    }
#pragma unroll
    for (int r = 0; r < R; ++r) {
      acc[r] = 0.f;
      pre[r] = pre_next[r];
    }
  }
  if constexpr (EPI == EPI_LOGITS) cta_argmax_partial(p, best_v, best_i, red);
}

// Same contract for any K and any alignment (element loads); used when K is not a multiple of the vector width.
template <typename WT, typename KVT, int EPI, int FORM = FORM_PLAIN>
__global__ void __launch_bounds__(kThreads) gemv_scalar_kernel(const GemvParams p) {
  extern __shared__ __align__(16) float smem[];
  float* red = smem;
  float* xs = smem + kSmemHeader;
  constexpr int R = 2;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const uint32_t nrb = (p.N + R - 1) / R;
  load_gain<FORM == FORM_POST_NORM>(p, xs);
  prefetch_plan(p.pf, kPrefetchChunk);
  pdl_launch_dependents();
  pdl_wait();
  const uint32_t pos = EPI == EPI_STORE && p.y_ring ? (p.state ? p.state->pos : p.pos_imm) : 0u;
  float* const area = xs + gemv_x_floats(p);
  const ChosenRows rows(p, area);
  if constexpr (FORM == FORM_EXPERT_ROWS) ChosenRows::choose(p, area);
  const uint32_t mine = FORM == FORM_EXPERT_COLUMNS ? chosen_lane(p) : 0u;
  load_x<false, FORM == FORM_POST_NORM>(p, xs, red);
  if constexpr (FORM == FORM_EXPERT_COLUMNS) scale_shared(p, xs);
  float best_v = -INFINITY;
  uint32_t best_i = 0xffffffffu;
  for (uint32_t rb = blockIdx.x * kWarps + warp; rb < nrb; rb += gridDim.x * kWarps) {
    float acc[R];
#pragma unroll
    for (int r = 0; r < R; ++r) {
      uint32_t n = rb * R + r < p.N ? rb * R + r : p.N - 1;
      float a = 0.f;
      if constexpr (FORM == FORM_EXPERT_COLUMNS) {
        for (uint32_t k = lane; k < ((p.K + 31u) & ~31u); k += 32) {
          uint32_t ld;
          const WT* col = chosen_column<WT>(p, k, mine, &ld);
          if (k < p.K) a = fmaf(to_float(col[(size_t)n * ld]), xs[k], a);
        }
      } else {
        const WT* w = reinterpret_cast<const WT*>(p.W) + (FORM == FORM_EXPERT_ROWS ? rows.row(p, n) : (size_t)n) * p.K;
        for (uint32_t k = lane; k < p.K; k += 32) a = fmaf(to_float(w[k]), xs[k], a);
      }
      acc[r] = warp_sum(a);
    }
    if constexpr (EPI == EPI_STORE || EPI == EPI_HYPER || FORM == FORM_EXPERT_ROWS || FORM == FORM_POST_NORM) {
      float pre[R];
      if constexpr (FORM == FORM_EXPERT_ROWS) {
#pragma unroll
        for (int r = 0; r < R; ++r) pre[r] = rows.w[rb * R / p.expert.rows];  // (both rows of a pair: one expert)
      } else {
        epi_preload<R, EPI>(p, rb * R, pos, pre);
      }
      row_epilogue_pre<KVT, R, EPI, FORM>(p, rb * R, acc, pre, pos, best_v, best_i);
    } else {
      row_epilogue<KVT, R, EPI>(p, rb * R, acc, best_v, best_i);
    }
  }
  if constexpr (EPI == EPI_LOGITS) cta_argmax_partial(p, best_v, best_i, red);
}

template <typename K>
cudaError_t launch_k(K kernel, dim3 grid, size_t smem, cudaStream_t s, bool pdl, const GemvParams& p) {
  cudaError_t e = cudaSuccess;
  if (smem > 48 * 1024) {
    e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return e;
  }
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = grid;
  cfg.blockDim = dim3(kThreads);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = s;
  cudaLaunchAttribute attr[1];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = pdl ? 1 : 0;
  cfg.attrs = attr;
  cfg.numAttrs = 1;
  return cudaLaunchKernelEx(&cfg, kernel, p);
}

template <typename WT, typename KVT, int R, int EPI, int FORM = FORM_PLAIN>
cudaError_t launch_u(int U, dim3 grid, size_t smem, cudaStream_t s, bool pdl, const GemvParams& p) {
  switch (U) {
    case 2: return launch_k(gemv_kernel<WT, KVT, R, 2, EPI, FORM>, grid, smem, s, pdl, p);
    case 4: return launch_k(gemv_kernel<WT, KVT, R, 4, EPI, FORM>, grid, smem, s, pdl, p);
    case 8:
      if constexpr (R <= 2) return launch_k(gemv_kernel<WT, KVT, R, 8, EPI, FORM>, grid, smem, s, pdl, p);
      return cudaErrorInvalidValue;  // 4 rows x 8 steps x 2 buffers would not fit the register file
    default: return cudaErrorInvalidValue;
  }
}

template <typename WT, typename KVT, int EPI, int FORM = FORM_PLAIN>
cudaError_t launch_r(int R, int U, dim3 grid, size_t smem, cudaStream_t s, bool pdl, const GemvParams& p) {
  if constexpr (EPI == EPI_STORE || EPI == EPI_LOGITS || EPI == EPI_HYPER) {
    if (R == 1) return launch_u<WT, KVT, 1, EPI, FORM>(U, grid, smem, s, pdl, p);
  }
  if (R == 2) return launch_u<WT, KVT, 2, EPI, FORM>(U, grid, smem, s, pdl, p);
  if (R == 4) return launch_u<WT, KVT, 4, EPI, FORM>(U, grid, smem, s, pdl, p);
  return cudaErrorInvalidValue;
}

}  // namespace

}  // namespace nfai
