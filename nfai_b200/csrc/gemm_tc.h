// Tensor-core GEMM for prompt ingestion (internal interface).
#pragma once
#include <cuda_fp16.h>
#include <cuda_runtime.h>
#include <stdint.h>

namespace nfai {

enum GemmEpilogueKind { GEMM_EPI_STORE = 0, GEMM_EPI_GATED = 1, GEMM_EPI_QKV_ROPE = 2, GEMM_EPI_STORE_ACT = 3, GEMM_EPI_GATED_CLAMPED = 4 };

struct GemmEpilogue {
  int kind = GEMM_EPI_STORE;
  float* out_f32 = nullptr;      // STORE: [M][N]; QKV_ROPE: q rows [M][qDim]
  const float* resid = nullptr;  // STORE: optional [M][N] addend
  const float* bias = nullptr;   // STORE, STORE_ACT, GATED: optional [N]
  void* out_act = nullptr;       // GATED: [M][N/2], STORE_ACT: [M][N], of out_dtype
  int out_dtype = 1;             // 0 float32, 1 float16, 2 bfloat16
  int act = 0;                   // GATED: Activation (kernels.h)
  // GATED_CLAMPED: as GATED with the clamped activation and its limit, without bias
  float act_limit = 0.f;
  uint32_t gated_cols = 0;       // only this many columns are gate/up pairs (0: all), the rest go plainly to out_f32
                                 // [M][N - gated_cols]; even, as is N
  uint32_t operands_bf16 = 0;    // 1: A and W are bfloat16 (both), 0: float16 (both)
  // QKV_ROPE
  void* kcache = nullptr;
  void* vcache = nullptr;
  int kv_f16 = 0;
  uint32_t qDim = 0, kvDim = 0, d = 0, ropeDim = 0, pos0 = 0;
  const float2* rope_cs = nullptr;
  // Optional scratch for split-K: when the tile grid alone would leave most SMs idle (a short prompt chunk), the K
  // range is divided over several CTAs, each stores its float32 partial tile here ([split][M][N]) and a second
  // kernel adds the partials in split order and applies the epilogue. Without scratch the GEMM never splits.
  float* scratch = nullptr;
  size_t scratch_floats = 0;
};

// Rows of A sorted into groups (experts), each multiplied by its own matrix: group g's rows are rows[g] .. rows[g+1]-1 of A
// and of the output, its matrix is rows g*N .. g*N+N-1 of W. All of it is device data; a kernel walks the tile list.
struct GemmGroups {
  uint32_t count = 0;               // number of groups
  const uint32_t* rows = nullptr;   // [count + 1] first row of each group
  const uint2* tiles = nullptr;     // (group, first row) of every kGroupTile rows of a group, groups in order
  const uint32_t* n_tiles = nullptr;
  uint32_t max_tiles = 0;           // upper bound of *n_tiles
};
constexpr uint32_t kGroupTile = 128;

// Number of K splits launch_gemm_tc would use for this shape given enough scratch (1 = no split).
uint32_t gemm_tc_splits(uint32_t M, uint32_t N, uint32_t K);

// C = A[M][K] * W[N][K]^T with the epilogue applied; A and W are float16, K contiguous, K % 8 == 0, 16-byte aligned.
// err (optional device word) gets bit 4 when a bounded wait inside the kernel gave up.
cudaError_t launch_gemm_tc(cudaStream_t s, const __half* A, const __half* W, uint32_t M, uint32_t N, uint32_t K,
                           const GemmEpilogue& ep, uint32_t* err);

// The same for grouped rows: A [rows][K] in group order, W [groups][N][K]; epilogues GATED, GATED_CLAMPED, STORE and
// STORE_ACT without bias or residual. max_rows bounds the rows of A.
cudaError_t launch_gemm_tc_grouped(cudaStream_t s, const __half* A, const __half* W, uint32_t max_rows, uint32_t N, uint32_t K,
                                   const GemmGroups& g, const GemmEpilogue& ep, uint32_t* err);
cudaError_t launch_gemm_simt_grouped(cudaStream_t s, int dtype, const void* A, const void* W, uint32_t N, uint32_t K, const GemmGroups& g,
                                     const GemmEpilogue& ep);

// x[M][H] float32 -> RMS-normalised, gain-scaled float16 rows (the A operand of the QKV and gate/up GEMMs).
// after_collective: x was produced by a library collective enqueued just before; the kernel is then launched with
// plain stream order (no programmatic dependent launch across the library's kernels).
cudaError_t launch_rmsnorm_to_half(cudaStream_t s, const float* x, const float* gain, float eps, uint32_t M, uint32_t H,
                                   __half* out, bool after_collective = false);
// The same product with any K and any alignment on the CUDA cores, A and W both of `dtype` (0 float32, 2 bfloat16): true
// float32 models, and shapes the tensor-core kernel cannot take.
cudaError_t launch_gemm_simt(cudaStream_t s, int dtype, const void* A, const void* W, uint32_t M, uint32_t N, uint32_t K,
                             const GemmEpilogue& ep);
// rows of the embedding matrix (float16) widened to float32: x[t] = E[tokens[t]].
cudaError_t launch_embed_rows(cudaStream_t s, const __half* E, const uint32_t* tokens, uint32_t M, uint32_t H, float* x);
cudaError_t launch_float_to_half(cudaStream_t s, const float* in, __half* out, size_t n);

}  // namespace nfai
