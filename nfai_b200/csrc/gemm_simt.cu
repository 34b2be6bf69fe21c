// C[M][N] = A[M][K] W[N][K]^T on the CUDA cores with the epilogues of the tensor-core GEMM: prompt ingestion of true
// float32 models (a reduced-precision tensor mode would not do) and of matrices whose rows are not 16-byte aligned.
// 64 x 64 tiles, 256 threads with 4 x 4 outputs each (two column pairs), K in steps of 16 through shared memory.
#include "gemm_epilogue.cuh"
#include "kernels.h"

namespace nfai {

namespace {

constexpr int kT = 64, kKS = 16;

template <typename T, bool GROUPED>
__global__ void __launch_bounds__(256) gemm_simt_kernel(const T* __restrict__ A, const T* __restrict__ W, uint32_t M, uint32_t N,
                                                        uint32_t K, const GemmGroups grp, const GemmEpilogue ep) {
  __shared__ float As[kKS][kT + 4], Ws[kKS][kT + 4];
  pdl_launch_dependents();
  pdl_wait();
  uint32_t m0 = blockIdx.y * kT;
  const uint32_t n0 = blockIdx.x * kT;
  if constexpr (GROUPED) {  // blockIdx.y counts the kT-row parts of the group tiles
    const uint32_t i = blockIdx.y / (kGroupTile / kT);
    if (i >= *grp.n_tiles) return;
    const uint2 tile = grp.tiles[i];
    m0 = tile.y + blockIdx.y % (kGroupTile / kT) * kT;
    M = grp.rows[tile.x + 1];
    if (m0 >= M) return;
    W += (size_t)tile.x * N * K;
  }
  const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
  float acc[4][4] = {};
  float a_reg[4], w_reg[4];
  auto fetch = [&](uint32_t k0) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int e = tid + 256 * i, row = e >> 4, k = e & 15;
      const bool in_k = k0 + k < K;
      a_reg[i] = in_k && m0 + row < M ? to_float(A[(size_t)(m0 + row) * K + k0 + k]) : 0.f;
      w_reg[i] = in_k && n0 + row < N ? to_float(W[(size_t)(n0 + row) * K + k0 + k]) : 0.f;
    }
  };
  fetch(0);
  for (uint32_t k0 = 0; k0 < K; k0 += kKS) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int e = tid + 256 * i, row = e >> 4, k = e & 15;
      As[k][row] = a_reg[i];
      Ws[k][row] = w_reg[i];
    }
    __syncthreads();
    if (k0 + kKS < K) fetch(k0 + kKS);
#pragma unroll
    for (int k = 0; k < kKS; ++k) {
      float av[4], wv[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) av[i] = As[k][ty * 4 + i];
#pragma unroll
      for (int j = 0; j < 4; ++j) wv[j] = Ws[k][tx * 4 + j];
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], wv[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const uint32_t m = m0 + ty * 4 + i;
    if (m >= M) break;
#pragma unroll
    for (int j = 0; j < 4; j += 2) {
      const uint32_t n = n0 + tx * 4 + j;
      if (n < N) epilogue_pair(ep, m, n, N, acc[i][j], acc[i][j + 1], epilogue_aux(ep, m, n, N));
    }
  }
}

}  // namespace

cudaError_t launch_gemm_simt(cudaStream_t s, int dtype, const void* A, const void* W, uint32_t M, uint32_t N, uint32_t K,
                             const GemmEpilogue& ep) {
  if (!A || !W || !M || !N || !K || ((ep.kind == GEMM_EPI_GATED || ep.kind == GEMM_EPI_GATED_CLAMPED) && (N & 1u))) return cudaErrorInvalidValue;
  const dim3 grid((N + kT - 1) / kT, (M + kT - 1) / kT);
  const GemmGroups none;
  if (dtype == 0)
    return launch_pdl(gemm_simt_kernel<float, false>, grid, dim3(256), 0, s, prefill_pdl(), (const float*)A, (const float*)W, M, N, K, none, ep);
  if (dtype == 2)
    return launch_pdl(gemm_simt_kernel<__nv_bfloat16, false>, grid, dim3(256), 0, s, prefill_pdl(), (const __nv_bfloat16*)A,
                      (const __nv_bfloat16*)W, M, N, K, none, ep);
  return cudaErrorInvalidValue;
}

cudaError_t launch_gemm_simt_grouped(cudaStream_t s, int dtype, const void* A, const void* W, uint32_t N, uint32_t K, const GemmGroups& g,
                                     const GemmEpilogue& ep) {
  if (!A || !W || !N || !K || !g.max_tiles || ep.bias || ep.resid || ((ep.kind == GEMM_EPI_GATED || ep.kind == GEMM_EPI_GATED_CLAMPED) && (N & 1u))) return cudaErrorInvalidValue;
  const dim3 grid((N + kT - 1) / kT, g.max_tiles * (kGroupTile / kT));
  if (grid.y > 65535) return cudaErrorInvalidValue;
  if (dtype == 0)
    return launch_pdl(gemm_simt_kernel<float, true>, grid, dim3(256), 0, s, prefill_pdl(), (const float*)A, (const float*)W, 0u, N, K, g, ep);
  if (dtype == 2)
    return launch_pdl(gemm_simt_kernel<__nv_bfloat16, true>, grid, dim3(256), 0, s, prefill_pdl(), (const __nv_bfloat16*)A,
                      (const __nv_bfloat16*)W, 0u, N, K, g, ep);
  return cudaErrorInvalidValue;
}

}  // namespace nfai
