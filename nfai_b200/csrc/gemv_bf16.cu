// Instantiations of the register-streaming GEMV for bfloat16 weights, and of the hyper-connection epilogue for every
// weight type (kept out of gemv.cu so that the two compile in parallel).
#include "gemv_kernel.cuh"

namespace nfai {

namespace {

template <typename WT, int EPI>
cudaError_t launch_one(bool vec, int R, int U, dim3 grid, size_t smem, cudaStream_t s, bool pdl, const GemvParams& p) {
  if (!vec) return launch_k(gemv_scalar_kernel<WT, float, EPI>, grid, smem, s, pdl, p);
  return launch_r<WT, float, EPI>(R, U, grid, smem, s, pdl, p);
}

}  // namespace

cudaError_t launch_gemv_more(int wdtype, GemvEpilogue epi, bool vec, int R, int U, dim3 grid, size_t smem, cudaStream_t s,
                             bool pdl, const GemvParams& p) {
  if (wdtype == 2) {
    switch (epi) {
      case EPI_STORE: return launch_one<__nv_bfloat16, EPI_STORE>(vec, R, U, grid, smem, s, pdl, p);
      case EPI_GATED: return launch_one<__nv_bfloat16, EPI_GATED>(vec, R, U, grid, smem, s, pdl, p);
      case EPI_LOGITS: return launch_one<__nv_bfloat16, EPI_LOGITS>(vec, R, U, grid, smem, s, pdl, p);
      case EPI_HYPER: return launch_one<__nv_bfloat16, EPI_HYPER>(vec, R, U, grid, smem, s, pdl, p);
      default: return cudaErrorInvalidValue;
    }
  }
  if (epi != EPI_HYPER) return cudaErrorInvalidValue;
  if (wdtype == 1) return launch_one<__half, EPI_HYPER>(vec, R, U, grid, smem, s, pdl, p);
  return launch_one<float, EPI_HYPER>(vec, R, U, grid, smem, s, pdl, p);
}

}  // namespace nfai
