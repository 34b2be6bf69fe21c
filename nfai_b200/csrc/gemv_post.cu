// Instantiations of the register-streaming GEMV for models with a post-norm residual (FORM_POST_NORM).
#include "gemv_kernel.cuh"

namespace nfai {

namespace {

template <typename WT, int EPI>
cudaError_t launch_one(bool vec, int R, int U, dim3 grid, size_t smem, cudaStream_t s, bool pdl, const GemvParams& p) {
  if (!vec) return launch_k(gemv_scalar_kernel<WT, float, EPI, FORM_POST_NORM>, grid, smem, s, pdl, p);
  return launch_r<WT, float, EPI, FORM_POST_NORM>(R, U, grid, smem, s, pdl, p);
}

template <typename WT>
cudaError_t launch_wt(GemvEpilogue epi, bool vec, int R, int U, dim3 grid, size_t smem, cudaStream_t s, bool pdl, const GemvParams& p) {
  switch (epi) {
    case EPI_STORE: return launch_one<WT, EPI_STORE>(vec, R, U, grid, smem, s, pdl, p);
    case EPI_GATED: return launch_one<WT, EPI_GATED>(vec, R, U, grid, smem, s, pdl, p);
    case EPI_LOGITS: return launch_one<WT, EPI_LOGITS>(vec, R, U, grid, smem, s, pdl, p);
    default: return cudaErrorInvalidValue;
  }
}

}  // namespace

cudaError_t launch_gemv_post(int wdtype, GemvEpilogue epi, bool vec, int R, int U, dim3 grid, size_t smem, cudaStream_t s,
                             bool pdl, const GemvParams& p) {
  if (wdtype == 2) return launch_wt<__nv_bfloat16>(epi, vec, R, U, grid, smem, s, pdl, p);
  if (wdtype == 0) return launch_wt<float>(epi, vec, R, U, grid, smem, s, pdl, p);
  return cudaErrorInvalidValue;
}

}  // namespace nfai
