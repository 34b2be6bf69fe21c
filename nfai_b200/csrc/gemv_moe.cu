// Instantiations of the register-streaming GEMV whose weights are found through the chosen experts (GemvForm).
#include "gemv_kernel.cuh"

namespace nfai {

namespace {

template <typename WT, int EPI, int FORM, int R>
cudaError_t launch_unroll(int U, dim3 grid, size_t smem, cudaStream_t s, bool pdl, const GemvParams& p) {
  if (U == 2) return launch_k(gemv_kernel<WT, float, R, 2, EPI, FORM>, grid, smem, s, pdl, p);
  return launch_k(gemv_kernel<WT, float, R, 4, EPI, FORM>, grid, smem, s, pdl, p);
}

template <typename WT, int EPI, int FORM>
cudaError_t launch_form(bool vec, int R, int U, dim3 grid, size_t smem, cudaStream_t s, bool pdl, const GemvParams& p) {
  if (!vec) return launch_k(gemv_scalar_kernel<WT, float, EPI, FORM>, grid, smem, s, pdl, p);
  if constexpr (EPI == EPI_STORE) {
    if (R == 1) return launch_unroll<WT, EPI, FORM, 1>(U, grid, smem, s, pdl, p);
  }
  if (R == 4) return launch_unroll<WT, EPI, FORM, 4>(U, grid, smem, s, pdl, p);
  if (R == 2) return launch_unroll<WT, EPI, FORM, 2>(U, grid, smem, s, pdl, p);
  return cudaErrorInvalidValue;
}

template <typename WT>
cudaError_t launch_wt(GemvEpilogue epi, bool vec, int R, int U, dim3 grid, size_t smem, cudaStream_t s, bool pdl, const GemvParams& p) {
  if (U != 2 && U != 4) return cudaErrorInvalidValue;
  if (epi == EPI_GATED && p.form == FORM_EXPERT_ROWS) return launch_form<WT, EPI_GATED, FORM_EXPERT_ROWS>(vec, R, U, grid, smem, s, pdl, p);
  if (epi == EPI_STORE && p.form == FORM_EXPERT_COLUMNS) return launch_form<WT, EPI_STORE, FORM_EXPERT_COLUMNS>(vec, R, U, grid, smem, s, pdl, p);
  return cudaErrorInvalidValue;
}

}  // namespace

cudaError_t launch_gemv_experts(int wdtype, GemvEpilogue epi, bool vec, int R, int U, dim3 grid, size_t smem, cudaStream_t s,
                                bool pdl, const GemvParams& p) {
  if (wdtype == 2) return launch_wt<__nv_bfloat16>(epi, vec, R, U, grid, smem, s, pdl, p);
  if (wdtype == 0) return launch_wt<float>(epi, vec, R, U, grid, smem, s, pdl, p);
  return cudaErrorInvalidValue;
}

}  // namespace nfai
