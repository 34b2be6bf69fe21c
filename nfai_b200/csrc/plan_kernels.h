// Launch interface of the kernels that layer-plan models add to the shared ones (internal).
// Element types are codes: 0 float32, 1 float16, 2 bfloat16 (NFAI_F32, NFAI_F16, NFAI_BF16).
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

#include "kernels.h"
#include "plan.h"

namespace nfai {

// ---- hyper-connections over rows of tokens (hyper.cu) ---------------------------------------------------------------
// One row (token) per CTA: bring the S streams up to date, form what the next sublayer reads, normalise it.
//   source   embedding row of tokens[row] (all streams equal), or the streams X themselves, after the write of y if given
//   result   X_out (if given), u_out = sum_t next_in[t] x_t (if given), normed = RMS norm of u times gain (if given)
struct HyperRows {
  const uint32_t* tokens = nullptr;
  const void* embed = nullptr;  // [V][H] of embed_dtype
  int embed_dtype = 0;
  const float* X = nullptr;     // [T][S][H]
  const uint32_t* rows = nullptr;  // optional: CTA i works on row rows[i] of X (outputs stay at row i)
  const float* y = nullptr;     // [T][H]
  const float* mix = nullptr;   // [S][S], [from][to]
  const float* out = nullptr;   // [S]
  const float* next_in = nullptr;  // [S], null: plain sum
  float* X_out = nullptr;
  float* u_out = nullptr;       // [T][H]
  const float* gain = nullptr;
  float eps = 0.f;
  void* normed = nullptr;       // [T][H] of normed_dtype
  int normed_dtype = 0;
  uint32_t S = 1, H = 0;
};
cudaError_t launch_hyper_rows(cudaStream_t s, const HyperRows& p, uint32_t n_rows);
// Decode step: streams and first read of the token in *state (its prompt buffer if given).
cudaError_t launch_embed_streams(cudaStream_t s, int wdtype, const void* E, uint32_t H, uint32_t V, uint32_t S, StepState* state,
                                 const uint32_t* prompt, const float* first_in, float* X, float* u, bool pdl);

// ---- latent attention (latent.cu) -----------------------------------------------------------------------------------
struct LatentParams {
  LatentSpec spec;
  const float* in = nullptr;        // projected rows [q | latent, key part | gate], in_ld floats apart
  uint32_t in_ld = 0;
  const float* lat_gain = nullptr;  // [rank]
  float eps = 0.f;
  const float2* rope_cs = nullptr;  // [ctx][rope_dims/2]
  const void* Wkv = nullptr;        // [heads*dim | heads*vdim][rank] of dtype: per-head keys, then per-head values
  void* c_cache = nullptr;          // [ctx][rank] of dtype
  void* kr_cache = nullptr;         // [ctx][rot] of dtype
  int dtype = 0;                    // of Wkv, caches and (prompt path) operands: 0 or 2
  uint32_t ctx = 0;
  StepState* state = nullptr;       // decode: position
  uint32_t pos0 = 0;                // prompt path (and decode without state): position of the first token
  // decode
  float* out = nullptr;             // [heads*vdim], gated
  void* scratch = nullptr;          // latent_decode_scratch bytes, zero-filled once
  // prompt path
  void* q = nullptr;                // [T][heads*(dim+rot)] of dtype, rotated
  const void* kv = nullptr;         // [rows][heads*dim | heads*vdim] of dtype; row 0 is position kv_pos0
  uint32_t kv_pos0 = 0;
  void* ao = nullptr;               // [T][heads*vdim] of dtype, gated
};
bool latent_supported(const LatentSpec& s, int dtype, std::string* why);
size_t latent_decode_scratch(const LatentSpec& s, int dtype, uint32_t ctx);
// Adds the number of kernels it launched to *launches (may be null).
cudaError_t launch_latent_decode(cudaStream_t s, const LatentParams& p, bool pdl, int* launches);
// Norm and rotate what the projection of T tokens left: cache rows pos0 .. pos0+T-1 and p.q.
cudaError_t launch_latent_prep(cudaStream_t s, const LatentParams& p, uint32_t T);
// Windowed causal attention of the T tokens over the expanded keys and values, gated.
cudaError_t launch_latent_prefill(cudaStream_t s, const LatentParams& p, uint32_t T);

// ---- state space layers (ssm.cu) ------------------------------------------------------------------------------------
struct SsmParams {
  SsmSpec spec;
  // Projected rows [z | x B C | dt]. Decode: a ring of `taps` rows indexed by position, the row of the current position
  // already in place. Prompt path: `in` holds the T rows, the ring the rows of earlier positions.
  float* ring = nullptr;
  const float* in = nullptr;
  const float* conv_w = nullptr;  // [channels][taps]
  const float* conv_b = nullptr;
  const float* dt_bias = nullptr;
  const float* A_log = nullptr;
  const float* D = nullptr;
  float* S = nullptr;             // [heads][vdim][state]
  StepState* state = nullptr;
  uint32_t pos0 = 0;
  float* y = nullptr;             // decode: [inner], prompt: [T][inner]; silu(z)-gated, not yet normed
  // prompt path workspace
  void* xbc = nullptr;            // [T][channels] of xbc_dtype, after convolution and silu
  int xbc_dtype = 0;
  float* dt = nullptr;            // [T][heads] after softplus
  float* chunk = nullptr;         // chunked scan: per-chunk states (ssm_chunk_floats)
  size_t chunk_floats = 0;
};
cudaError_t launch_ssm_step(cudaStream_t s, const SsmParams& p, bool pdl);
// Convolution, step sizes and the recurrence of T tokens; leaves the state and the ring as decoding them would.
cudaError_t launch_ssm_prefill(cudaStream_t s, const SsmParams& p, uint32_t T);
size_t ssm_chunk_floats(const SsmSpec& s, uint32_t T);
// out[t] = RMS norm of y[t] in `groups` equal parts, times gain, as out_dtype.
cudaError_t launch_group_norm_rows(cudaStream_t s, const float* y, const float* gain, float eps, uint32_t groups, uint32_t T,
                                   uint32_t K, void* out, int out_dtype);

}  // namespace nfai
