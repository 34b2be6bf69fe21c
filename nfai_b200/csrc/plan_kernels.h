// Launch interface of the kernels that layer-plan models add to the shared ones (internal).
// Element types are codes: 0 float32, 1 float16, 2 bfloat16 (NFAI_F32, NFAI_F16, NFAI_BF16).
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

#include <string>

#include "gemm_tc.h"
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

// ---- residual with post-norms over rows of tokens (post_rows.cu) -----------------------------------------------------
// One row (token) per CTA: x = base + mult * gain * (y / rms(y)); the row itself, or its RMS norm, is the next operand.
//   base   embedding row of tokens[row] plus the position vector of pos0 + row, or row rows[i] (default i) of X
//   y      a sublayer's rows, or the weighted sum of expert rows and a gated shared row (moe_top > 0); null: x = base
struct PostRows {
  const uint32_t* tokens = nullptr;
  const void* embed = nullptr;        // [V][H] of embed_dtype
  int embed_dtype = 0;
  const double* freq = nullptr;       // [(H+1)/2] angles per position of the position vector; null: none
  uint32_t pos0 = 0;
  const float* X = nullptr;           // [..][H]
  const uint32_t* rows = nullptr;
  const float* y = nullptr;           // [T][H]; with moe_top: the shared feed-forward's rows (may be null)
  uint32_t moe_top = 0;
  const float* ye = nullptr;          // expert rows [T*top][H]
  const uint32_t* where = nullptr;    // [T][top] rows of ye
  const float* w = nullptr;           // [T][top]
  const float* shared_gate = nullptr; // its sigmoid scales row t of y; shared_ld floats apart
  uint32_t shared_ld = 0;
  const float* gain = nullptr;        // one number
  float mult = 0.f, eps = 0.f;
  float* X_out = nullptr;             // [T][H]
  void* operand = nullptr;            // [T][H] of operand_dtype
  int operand_dtype = 0;
  const float* norm_gain = nullptr;   // one number: the operand is x / rms(x) * norm_gain
  float* tap = nullptr;               // [H] copy of row tap_row of x
  uint32_t tap_row = 0;
  uint32_t H = 0;
};
cudaError_t launch_post_rows(cudaStream_t s, const PostRows& p, uint32_t n_rows);
// Decode step: embedding plus position vector of the token in *state (its prompt buffer if given).
cudaError_t launch_embed_position(cudaStream_t s, int wdtype, const void* E, uint32_t H, uint32_t V, StepState* state,
                                  const uint32_t* prompt, const double* freq, float* x, bool pdl);

// ---- grouped-query attention with head norms, distance bias and head gates (gqa_decode.cu, gqa_prefill.cu) ---------------
struct GqaParams {
  GqaSpec spec;
  const float* in = nullptr;   // projected rows [q | k | v | gate], in_ld floats apart
  uint32_t in_ld = 0;
  float eps = 0.f;
  void* k_cache = nullptr;     // [ctx][kv_heads*dim] of dtype, normed
  void* v_cache = nullptr;     // [ctx][kv_heads*vdim] of dtype, normed
  int dtype = 0;               // of caches and operands: 0 or 2
  uint32_t ctx = 0;
  StepState* state = nullptr;  // decode: position
  uint32_t pos0 = 0;           // prompt path: position of the first token
  // decode
  float* out = nullptr;        // [heads*vdim], gated
  float* part = nullptr;       // gqa_decode_scratch bytes, zero-filled once (split partials, then tickets)
  // prompt path
  void* q = nullptr;           // [T][heads*dim] of dtype, normed, times scale * log2(e)
  void* ao = nullptr;          // [T][heads*vdim] of dtype, gated
};
bool gqa_supported(const GqaSpec& s, std::string* why);
size_t gqa_decode_scratch(const GqaSpec& s, uint32_t ctx);
// Rows of one KV head's keys a decode step at position `pos` has to read, summed over the KV heads.
uint64_t gqa_rows_read(const GqaSpec& s, uint32_t pos);
cudaError_t launch_gqa_decode(cudaStream_t s, const GqaParams& p, bool pdl);
// Norm what the projection of T tokens left: cache rows pos0 .. pos0+T-1 (unless borrowed) and p.q.
cudaError_t launch_gqa_prep(cudaStream_t s, const GqaParams& p, uint32_t T);
cudaError_t launch_gqa_prefill(cudaStream_t s, const GqaParams& p, uint32_t T);

// ---- routed feed-forwards over rows of tokens (moe.cu) -------------------------------------------------------------------
struct MoeRows {
  Router router;
  const float* logits = nullptr;  // [T][ld]
  uint32_t ld = 0;
  uint32_t* ids = nullptr;        // [T][top]
  float* w = nullptr;             // [T][top]
  uint32_t* where = nullptr;      // [T][top] row of the sorted order
  uint32_t* src = nullptr;        // [T*top] token of a sorted row
  uint32_t* rows = nullptr;       // [experts + 1]
  uint2* tiles = nullptr;         // moe_max_tiles entries
  uint32_t* n_tiles = nullptr;
};
uint32_t moe_max_tiles(const MoeSpec& s, uint32_t T);
// Choose experts for T tokens and sort the (token, choice) pairs by expert, tokens in order.
cudaError_t launch_moe_route(cudaStream_t s, const MoeRows& p, uint32_t T);
// out[i] = A[src[i]]: operand rows of H elements (elem bytes each) in sorted order.
cudaError_t launch_moe_gather(cudaStream_t s, const void* A, const uint32_t* src, uint32_t n, uint32_t H, uint32_t elem, void* out);

}  // namespace nfai
