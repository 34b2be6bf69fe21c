// Hyper-connections on rows of tokens: the residual is S streams per token. One CTA brings the streams of one token up to
// date with a sublayer's output, forms the weighted sum the next sublayer reads, and normalises it, in one pass over the
// streams (the S*H floats are read and written once; the combined row waits in shared memory for its root mean square).
// All of it is float32; only the normalised row, the operand of the next product, takes the operand type.
#include "plan_kernels.h"
#include "common.cuh"

namespace nfai {

namespace {

__device__ __forceinline__ void store_typed(void* p, int dtype, size_t at, float v) {
  if (dtype == 0) reinterpret_cast<float*>(p)[at] = v;
  else if (dtype == 1) store_as(reinterpret_cast<__half*>(p) + at, v);
  else store_as(reinterpret_cast<__nv_bfloat16*>(p) + at, v);
}
__device__ __forceinline__ float load_typed(const void* p, int dtype, size_t at) {
  if (dtype == 0) return reinterpret_cast<const float*>(p)[at];
  if (dtype == 1) return to_float(reinterpret_cast<const __half*>(p)[at]);
  return to_float(reinterpret_cast<const __nv_bfloat16*>(p)[at]);
}

template <int V>
struct Vec {
  float f[V];
};
template <int V>
__device__ __forceinline__ Vec<V> ldv(const float* p) {
  Vec<V> r;
  if constexpr (V == 4) {
    const float4 q = *reinterpret_cast<const float4*>(p);
    r.f[0] = q.x; r.f[1] = q.y; r.f[2] = q.z; r.f[3] = q.w;
  } else {
    r.f[0] = *p;
  }
  return r;
}
template <int V>
__device__ __forceinline__ void stv(float* p, const Vec<V>& v) {
  if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(v.f[0], v.f[1], v.f[2], v.f[3]);
  else *p = v.f[0];
}

// ST >= S streams held in registers; V elements per thread and step
template <int ST, int V>
__global__ void __launch_bounds__(256, ST <= 4 ? 3 : 1) hyper_rows_kernel(const HyperRows p) {
  extern __shared__ __align__(16) float hsm[];
  float* us = hsm;  // [H] combined row
  __shared__ float w_mix[kMaxStreams * kMaxStreams], w_out[kMaxStreams], w_in[kMaxStreams], red[8];
  const uint32_t S = p.S, H = p.H, tid = threadIdx.x;
  for (uint32_t i = tid; i < S * S; i += 256) w_mix[i] = p.mix ? p.mix[i] : 0.f;
  if (tid < S) {
    w_out[tid] = p.out ? p.out[tid] : 0.f;
    w_in[tid] = p.next_in ? p.next_in[tid] : 1.f;
  }
  pdl_launch_dependents();
  pdl_wait();
  __syncthreads();
  const size_t row = p.rows ? p.rows[blockIdx.x] : blockIdx.x;
  const float* X = p.X ? p.X + row * S * H : nullptr;
  float* Xo = p.X_out ? p.X_out + (size_t)blockIdx.x * S * H : nullptr;
  const size_t erow = p.tokens ? (size_t)p.tokens[blockIdx.x] * H : 0;
  float ss = 0.f;
#pragma unroll 1
  for (uint32_t i = tid * V; i < H; i += 256 * V) {
    Vec<V> x[ST];
    if (p.tokens) {
#pragma unroll
      for (int e = 0; e < V; ++e) {
        const float v = load_typed(p.embed, p.embed_dtype, erow + i + e);
#pragma unroll
        for (int s = 0; s < ST; ++s) x[s].f[e] = v;
      }
    } else {
#pragma unroll
      for (int s = 0; s < ST; ++s)
        if (s < (int)S) x[s] = ldv<V>(X + (size_t)s * H + i);
    }
    if (p.y) {
      const Vec<V> y = ldv<V>(p.y + row * H + i);
      Vec<V> n[ST];
#pragma unroll
      for (int t = 0; t < ST; ++t)
        if (t < (int)S) {
#pragma unroll
          for (int e = 0; e < V; ++e) n[t].f[e] = w_out[t] * y.f[e];
#pragma unroll
          for (int s = 0; s < ST; ++s)
            if (s < (int)S) {
              const float w = w_mix[s * S + t];
#pragma unroll
              for (int e = 0; e < V; ++e) n[t].f[e] = fmaf(w, x[s].f[e], n[t].f[e]);
            }
        }
#pragma unroll
      for (int t = 0; t < ST; ++t) x[t] = n[t];
    }
    Vec<V> u;
#pragma unroll
    for (int e = 0; e < V; ++e) u.f[e] = 0.f;
#pragma unroll
    for (int t = 0; t < ST; ++t)
      if (t < (int)S) {
        if (Xo) stv<V>(Xo + (size_t)t * H + i, x[t]);
#pragma unroll
        for (int e = 0; e < V; ++e) u.f[e] = fmaf(w_in[t], x[t].f[e], u.f[e]);
      }
    if (p.u_out) stv<V>(p.u_out + (size_t)blockIdx.x * H + i, u);
    stv<V>(us + i, u);
#pragma unroll
    for (int e = 0; e < V; ++e) ss = fmaf(u.f[e], u.f[e], ss);
  }
  if (!p.normed) return;
  ss = warp_sum(ss);
  if ((tid & 31) == 0) red[tid >> 5] = ss;
  __syncthreads();
  float tot = 0.f;
#pragma unroll
  for (int w = 0; w < 8; ++w) tot += red[w];
  const float rms = sqrtf(__fdiv_rn(tot, (float)H) + p.eps);
  for (uint32_t i = tid * V; i < H; i += 256 * V) {
    const Vec<V> u = ldv<V>(us + i), g = ldv<V>(p.gain + i);
    float o[V];
#pragma unroll
    for (int e = 0; e < V; ++e) o[e] = __fmul_rn(__fdiv_rn(u.f[e], rms), g.f[e]);
    const size_t at = (size_t)blockIdx.x * H + i;
    if (V == 4 && p.normed_dtype == 2) {
      __nv_bfloat162 b[2] = {__floats2bfloat162_rn(o[0], o[1]), __floats2bfloat162_rn(o[V > 2 ? 2 : 0], o[V > 3 ? 3 : 0])};
      *reinterpret_cast<uint2*>(reinterpret_cast<__nv_bfloat16*>(p.normed) + at) = *reinterpret_cast<uint2*>(b);
    } else {
#pragma unroll
      for (int e = 0; e < V; ++e) store_typed(p.normed, p.normed_dtype, at + e, o[e]);
    }
  }
}

template <int ST>
cudaError_t launch_st(cudaStream_t s, const HyperRows& p, uint32_t n) {
  const size_t smem = (size_t)p.H * 4;
  if (smem > 200 * 1024) return cudaErrorInvalidValue;
  auto kern = hyper_rows_kernel<ST, 1>;
  if constexpr (ST <= 8) {  // more streams would not fit the register file in quads
    if (p.H % 4 == 0) kern = hyper_rows_kernel<ST, 4>;
  }
  if (smem > 40 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return e;
  }
  return launch_pdl(kern, dim3(n), dim3(256), smem, s, prefill_pdl(), p);
}

template <typename WT>
__global__ void embed_streams_kernel(const WT* __restrict__ E, uint32_t H, uint32_t V, uint32_t S, StepState* state,
                                     const uint32_t* __restrict__ prompt, const float* __restrict__ first_in,
                                     float* __restrict__ X, float* __restrict__ u) {
  pdl_launch_dependents();
  pdl_wait();
  uint32_t tok = prompt ? prompt[state->prompt_idx] : state->cur_token;
  if (tok >= V) {
    if (threadIdx.x == 0 && blockIdx.x == 0) atomicOr(&state->err, 1u);
    tok = 0;
  }
  float w = 0.f;
  for (uint32_t s = 0; s < S; ++s) w += first_in[s];
  for (uint32_t i = blockIdx.x * blockDim.x + threadIdx.x; i < H; i += gridDim.x * blockDim.x) {
    const float v = to_float(E[(size_t)tok * H + i]);
    for (uint32_t s = 0; s < S; ++s) X[(size_t)s * H + i] = v;
    u[i] = w * v;
  }
}

}  // namespace

cudaError_t launch_hyper_rows(cudaStream_t s, const HyperRows& p, uint32_t n) {
  if (!n || !p.H || !p.S || p.S > kMaxStreams || (!p.tokens && !p.X)) return cudaErrorInvalidValue;
  if (p.S == 1) return launch_st<1>(s, p, n);
  if (p.S == 2) return launch_st<2>(s, p, n);
  if (p.S <= 4) return launch_st<4>(s, p, n);
  if (p.S <= 8) return launch_st<8>(s, p, n);
  return launch_st<16>(s, p, n);
}

cudaError_t launch_embed_streams(cudaStream_t s, int wdtype, const void* E, uint32_t H, uint32_t V, uint32_t S, StepState* state,
                                 const uint32_t* prompt, const float* first_in, float* X, float* u, bool pdl) {
  const dim3 grid((H + 255) / 256), block(256);
  if (wdtype == 2)
    return launch_pdl(embed_streams_kernel<__nv_bfloat16>, grid, block, 0, s, pdl, (const __nv_bfloat16*)E, H, V, S, state, prompt, first_in, X, u);
  if (wdtype == 1)
    return launch_pdl(embed_streams_kernel<__half>, grid, block, 0, s, pdl, (const __half*)E, H, V, S, state, prompt, first_in, X, u);
  return launch_pdl(embed_streams_kernel<float>, grid, block, 0, s, pdl, (const float*)E, H, V, S, state, prompt, first_in, X, u);
}

}  // namespace nfai
