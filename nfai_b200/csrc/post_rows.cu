// A residual that takes normed sublayer outputs, on rows of tokens: x += mult * gain * y / rms(y), one CTA per token. The
// weighted sum of a routed feed-forward's expert rows is formed on the way in, the operand of the next product (the row
// itself, or its norm in front of the output matrix) on the way out, so a sublayer boundary is one pass over the rows.
// All of it is float32 but the operand. Also the start of the stream: embedding plus a sinusoidal position vector.
#include "common.cuh"
#include "plan_kernels.h"

namespace nfai {

namespace {

constexpr int kPT = 256;

__device__ __forceinline__ float load_embed(const void* p, int dtype, size_t at) {
  if (dtype == 0) return reinterpret_cast<const float*>(p)[at];
  if (dtype == 1) return to_float(reinterpret_cast<const __half*>(p)[at]);
  return to_float(reinterpret_cast<const __nv_bfloat16*>(p)[at]);
}

// Entry i of the position vector: sine (even i) or cosine of position * freq[i/2]. The angle is formed and reduced in
// double precision: as one float32 product it would lose the place within a turn at large positions.
__device__ __forceinline__ float position_entry(const double* freq, uint32_t pos, uint32_t i) {
  constexpr double kTurn = 6.283185307179586;
  double a = (double)pos * freq[i >> 1];
  a -= kTurn * rint(a / kTurn);
  return i & 1u ? cosf((float)a) : sinf((float)a);
}

__device__ __forceinline__ float rows_sum(float v, float* red) {
  v = warp_sum(v);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = 0.f;
#pragma unroll
  for (int w = 0; w < kPT / 32; ++w) t += red[w];
  __syncthreads();
  return t;
}

template <int V>
struct Vals {
  float f[V];
};
template <int V>
__device__ __forceinline__ Vals<V> get(const float* p) {
  Vals<V> r;
  if constexpr (V == 4) {
    const float4 q = *reinterpret_cast<const float4*>(p);
    r.f[0] = q.x; r.f[1] = q.y; r.f[2] = q.z; r.f[3] = q.w;
  } else {
    r.f[0] = *p;
  }
  return r;
}
template <int V>
__device__ __forceinline__ void put(float* p, const Vals<V>& v) {
  if constexpr (V == 4) *reinterpret_cast<float4*>(p) = make_float4(v.f[0], v.f[1], v.f[2], v.f[3]);
  else *p = v.f[0];
}
template <int V>
__device__ __forceinline__ void put_operand(void* out, int dtype, size_t at, const Vals<V>& v) {
  if (V == 4 && dtype == 2) {
    __nv_bfloat162 b[2] = {__floats2bfloat162_rn(v.f[0], v.f[V > 1 ? 1 : 0]), __floats2bfloat162_rn(v.f[V > 2 ? 2 : 0], v.f[V > 3 ? 3 : 0])};
    *reinterpret_cast<uint2*>(reinterpret_cast<__nv_bfloat16*>(out) + at) = *reinterpret_cast<uint2*>(b);
    return;
  }
#pragma unroll
  for (int e = 0; e < V; ++e) {
    if (dtype == 0) reinterpret_cast<float*>(out)[at + e] = v.f[e];
    else if (dtype == 1) store_as(reinterpret_cast<__half*>(out) + at + e, v.f[e]);
    else store_as(reinterpret_cast<__nv_bfloat16*>(out) + at + e, v.f[e]);
  }
}

template <int V>
__global__ void __launch_bounds__(kPT) post_rows_kernel(const PostRows p) {
  extern __shared__ __align__(16) float psm[];
  float* const ys = psm;  // [H] y, then x when its norm is wanted
  __shared__ float red[kPT / 32], wk[kMaxChosen];
  __shared__ uint32_t wh[kMaxChosen];
  const uint32_t H = p.H, tid = threadIdx.x, b = blockIdx.x;
  pdl_launch_dependents();
  pdl_wait();
  const size_t row = p.rows ? p.rows[b] : b;
  const bool add = p.y || p.moe_top;
  float c = 0.f, rms = 1.f;
  if (add) {
    float ss = 0.f, sg = 1.f;
    if (p.moe_top) {
      if (tid < p.moe_top) {
        wk[tid] = p.w[(size_t)b * p.moe_top + tid];
        wh[tid] = p.where[(size_t)b * p.moe_top + tid];
      }
      if (p.y) sg = __fdiv_rn(1.0f, 1.0f + expf(-p.shared_gate[(size_t)b * p.shared_ld]));
      __syncthreads();
    }
    for (uint32_t i = tid * V; i < H; i += kPT * V) {
      Vals<V> y;
      if (p.y) y = get<V>(p.y + row * H + i);
      if (p.moe_top) {
#pragma unroll
        for (int e = 0; e < V; ++e) y.f[e] = p.y ? sg * y.f[e] : 0.f;
#pragma unroll 4
        for (uint32_t k = 0; k < p.moe_top; ++k) {
          const Vals<V> v = get<V>(p.ye + (size_t)wh[k] * H + i);
#pragma unroll
          for (int e = 0; e < V; ++e) y.f[e] = fmaf(wk[k], v.f[e], y.f[e]);
        }
      }
      put<V>(ys + i, y);
#pragma unroll
      for (int e = 0; e < V; ++e) ss = fmaf(y.f[e], y.f[e], ss);
    }
    rms = sqrtf(__fdiv_rn(rows_sum(ss, red), (float)H) + p.eps);
    c = p.mult * *p.gain;
  }
  const size_t erow = p.tokens ? (size_t)p.tokens[b] * H : 0;
  float sx = 0.f;
  for (uint32_t i = tid * V; i < H; i += kPT * V) {
    Vals<V> x;
    if (p.tokens) {
#pragma unroll
      for (int e = 0; e < V; ++e) {
        x.f[e] = load_embed(p.embed, p.embed_dtype, erow + i + e);
        if (p.freq) x.f[e] += position_entry(p.freq, p.pos0 + b, i + e);
      }
    } else {
      x = get<V>(p.X + row * H + i);
    }
    if (add) {
      const Vals<V> y = get<V>(ys + i);
#pragma unroll
      for (int e = 0; e < V; ++e) x.f[e] = fmaf(c, __fdiv_rn(y.f[e], rms), x.f[e]);
    }
    if (p.X_out) put<V>(p.X_out + (size_t)b * H + i, x);
    if (p.tap && b == p.tap_row) put<V>(p.tap + i, x);
    if (!p.operand) continue;
    if (!p.norm_gain) {
      put_operand<V>(p.operand, p.operand_dtype, (size_t)b * H + i, x);
    } else {
      put<V>(ys + i, x);  // (this thread's own elements)
#pragma unroll
      for (int e = 0; e < V; ++e) sx = fmaf(x.f[e], x.f[e], sx);
    }
  }
  if (!p.operand || !p.norm_gain) return;
  const float rx = sqrtf(__fdiv_rn(rows_sum(sx, red), (float)H) + p.eps), g = *p.norm_gain;
  for (uint32_t i = tid * V; i < H; i += kPT * V) {
    Vals<V> x = get<V>(ys + i);
#pragma unroll
    for (int e = 0; e < V; ++e) x.f[e] = __fmul_rn(__fdiv_rn(x.f[e], rx), g);
    put_operand<V>(p.operand, p.operand_dtype, (size_t)b * H + i, x);
  }
}

template <typename WT>
__global__ void embed_position_kernel(const WT* __restrict__ E, uint32_t H, uint32_t V, StepState* state, const uint32_t* __restrict__ prompt,
                                      const double* __restrict__ freq, float* __restrict__ x) {
  pdl_launch_dependents();
  pdl_wait();
  uint32_t tok = prompt ? prompt[state->prompt_idx] : state->cur_token;
  if (tok >= V) {
    if (threadIdx.x == 0 && blockIdx.x == 0) atomicOr(&state->err, 1u);
    tok = 0;
  }
  const uint32_t pos = state->pos;
  for (uint32_t i = blockIdx.x * blockDim.x + threadIdx.x; i < H; i += gridDim.x * blockDim.x)
    x[i] = to_float(E[(size_t)tok * H + i]) + (freq ? position_entry(freq, pos, i) : 0.f);
}

}  // namespace

cudaError_t launch_post_rows(cudaStream_t s, const PostRows& p, uint32_t n) {
  if (!n || !p.H || (!p.tokens && !p.X) || p.moe_top > kMaxChosen || ((p.y || p.moe_top) && !p.gain)) return cudaErrorInvalidValue;
  if (p.moe_top && (!p.ye || !p.where || !p.w || (p.y && !p.shared_gate) || p.rows)) return cudaErrorInvalidValue;
  const size_t smem = (size_t)p.H * 4;
  if (smem > 200 * 1024) return cudaErrorInvalidValue;
  auto kern = p.H % 4 == 0 ? post_rows_kernel<4> : post_rows_kernel<1>;
  if (smem > 40 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return e;
  }
  return launch_pdl(kern, dim3(n), dim3(kPT), smem, s, prefill_pdl(), p);
}

cudaError_t launch_embed_position(cudaStream_t s, int wdtype, const void* E, uint32_t H, uint32_t V, StepState* state,
                                  const uint32_t* prompt, const double* freq, float* x, bool pdl) {
  const dim3 grid((H + 255) / 256), block(256);
  if (wdtype == 2) return launch_pdl(embed_position_kernel<__nv_bfloat16>, grid, block, 0, s, pdl, (const __nv_bfloat16*)E, H, V, state, prompt, freq, x);
  if (wdtype == 1) return launch_pdl(embed_position_kernel<__half>, grid, block, 0, s, pdl, (const __half*)E, H, V, state, prompt, freq, x);
  return launch_pdl(embed_position_kernel<float>, grid, block, 0, s, pdl, (const float*)E, H, V, state, prompt, freq, x);
}

}  // namespace nfai
