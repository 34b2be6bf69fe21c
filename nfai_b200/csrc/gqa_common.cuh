// Shared by the decode and prompt kernels of grouped-query attention with head norms and a distance bias.
#pragma once
#include <math.h>

#include "attn_core.cuh"
#include "plan_kernels.h"

namespace nfai {
namespace gqa_detail {

constexpr float kLog2e = 1.4426950408889634f;
constexpr uint32_t kMaxHeadDim = 512;

__device__ __forceinline__ float gqa_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float head_sigmoid(float z) { return __fdiv_rn(1.0f, 1.0f + expf(-z)); }

// Distance bias of head h per position, in the base-2 domain; 0 without one.
__host__ __device__ __forceinline__ float slope2(const GqaSpec& s, uint32_t h) {
  return s.distance_bias ? exp2f(-8.0f * (float)(h + 1) / (float)s.heads) * kLog2e : 0.f;
}
// How many positions back a key can still count. Normed queries and keys bound a score by |scale| * dim, the key at the
// query's own position scores at least minus that, so a key whose bias exceeds twice the bound by 64 (base 2; 1 % on top for
// the rounding of cached rows) weighs less than 2^-64 of it: leaving those out is far below float32 rounding.
__host__ __device__ __forceinline__ uint32_t reach(const GqaSpec& s, float slope_2) {
  if (!s.qk_norm || !s.distance_bias) return 0xffffffffu;
  const float r = (2.04f * kLog2e * fabsf(s.scale) * (float)s.dim + 40.f) / slope_2;
  return r < 4.0e9f ? (uint32_t)r + 1u : 0xffffffffu;
}

// Eight consecutive cache elements, raw, of which the first n exist. VECT: n is 0 or at least 8 and p is 16-byte aligned.
template <typename CT, bool VECT>
struct Cache8;
template <bool VECT>
struct Cache8<float, VECT> {
  struct Raw { float f[8]; };
  __device__ __forceinline__ static Raw ld(const float* p, int n) {
    Raw r;
    if constexpr (VECT) {
      const float4 z = make_float4(0.f, 0.f, 0.f, 0.f);
      const float4 a = n > 0 ? __ldcg(reinterpret_cast<const float4*>(p)) : z, b = n > 0 ? __ldcg(reinterpret_cast<const float4*>(p) + 1) : z;
      r.f[0] = a.x; r.f[1] = a.y; r.f[2] = a.z; r.f[3] = a.w;
      r.f[4] = b.x; r.f[5] = b.y; r.f[6] = b.z; r.f[7] = b.w;
    } else {
#pragma unroll
      for (int e = 0; e < 8; ++e) r.f[e] = e < n ? __ldcg(p + e) : 0.f;
    }
    return r;
  }
  __device__ __forceinline__ static void unpack(const Raw& r, float (&f)[8]) {
#pragma unroll
    for (int e = 0; e < 8; ++e) f[e] = r.f[e];
  }
  __device__ __forceinline__ static Raw pack(const float (&f)[8]) {
    Raw r;
#pragma unroll
    for (int e = 0; e < 8; ++e) r.f[e] = f[e];
    return r;
  }
  __device__ __forceinline__ static void st(float* p, const Raw& r, int n) {
#pragma unroll
    for (int e = 0; e < 8; ++e)
      if (e < n) p[e] = r.f[e];
  }
};
template <bool VECT>
struct Cache8<__nv_bfloat16, VECT> {
  struct Raw { uint32_t w[4]; };
  __device__ __forceinline__ static Raw ld(const __nv_bfloat16* p, int n) {
    Raw r;
    if constexpr (VECT) {
      const uint4 v = n > 0 ? __ldcg(reinterpret_cast<const uint4*>(p)) : make_uint4(0, 0, 0, 0);
      r.w[0] = v.x; r.w[1] = v.y; r.w[2] = v.z; r.w[3] = v.w;
    } else {
      const unsigned short* h = reinterpret_cast<const unsigned short*>(p);
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const uint32_t lo = 2 * e < n ? __ldcg(h + 2 * e) : 0u, hi = 2 * e + 1 < n ? __ldcg(h + 2 * e + 1) : 0u;
        r.w[e] = lo | hi << 16;
      }
    }
    return r;
  }
  __device__ __forceinline__ static void unpack(const Raw& r, float (&f)[8]) {
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      f[2 * e] = __uint_as_float(r.w[e] << 16);
      f[2 * e + 1] = __uint_as_float(r.w[e] & 0xffff0000u);
    }
  }
  __device__ __forceinline__ static Raw pack(const float (&f)[8]) {
    Raw r;
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const __nv_bfloat162 h = __floats2bfloat162_rn(f[2 * e], f[2 * e + 1]);
      r.w[e] = *reinterpret_cast<const uint32_t*>(&h);
    }
    return r;
  }
  __device__ __forceinline__ static void st(__nv_bfloat16* p, const Raw& r, int n) {
    unsigned short* h = reinterpret_cast<unsigned short*>(p);
#pragma unroll
    for (int e = 0; e < 8; ++e)
      if (e < n) h[e] = (unsigned short)(r.w[e >> 1] >> (16 * (e & 1)));
  }
};

}  // namespace gqa_detail
}  // namespace nfai
