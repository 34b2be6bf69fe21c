// Device helpers shared by the latent attention kernels.
#pragma once
#include "attn_core.cuh"
#include "plan_kernels.h"

namespace nfai {
namespace latent_detail {

constexpr float kNeg = attn_detail::kNegBig;

__device__ __forceinline__ float sigmoid_f(float v) { return 1.0f / (1.0f + expf(-v)); }

// Rotated entry i of a key/query part held in `src`: entry i < half pairs with i + half; entries past 2 half pass.
__device__ __forceinline__ float rotated(const float* src, uint32_t i, uint32_t dims, const float2* cs) {
  const uint32_t half = dims >> 1;
  if (i >= dims) return src[i];
  const uint32_t j = i < half ? i : i - half;
  const float2 r = cs[j];
  const float u = src[j], v = src[j + half];
  return i < half ? __fsub_rn(__fmul_rn(u, r.x), __fmul_rn(v, r.y)) : __fadd_rn(__fmul_rn(v, r.x), __fmul_rn(u, r.y));
}

template <typename T>
__device__ __forceinline__ T cast_to(float v) {
  T t;
  store_as(&t, v);
  return t;
}

// V consecutive elements -> float
template <typename T, int V>
__device__ __forceinline__ void load_vec(const T* p, float (&f)[V]) {
  if constexpr (V > 1) {
    static_assert(V == WeightVec<T>::kElems, "16-byte vectors");
    WeightVec<T>::unpack(*reinterpret_cast<const uint4*>(p), f);
  } else {
    f[0] = to_float(*p);
  }
}

__device__ __forceinline__ uint32_t cluster_rank() {
  uint32_t r;
  asm volatile("mov.u32 %0, %%cluster_ctarank;" : "=r"(r));
  return r;
}
__device__ __forceinline__ void cluster_arrive() { asm volatile("barrier.cluster.arrive.release;" ::: "memory"); }
__device__ __forceinline__ void cluster_wait() { asm volatile("barrier.cluster.wait.acquire;" ::: "memory"); }
// address of the same shared-memory location in CTA `rank` of the cluster
__device__ __forceinline__ uint32_t peer_addr(const void* p, uint32_t rank) {
  uint32_t a = (uint32_t)__cvta_generic_to_shared(p), r;
  asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(r) : "r"(a), "r"(rank));
  return r;
}
__device__ __forceinline__ void st_peer(uint32_t addr, float v) { asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(addr), "f"(v) : "memory"); }
__device__ __forceinline__ float ld_peer(uint32_t addr) {
  float v;
  asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(addr) : "memory");
  return v;
}
__device__ __forceinline__ void cp16(uint32_t dst, const void* src, uint32_t bytes) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// Vectors of eight floats are kept as two planes of float4, so that the 16-byte reads of neighbouring lanes are contiguous.
template <int VEC>
__device__ __forceinline__ uint32_t plane(uint32_t i, uint32_t nvec) {
  if constexpr (VEC == 8) {
    const uint32_t v = i >> 3, e = i & 7u;
    return (e >> 2) * nvec * 4 + v * 4 + (e & 3u);
  }
  return i;
}
template <int VEC>
__device__ __forceinline__ void load_plane(const float* p, uint32_t v, uint32_t nvec, float (&f)[VEC]) {
  if constexpr (VEC == 1) {
    f[0] = p[v];
  } else {
#pragma unroll
    for (int h = 0; h < VEC / 4; ++h) {
      const float4 a = *reinterpret_cast<const float4*>(p + h * nvec * 4 + v * 4);
      f[4 * h] = a.x; f[4 * h + 1] = a.y; f[4 * h + 2] = a.z; f[4 * h + 3] = a.w;
    }
  }
}

}  // namespace latent_detail
}  // namespace nfai
