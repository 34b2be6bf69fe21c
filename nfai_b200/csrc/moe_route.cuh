// Choice of experts for one token by one warp, shared by the decode GEMV and the prompt path.
//   score s_e = sigmoid(z_e), choice score c_e = s_e + correction_e
//   a group's score is the sum of its two largest choice scores; the best `keep` groups stay
//   the `top` largest choice scores among their experts are chosen, equal scores in the order of the experts
//   weight of a chosen expert: s_e / (sum of the chosen s + 1e-20) * scale
// All of it is float32.
#pragma once
#include <math.h>

#include "common.cuh"
#include "kernels.h"
#include "plan.h"

namespace nfai {

// float -> unsigned with the same order, so that a warp's maximum is one reduction
__device__ __forceinline__ uint32_t ordered_bits(float v) {
  const uint32_t b = __float_as_uint(v);
  return b & 0x80000000u ? ~b : b | 0x80000000u;
}
__device__ __forceinline__ float route_sigmoid(float z) { return __fdiv_rn(1.0f, 1.0f + expf(-z)); }

constexpr uint32_t kRouteScratch = kMaxGroups;  // floats beside the experts' scores and choice scores
constexpr uint32_t route_floats(uint32_t experts) { return 2 * experts + kRouteScratch; }

// scratch: route_floats(experts) floats of shared memory of this warp; ids and w: [top], shared memory or global. Every lane
// calls it; the results are visible to the warp when it returns.
__device__ __forceinline__ void route_warp(const Router& r, const float* z, float* scratch, uint32_t* ids, float* w) {
  const uint32_t lane = threadIdx.x & 31, E = r.experts;
  constexpr uint32_t kAll = 0xffffffffu;
  float *const gs = scratch, *const cs = gs + kRouteScratch, *const sc = cs + E;
#pragma unroll 4
  for (uint32_t e = lane; e < E; e += 32) {
    const float s = route_sigmoid(__ldcg(z + e));
    sc[e] = s;
    cs[e] = s + __ldg(r.correction + e);
  }
  __syncwarp();
  if (r.keep < r.groups) {
    const uint32_t size = E / r.groups;
    // LG lanes share a group, so that small numbers of groups do not leave most lanes idle
    uint32_t LG = 1;
    while (2 * LG * r.groups <= 32) LG <<= 1;
    for (uint32_t g0 = 0; g0 < r.groups; g0 += 32 / LG) {
      const uint32_t g = g0 + lane / LG;
      float a = -INFINITY, b = -INFINITY;  // the two largest
      if (g < r.groups)
        for (uint32_t i = lane % LG; i < size; i += LG) {
          const float v = cs[g * size + i];
          b = fmaxf(b, fminf(a, v));
          a = fmaxf(a, v);
        }
      for (uint32_t o = 1; o < LG; o <<= 1) {
        const float a2 = __shfl_xor_sync(kAll, a, o), b2 = __shfl_xor_sync(kAll, b, o);
        b = fmaxf(fmaxf(b, b2), fminf(a, a2));
        a = fmaxf(a, a2);
      }
      if (g < r.groups && lane % LG == 0) gs[g] = size > 1 ? a + b : a;
    }
    __syncwarp();
    // a group stays if fewer than `keep` are better (lower index first among equals)
    for (uint32_t g = lane; g < r.groups; g += 32) {
      const float v = gs[g];
      uint32_t better = 0;
      for (uint32_t j = 0; j < r.groups; ++j) better += gs[j] > v || (gs[j] == v && j < g) ? 1u : 0u;
      if (better >= r.keep)
        for (uint32_t i = 0; i < size; ++i) cs[g * size + i] = -INFINITY;
    }
    __syncwarp();
  }
  // a lane keeps the best of its own experts (lane, lane + 32, ...) and looks again only after losing it
  uint32_t best = 0u, best_e = 0xffffffffu;
  auto scan = [&]() {
    best = 0u;
    best_e = 0xffffffffu;
    for (uint32_t e = lane; e < E; e += 32) {
      const uint32_t b = ordered_bits(cs[e]);
      if (best_e == 0xffffffffu || b > best) {
        best = b;
        best_e = e;
      }
    }
  };
  scan();
  float sum = 0.f, mine = 0.f;
  uint32_t my_id = 0;
  for (uint32_t k = 0; k < r.top; ++k) {
    const uint32_t m = __reduce_max_sync(kAll, best);
    uint32_t e = __reduce_min_sync(kAll, best == m ? best_e : 0xffffffffu);
    if (e >= E) e = 0;  // (a score that is not a number: any valid index)
    if (best_e == e) {
      cs[e] = -INFINITY;
      scan();
    }
    const float s = sc[e];
    sum += s;
    if (lane == k) {
      mine = s;
      my_id = e;
    }
  }
  if (lane < r.top) {
    ids[lane] = my_id;
    w[lane] = __fdiv_rn(mine, sum + 1e-20f) * r.scale;
  }
  __syncwarp();
}

}  // namespace nfai
