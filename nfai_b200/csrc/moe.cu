// Routed feed-forwards over rows of tokens: choice of experts, and the order in which their products run. The (token, choice)
// pairs are sorted by expert so that an expert's rows are neighbours and every weight matrix is read once per pass:
//   moe_choose  a warp per token (moe_route.cuh)
//   moe_sort    a CTA per expert counts the pairs of the lower experts and ranks its own in token order; no atomics on the
//               order, so a pass gives the same rows at the same places every time. It also lists the row tiles of the
//               grouped product.
//   moe_gather  operand rows in sorted order
// The grouped products themselves are gemm_tc.cu / gemm_simt.cu, the weighted sum is formed in post_rows.cu.
#include "moe_route.cuh"
#include "plan_kernels.h"

namespace nfai {

namespace {

constexpr int kCW = 8;    // warps (tokens) per CTA of moe_choose
constexpr int kST = 512;  // threads of moe_sort

__global__ void __launch_bounds__(kCW * 32) moe_choose_kernel(const MoeRows p, const uint32_t T) {
  extern __shared__ float csm[];  // route_floats(experts) per warp
  pdl_launch_dependents();
  pdl_wait();
  const uint32_t warp = threadIdx.x >> 5, t = blockIdx.x * kCW + warp;
  if (t >= T) return;
  route_warp(p.router, p.logits + (size_t)t * p.ld, csm + warp * route_floats(p.router.experts), p.ids + (size_t)t * p.router.top, p.w + (size_t)t * p.router.top);
}

// exclusive prefix sum over the CTA; *total receives the sum
__device__ __forceinline__ uint32_t cta_prefix(uint32_t v, uint32_t* sums, uint32_t* total) {
  const uint32_t lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  uint32_t x = v;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const uint32_t n = __shfl_up_sync(0xffffffffu, x, o);
    if ((int)lane >= o) x += n;
  }
  __syncthreads();
  if (lane == 31) sums[warp] = x;
  __syncthreads();
  uint32_t before = 0, all = 0;
  for (uint32_t w = 0; w < kST / 32; ++w) {
    const uint32_t s = sums[w];
    before += w < warp ? s : 0u;
    all += s;
  }
  *total = all;
  return before + x - v;
}

__global__ void __launch_bounds__(kST) moe_sort_kernel(const MoeRows p, const uint32_t n) {
  extern __shared__ uint32_t hist[];  // [experts]
  __shared__ uint32_t sums[kST / 32];
  const uint32_t E = p.router.experts, top = p.router.top, e = blockIdx.x, tid = threadIdx.x;
  for (uint32_t i = tid; i < E; i += kST) hist[i] = 0;
  __syncthreads();
  pdl_launch_dependents();
  pdl_wait();
  for (uint32_t i = tid; i < n; i += kST) atomicAdd(&hist[min(p.ids[i], E - 1)], 1u);
  __syncthreads();
  // rows and row tiles of the experts before this one
  uint32_t rows = 0, tiles = 0;
  for (uint32_t i = tid; i < e; i += kST) {
    rows += hist[i];
    tiles += (hist[i] + kGroupTile - 1) / kGroupTile;
  }
  uint32_t row0, tile0, any;
  cta_prefix(rows, sums, &row0);
  cta_prefix(tiles, sums, &tile0);
  const uint32_t mine = hist[e], my_tiles = (mine + kGroupTile - 1) / kGroupTile;
  if (tid == 0) {
    p.rows[e] = row0;
    if (e == E - 1) {
      p.rows[E] = row0 + mine;
      *p.n_tiles = tile0 + my_tiles;
    }
  }
  for (uint32_t i = tid; i < my_tiles; i += kST) p.tiles[tile0 + i] = make_uint2(e, row0 + i * kGroupTile);
  // this expert's pairs, in order: a warp takes a run of them, counts its hits, and ranks them behind the earlier warps'
  const uint32_t lane = tid & 31, warp = tid >> 5, run = ((n + kST / 32 - 1) / (kST / 32) + 31) & ~31u;
  const uint32_t i0 = min(warp * run, n), i1 = min(i0 + run, n);
  uint32_t hits = 0;
#pragma unroll 4
  for (uint32_t i = i0 + lane; i < i1; i += 32) hits += min(p.ids[i], E - 1) == e ? 1u : 0u;
  hits = __reduce_add_sync(0xffffffffu, hits);
  uint32_t at = row0 + cta_prefix(lane == 0 ? hits : 0u, sums, &any);
  at = __shfl_sync(0xffffffffu, at, 0);
  if (!hits) return;
#pragma unroll 4
  for (uint32_t base = i0; base < i1; base += 32) {
    const uint32_t i = base + lane;
    const bool hit = i < i1 && min(p.ids[i], E - 1) == e;
    const uint32_t mask = __ballot_sync(0xffffffffu, hit);
    if (hit) {
      const uint32_t to = at + __popc(mask & ((1u << lane) - 1u));
      p.where[i] = to;
      p.src[to] = i / top;
    }
    at += __popc(mask);
  }
}

template <typename V>
__global__ void __launch_bounds__(256) moe_gather_kernel(const V* __restrict__ A, const uint32_t* __restrict__ src, uint32_t per_row, V* __restrict__ out) {
  pdl_launch_dependents();
  pdl_wait();
  const V* a = A + (size_t)src[blockIdx.x] * per_row;
  V* o = out + (size_t)blockIdx.x * per_row;
  for (uint32_t i = threadIdx.x; i < per_row; i += 256) o[i] = a[i];
}

}  // namespace

uint32_t moe_max_tiles(const MoeSpec& s, uint32_t T) { return (T * s.top + kGroupTile - 1) / kGroupTile + s.experts; }

cudaError_t launch_moe_route(cudaStream_t s, const MoeRows& p, uint32_t T) {
  const Router& r = p.router;
  if (!T || !r.experts || r.experts > kMaxExperts || !r.top || r.top > kMaxChosen || r.groups > kMaxGroups || !r.groups || r.experts % r.groups)
    return cudaErrorInvalidValue;
  const size_t smem = (size_t)kCW * route_floats(r.experts) * 4;
  cudaError_t e = cudaSuccess;
  if (smem > 40 * 1024 &&
      (e = cudaFuncSetAttribute(moe_choose_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem)) != cudaSuccess)
    return e;
  e = launch_pdl(moe_choose_kernel, dim3((T + kCW - 1) / kCW), dim3(kCW * 32), smem, s, prefill_pdl(), p, T);
  if (e != cudaSuccess) return e;
  return launch_pdl(moe_sort_kernel, dim3(r.experts), dim3(kST), (size_t)r.experts * 4, s, prefill_pdl(), p, T * r.top);
}

cudaError_t launch_moe_gather(cudaStream_t s, const void* A, const uint32_t* src, uint32_t n, uint32_t H, uint32_t elem, void* out) {
  const size_t bytes = (size_t)H * elem;
  if (!n || !H) return cudaErrorInvalidValue;
  if (bytes % 16 == 0 && (((uintptr_t)A | (uintptr_t)out) & 15) == 0)
    return launch_pdl(moe_gather_kernel<uint4>, dim3(n), dim3(256), 0, s, prefill_pdl(), (const uint4*)A, src, (uint32_t)(bytes / 16), (uint4*)out);
  return launch_pdl(moe_gather_kernel<uint16_t>, dim3(n), dim3(256), 0, s, prefill_pdl(), (const uint16_t*)A, src, (uint32_t)(bytes / 2), (uint16_t*)out);
}

}  // namespace nfai
