// Latent attention of one token with a bfloat16 cache, the products over the cached rows on the warp-level tensor cores.
//
// Three small kernels, so that programmatic launch can overlap each with its neighbours (one kernel with a cluster per head
// was slower inside the step: its shared memory keeps it from starting before its predecessor has left the SM):
//   latent_query   q_lat = W_uk^T q of every head, a slice of the latent dimensions per CTA, weights requested before the
//                  dependency wait; one more CTA norms and rotates the new position's latent and writes the cache rows.
//   latent_window  a CTA takes a run of cached rows and up to 16 heads, the rows of one MMA tile. The float32 query is split
//                  into three bfloat16 terms (24 bits together), one tile each, that accumulate into the same sums: one pass
//                  over a cached row serves all heads and all terms, and a row is read from memory once. Softmax over the
//                  run; the weights of the second product are split the same way. Leaves (sum of latents, maximum, sum of
//                  weights) per head.
//   latent_value   a cluster per head: each CTA merges its slice of the latent dimensions over all runs (in run order), the
//                  slices are shared through distributed shared memory, and each CTA maps them to a slice of the values
//                  through W_uv and applies the gate.
#include "latent_common.cuh"

namespace nfai {

namespace {

using namespace latent_detail;
using T = __nv_bfloat16;

constexpr int kMT = 256;          // threads of every kernel here
constexpr uint32_t kStage = 32;   // cache rows per stage of latent_window, one per lane in the softmax
constexpr uint32_t kHeads = 16;   // heads per CTA of latent_window, at most: the rows of a tile
constexpr uint32_t kSlice = 8;    // vectors of eight latent dimensions per CTA of latent_query
constexpr uint32_t kTerms = 3;

__host__ __device__ inline uint32_t head_groups(uint32_t heads) { return (heads + kHeads - 1) / kHeads; }
__host__ __device__ inline uint32_t heads_per_cta(uint32_t heads) { return (heads + head_groups(heads) - 1) / head_groups(heads); }

__device__ __forceinline__ void split3_pair(float a, float b, uint32_t& p0, uint32_t& p1, uint32_t& p2) {
  auto pk = [](float x, float y) {
    __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
    return *reinterpret_cast<uint32_t*>(&h);
  };
  p0 = pk(a, b);
  a -= __uint_as_float(p0 << 16);
  b -= __uint_as_float(p0 & 0xffff0000u);
  p1 = pk(a, b);
  p2 = pk(a - __uint_as_float(p1 << 16), b - __uint_as_float(p1 & 0xffff0000u));
}
__device__ __forceinline__ void split3_one(float a, T* r0, T* r1, T* r2) {
  *r0 = __float2bfloat16_rn(a);
  a -= __bfloat162float(*r0);
  *r1 = __float2bfloat16_rn(a);
  *r2 = __float2bfloat16_rn(a - __bfloat162float(*r1));
}
__device__ __forceinline__ void mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldsm(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm2(uint32_t addr, uint32_t& r0, uint32_t& r1) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];" : "=r"(r0), "=r"(r1) : "r"(addr));
}
__device__ __forceinline__ void ldsm_t(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr));
}

struct Window {
  uint32_t pos, lo, n;
};
__device__ __forceinline__ Window window_of(const LatentParams& p) {
  Window w;
  w.pos = p.state ? p.state->pos : p.pos0;
  if (w.pos >= p.ctx) w.pos = p.ctx - 1;  // reported by latent_query
  w.lo = p.spec.window && w.pos + 1 > p.spec.window ? w.pos + 1 - p.spec.window : 0u;
  w.n = w.pos - w.lo + 1;
  return w;
}

// ---- queries to latents; the new position's cache row ----------------------------------------------------------------------
// grid: heads x slices, then one CTA for the cache row. `qs`: [head groups][term][16 heads][rank + rot] bfloat16.
__global__ void __launch_bounds__(kMT) latent_query_kernel(const LatentParams p, T* __restrict__ qs, const uint32_t slices) {
  __shared__ float q[1024];
  __shared__ __align__(16) float part[kMT * 8];
  const LatentSpec& s = p.spec;
  const uint32_t rank = s.rank, rot = s.rot, dim = s.dim, D = rank + rot, hd = dim + rot, nv = rank / 8, tid = threadIdx.x;
  const uint32_t lane = tid & 31, warp = tid >> 5;
  if (blockIdx.x == s.heads * slices) {
    float* const raw = part;  // [D] <= 8 * kMT
    pdl_launch_dependents();
    pdl_wait();
    const uint32_t at = p.state ? p.state->pos : p.pos0;
    const bool full = at >= p.ctx;
    const uint32_t pos = full ? p.ctx - 1 : at;
    const float2* cs = p.rope_cs + (size_t)pos * (s.rope_dims / 2);
    const float* kv = p.in + s.q_rows();
    float ss = 0.f;
    for (uint32_t i = tid; i < D; i += kMT) {
      const float v = __ldcg(kv + i);
      raw[i] = v;
      if (i < rank) ss = fmaf(v, v, ss);
    }
    ss = warp_sum(ss);
    if (lane == 0) q[warp] = ss;
    __syncthreads();
    float tot = 0.f;
#pragma unroll
    for (int w = 0; w < kMT / 32; ++w) tot += q[w];
    const float rms = sqrtf(__fdiv_rn(tot, (float)rank) + p.eps);
    if (full) {
      if (tid == 0 && p.state) atomicOr(&p.state->err, 2u);
      return;
    }
    T* c = reinterpret_cast<T*>(p.c_cache) + (size_t)pos * rank;
    T* k = reinterpret_cast<T*>(p.kr_cache) + (size_t)pos * rot;
    for (uint32_t i = tid; i < rank; i += kMT) c[i] = __float2bfloat16_rn(__fmul_rn(__fdiv_rn(raw[i], rms), p.lat_gain[i]));
    for (uint32_t i = tid; i < rot; i += kMT) k[i] = __float2bfloat16_rn(rotated(raw + rank, i, s.rope_dims, cs));
    return;
  }
  const uint32_t h = blockIdx.x / slices, sl = blockIdx.x - h * slices, v0 = sl * kSlice, ns = min(kSlice, nv - v0);
  const T* W = reinterpret_cast<const T*>(p.Wkv) + (size_t)h * dim * rank + (size_t)v0 * 8;
  const uint32_t groups = kMT / ns, gi = tid / ns, vi = tid - gi * ns;
  constexpr int kPre = 8;
  uint4 w[kPre];
#pragma unroll
  for (int j = 0; j < kPre; ++j) {
    const uint32_t d = gi + j * groups;
    w[j] = gi < groups && d < dim ? ld_stream16(W + (size_t)d * rank + vi * 8) : make_uint4(0, 0, 0, 0);
  }
  pdl_launch_dependents();
  pdl_wait();
  const float* qrow = p.in + (size_t)h * hd;
  for (uint32_t i = tid; i < hd; i += kMT) q[i] = __ldcg(qrow + i);
  __syncthreads();
  // this head's row of the three operand tiles
  const uint32_t HG = heads_per_cta(s.heads), grp = h / HG, hh = h - grp * HG;
  T* const out = qs + ((size_t)grp * kTerms * kHeads + hh) * D;
  const size_t term = (size_t)kHeads * D;
  if (gi < groups) {
    float acc[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) acc[e] = 0.f;
    auto add = [&](const uint4& x, uint32_t d) {
      float f[8];
      WeightVec<T>::unpack(x, f);
      const float qd = q[d];
#pragma unroll
      for (int e = 0; e < 8; ++e) acc[e] = fmaf(qd, f[e], acc[e]);
    };
    uint32_t d = gi;
#pragma unroll
    for (int j = 0; j < kPre; ++j, d += groups)
      if (d < dim) add(w[j], d);
    for (; d < dim; d += groups) add(ld_stream16(W + (size_t)d * rank + vi * 8), d);
    float4* dst = reinterpret_cast<float4*>(part + (gi * ns + vi) * 8);
    dst[0] = make_float4(acc[0], acc[1], acc[2], acc[3]);
    dst[1] = make_float4(acc[4], acc[5], acc[6], acc[7]);
  }
  if (sl == 0) {
    const Window win = window_of(p);
    const float2* cs = p.rope_cs + (size_t)win.pos * (s.rope_dims / 2);
    for (uint32_t i = tid; i < rot; i += kMT) {
      T* at = out + rank + i;
      split3_one(rotated(q + dim, i, s.rope_dims, cs), at, at + term, at + 2 * term);
    }
  }
  __syncthreads();
  // pairs of values: eight lanes share a pair's sum over the groups (ns * 4 is a multiple of 4: warps stay together)
  for (uint32_t i = tid / 8; i < ns * 4; i += kMT / 8) {
    float a = 0.f, b = 0.f;
#pragma unroll 4
    for (uint32_t g = tid & 7; g < groups; g += 8) {
      const float2 t = *reinterpret_cast<const float2*>(part + g * ns * 8 + 2 * i);
      a += t.x;
      b += t.y;
    }
#pragma unroll
    for (int o = 4; o > 0; o >>= 1) {
      a += __shfl_xor_sync(0xffffffffu, a, o);
      b += __shfl_xor_sync(0xffffffffu, b, o);
    }
    if ((tid & 7) == 0) {
      uint32_t t0, t1, t2;
      split3_pair(a, b, t0, t1, t2);
      T* at = out + v0 * 8 + 2 * i;
      *reinterpret_cast<uint32_t*>(at) = t0;
      *reinterpret_cast<uint32_t*>(at + term) = t1;
      *reinterpret_cast<uint32_t*>(at + 2 * term) = t2;
    }
  }
}

// ---- a run of cached rows, up to 16 heads --------------------------------------------------------------------------------------
// Partial of head h over run r: part[(r * heads + h) * (rank + 4)] = sum of latents, then maximum and sum of weights.
__global__ void __launch_bounds__(kMT) latent_window_kernel(const LatentParams p, const T* __restrict__ qs, float* __restrict__ part,
                                                           const uint32_t run) {
  extern __shared__ __align__(16) unsigned char lw_raw[];
  const LatentSpec& s = p.spec;
  const uint32_t rank = s.rank, rot = s.rot, D = rank + rot, ld = D + 8;
  constexpr uint32_t PL = kStage + 8, ROWS = kTerms * kHeads;
  float* const sp = reinterpret_cast<float*>(lw_raw);       // [2][16][kStage] scores, in two halves of the inner dimension
  float* const ml = sp + 2 * kHeads * kStage;               // [16][3]: rescale factor, maximum, sum
  T* const ps = reinterpret_cast<T*>(ml + 3 * kHeads);      // [term][16][PL] weights
  T* const Q = ps + ROWS * PL;                              // [term][16][ld]
  T* const rows0 = Q + ROWS * ld;                           // [1 or 2][kStage][ld]
  const uint32_t tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const uint32_t HG = heads_per_cta(s.heads), h0 = blockIdx.y * HG, nh = min(HG, s.heads - h0);
  const Window win = window_of(p);
  const uint32_t k0 = win.lo + blockIdx.x * run, k1 = min(win.lo + win.n, k0 + run);
  const T* const cc = reinterpret_cast<const T*>(p.c_cache);
  const T* const kc = reinterpret_cast<const T*>(p.kr_cache);
  auto stage_row = [&](T* st, uint32_t r, uint32_t key) {
    for (uint32_t v = lane; v < D / 8; v += 32)
      cp16((uint32_t)__cvta_generic_to_shared(st + r * ld + v * 8), v * 8 < rank ? cc + (size_t)key * rank + v * 8 : kc + (size_t)key * rot + v * 8 - rank, 16);
  };
  // a row per warp; `skip`: a row that is not there yet
  auto stage = [&](uint32_t buf, uint32_t kb, uint32_t nk, uint32_t skip) {
    T* const st = rows0 + buf * kStage * ld;
    for (uint32_t r = warp; r < nk; r += kMT / 32)
      if (kb + r != skip) stage_row(st, r, kb + r);
    // rows that complete the last tile of 16: zeros (their weights are zero)
    const uint32_t end = (nk + 15u) & ~15u;
    for (uint32_t r = nk + warp; r < end; r += kMT / 32)
      for (uint32_t v = lane; v < D / 8; v += 32) *reinterpret_cast<uint4*>(st + r * ld + v * 8) = make_uint4(0, 0, 0, 0);
  };
  const bool empty = k0 >= win.lo + win.n;
  // rows of earlier positions were written by earlier steps: requested before the dependency wait
  uint32_t nk = empty ? 0u : min(kStage, k1 - k0);
  if (!empty) stage(0, k0, nk, win.pos);
  for (uint32_t i = tid; i < ROWS * PL / 8; i += kMT) reinterpret_cast<uint4*>(ps)[i] = make_uint4(0, 0, 0, 0);
  if (tid < kHeads) {
    ml[3 * tid + 1] = kNeg;
    ml[3 * tid + 2] = 0.f;
  }
  pdl_launch_dependents();
  pdl_wait();
  if (empty) return;
  if (win.pos - k0 < nk && warp == 0) stage_row(rows0, win.pos - k0, win.pos);
  {
    const T* src = qs + (size_t)blockIdx.y * ROWS * D;
    for (uint32_t r = warp; r < ROWS; r += kMT / 32)
      for (uint32_t v = lane; v < D / 8; v += 32) cp16((uint32_t)__cvta_generic_to_shared(Q + r * ld + v * 8), src + (size_t)r * D + v * 8, 16);
  }
  cp_commit();
  // latent columns of this warp: pairs of 8-column tiles c0 = (t * 8 + warp) * 16
  constexpr int NT = 4;  // rank <= 512
  float o[NT][2][4];
#pragma unroll
  for (int t = 0; t < NT; ++t)
#pragma unroll
    for (int u = 0; u < 2; ++u) o[t][u][0] = o[t][u][1] = o[t][u][2] = o[t][u][3] = 0.f;
  const uint32_t lm = lane >> 3, lr = lane & 7, qr = lane >> 2, qc = (lane & 3) * 2;
  const uint32_t q_a = (uint32_t)__cvta_generic_to_shared(Q) + (((lm & 1) * 8 + lr) * ld + (lm >> 1) * 8) * 2, q_term = kHeads * ld * 2;
  const uint32_t p_a = (uint32_t)__cvta_generic_to_shared(ps) + (((lm & 1) * 8 + lr) * PL + (lm >> 1) * 8) * 2;
  const uint32_t rows_s = (uint32_t)__cvta_generic_to_shared(rows0);
  // scores: warp w takes 8 cached rows (w mod 4) and one half of the inner dimension (w / 4)
  const uint32_t KS = D / 16, kmid = (KS / 2 + 1) & ~1u, ks0 = warp < 4 ? 0u : kmid, ks1 = warp < 4 ? min(kmid, KS) : KS;
  uint32_t buf = 0;
  bool first = true;
  for (uint32_t kb = k0; kb < k1; kb += kStage) {
    const uint32_t nk_next = kb + kStage < k1 ? min(kStage, k1 - kb - kStage) : 0u;
    if (nk_next) {
      stage(buf ^ 1u, kb + kStage, nk_next, 0xffffffffu);
      cp_commit();
      cp_wait<1>();
    } else {
      cp_wait<0>();
    }
    __syncthreads();
    const uint32_t st = rows_s + buf * kStage * ld * 2;
    {
      const uint32_t t0 = warp & 3;
      if (t0 * 8 < nk) {
        float a[kTerms][4];
#pragma unroll
        for (int m = 0; m < (int)kTerms; ++m) a[m][0] = a[m][1] = a[m][2] = a[m][3] = 0.f;
        const uint32_t ba = st + ((t0 * 8 + lr) * ld + lm * 8) * 2;
        uint32_t k = ks0;
#pragma unroll 2
        for (; k + 1 < ks1; k += 2) {
          uint32_t b[4];
          ldsm(ba + k * 32, b);
#pragma unroll
          for (int m = 0; m < (int)kTerms; ++m) {
            uint32_t x[4], y[4];
            ldsm(q_a + m * q_term + k * 32, x);
            ldsm(q_a + m * q_term + k * 32 + 32, y);
            mma(a[m], x, b[0], b[1]);
            mma(a[m], y, b[2], b[3]);
          }
        }
        if (k < ks1) {
          uint32_t r0, r1;
          ldsm2(ba + k * 32 - (lm >= 2 ? 32u : 0u), r0, r1);  // (the x2 form reads the addresses of lanes 0-15 only)
#pragma unroll
          for (int m = 0; m < (int)kTerms; ++m) {
            uint32_t x[4];
            ldsm(q_a + m * q_term + k * 32, x);
            mma(a[m], x, r0, r1);
          }
        }
        float* at = sp + ((warp >> 2) * kHeads + qr) * kStage + t0 * 8 + qc;
        *reinterpret_cast<float2*>(at) = make_float2(a[0][0] + a[1][0] + a[2][0], a[0][1] + a[1][1] + a[2][1]);
        *reinterpret_cast<float2*>(at + 8 * kStage) = make_float2(a[0][2] + a[1][2] + a[2][2], a[0][3] + a[1][3] + a[2][3]);
      }
    }
    __syncthreads();
    // softmax of a head in a warp: lane = cached row
    for (uint32_t hh = warp; hh < nh; hh += kMT / 32) {
      const float* v = sp + hh * kStage + lane;
      const float sc = lane < nk ? (v[0] + v[kHeads * kStage]) * s.scale : -INFINITY;
      const float m_old = ml[3 * hh + 1], l_old = ml[3 * hh + 2];
      const float mn = fmaxf(m_old, warp_max(sc)), e = expf(sc - mn), sum = warp_sum(e);
      T* at = ps + hh * PL + lane;
      split3_one(e, at, at + kHeads * PL, at + 2 * kHeads * PL);
      __syncwarp();
      if (lane == 0) {
        const float al = expf(m_old - mn);
        ml[3 * hh] = al;
        ml[3 * hh + 1] = mn;
        ml[3 * hh + 2] = l_old * al + sum;
      }
    }
    __syncthreads();
    if (!first) {
      const float al_a = qr < nh ? ml[3 * qr] : 0.f, al_b = qr + 8 < nh ? ml[3 * (qr + 8)] : 0.f;
#pragma unroll
      for (int t = 0; t < NT; ++t)
#pragma unroll
        for (int u = 0; u < 2; ++u) {
          o[t][u][0] *= al_a;
          o[t][u][1] *= al_a;
          o[t][u][2] *= al_b;
          o[t][u][3] *= al_b;
        }
    }
    first = false;
    const uint32_t v_a = st + (((lm & 1) * 8 + lr) * ld + (lm >> 1) * 8) * 2;
    for (uint32_t r = 0; r < nk; r += 16) {
      uint32_t x[kTerms][4];
#pragma unroll
      for (int m = 0; m < (int)kTerms; ++m) ldsm(p_a + (m * kHeads * PL + r) * 2, x[m]);
#pragma unroll
      for (int t = 0; t < NT; ++t) {
        const uint32_t c0 = (t * (kMT / 32) + warp) * 16;
        if (c0 < rank) {
          uint32_t b[4];
          ldsm_t(v_a + (r * ld + c0) * 2, b);
#pragma unroll
          for (int m = 0; m < (int)kTerms; ++m) {
            mma(o[t][0], x[m], b[0], b[1]);
            mma(o[t][1], x[m], b[2], b[3]);
          }
        }
      }
    }
    __syncthreads();  // everybody is done with this stage, the scores and the weights
    buf ^= 1u;
    nk = nk_next;
  }
  float* const mine = part + ((size_t)blockIdx.x * s.heads + h0) * (rank + 4);
#pragma unroll
  for (int t = 0; t < NT; ++t)
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const uint32_t c = (t * (kMT / 32) + warp) * 16 + u * 8 + qc;
      if (c < rank) {
        if (qr < nh) *reinterpret_cast<float2*>(mine + (size_t)qr * (rank + 4) + c) = make_float2(o[t][u][0], o[t][u][1]);
        if (qr + 8 < nh) *reinterpret_cast<float2*>(mine + (size_t)(qr + 8) * (rank + 4) + c) = make_float2(o[t][u][2], o[t][u][3]);
      }
    }
  if (tid < nh) {
    float* at = mine + (size_t)tid * (rank + 4) + rank;
    at[0] = ml[3 * tid + 1];
    at[1] = ml[3 * tid + 2];
  }
}

// ---- merge the runs of a head, map to values, gate ----------------------------------------------------------------------------------
// grid (C, heads), cluster of C <= 8 CTAs per head
__global__ void __launch_bounds__(kMT) latent_value_kernel(const LatentParams p, const float* __restrict__ part, const uint32_t run,
                                                          const uint32_t runs_max, const uint32_t C) {
  extern __shared__ __align__(16) float lv_sm[];
  const LatentSpec& s = p.spec;
  const uint32_t rank = s.rank, nv = rank / 8, vdim = s.vdim, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const uint32_t h = blockIdx.y, cr = C > 1 ? cluster_rank() : 0u;
  float* const om = lv_sm;            // [rank] in planes of float4
  float* const half = om + rank;      // [kMT * 4] partial sums
  float* const wt = half + kMT * 4;   // [runs]
  if (C > 1) cluster_arrive();        // "this CTA runs": waited for before the first store into a peer
  const uint32_t o0 = cr * vdim / C, no = (cr + 1) * vdim / C - o0;
  const uint32_t quads = rank / 4, q0 = cr * quads / C, nq = (cr + 1) * quads / C - q0;
  const T* const W = reinterpret_cast<const T*>(p.Wkv) + ((size_t)s.heads * s.dim + (size_t)h * vdim + o0) * rank;
  // first rows of the map of this warp wait in registers: rows warp, warp + 8, ...; two vectors per lane and row
  constexpr int kPre = 4;
  uint4 w[kPre][2];
#pragma unroll
  for (int j = 0; j < kPre; ++j)
#pragma unroll
    for (int u = 0; u < 2; ++u) {
      const uint32_t r = warp + j * (kMT / 32), v = lane + 32 * u;
      w[j][u] = r < no && v < nv ? ld_stream16(W + (size_t)r * rank + v * 8) : make_uint4(0, 0, 0, 0);
    }
  const Window win = window_of(p);
  const uint32_t runs = min(runs_max, (win.n + run - 1) / run);
  // quads of this CTA's latent dimensions; the threads of a quad share its runs
  const uint32_t g = nq ? kMT / nq : 1u, gi = nq ? tid / nq : 0u, qi = nq ? tid - gi * nq : 0u;
  const size_t row = rank + 4, step = (size_t)s.heads * row;
  const float* const mine = part + (size_t)h * row;
  pdl_launch_dependents();
  pdl_wait();
  // the sums and the runs' maxima are requested together
  constexpr int kAhead = 4;
  float4 ahead[kAhead];
#pragma unroll
  for (int j = 0; j < kAhead; ++j) {
    const uint32_t r = gi + j * g;
    ahead[j] = nq && gi < g && r < runs ? __ldcg(reinterpret_cast<const float4*>(mine + r * step) + q0 + qi) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  float M = kNeg;
  for (uint32_t r = lane; r < runs; r += 32) M = fmaxf(M, __ldcg(mine + r * step + rank));
  M = warp_max(M);
  float L = 0.f;
  for (uint32_t r = lane; r < runs; r += 32) {
    const float2 ml = __ldcg(reinterpret_cast<const float2*>(mine + r * step + rank));
    const float e = expf(ml.x - M);
    L = fmaf(e, ml.y, L);
    if (warp == 0) wt[r] = e;
  }
  const float inv = 1.0f / warp_sum(L);
  __syncthreads();
  if (nq && gi < g) {
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
    auto add = [&](const float4& v, float e) {
      a.x = fmaf(e, v.x, a.x);
      a.y = fmaf(e, v.y, a.y);
      a.z = fmaf(e, v.z, a.z);
      a.w = fmaf(e, v.w, a.w);
    };
#pragma unroll
    for (int j = 0; j < kAhead; ++j)
      if (gi + j * g < runs) add(ahead[j], wt[gi + j * g]);
#pragma unroll 8
    for (uint32_t r = gi + kAhead * g; r < runs; r += g) add(__ldcg(reinterpret_cast<const float4*>(mine + r * step) + q0 + qi), wt[r]);
    *reinterpret_cast<float4*>(half + (gi * nq + qi) * 4) = a;
  }
  __syncthreads();
  if (C > 1) cluster_wait();
  for (uint32_t j = tid; j < nq * 4; j += kMT) {  // one latent dimension per thread
    float t = 0.f;
#pragma unroll 8
    for (uint32_t k = 0; k < g; ++k) t += half[k * nq * 4 + j];
    t *= inv;
    float* dst = om + plane<8>(q0 * 4 + j, nv);
    if (C == 1) *dst = t;
    else
      for (uint32_t c = 0; c < C; ++c) st_peer(peer_addr(dst, c), t);
  }
  if (C > 1) {
    cluster_arrive();  // the last access to a peer
    cluster_wait();
  } else {
    __syncthreads();
  }
  const float* gate = p.in + s.q_rows() + s.kv_rows() + (size_t)h * vdim + o0;
  auto finish = [&](uint32_t r, float acc) {
    acc = warp_sum(acc);
    if (lane == 0) p.out[(size_t)h * vdim + o0 + r] = acc * sigmoid_f(__ldcg(gate + r));
  };
  auto dot = [&](const uint4& x, uint32_t v, float acc) {
    float f[8], y[8];
    WeightVec<T>::unpack(x, f);
    load_plane<8>(om, v, nv, y);
#pragma unroll
    for (int e = 0; e < 8; ++e) acc = fmaf(f[e], y[e], acc);
    return acc;
  };
#pragma unroll
  for (int j = 0; j < kPre; ++j) {
    const uint32_t r = warp + j * (kMT / 32);
    if (r < no) {
      float acc = 0.f;
#pragma unroll
      for (int u = 0; u < 2; ++u)
        if (lane + 32 * u < nv) acc = dot(w[j][u], lane + 32 * u, acc);
      finish(r, acc);
    }
  }
  for (uint32_t r = warp + kPre * (kMT / 32); r < no; r += kMT / 32) {
    float acc = 0.f;
    for (uint32_t v = lane; v < nv; v += 32) acc = dot(ld_stream16(W + (size_t)r * rank + v * 8), v, acc);
    finish(r, acc);
  }
}

size_t window_smem(const LatentSpec& s, uint32_t stages) {
  const size_t ld = s.rank + s.rot + 8, rows = kTerms * kHeads;
  return (2 * kHeads * kStage + 3 * kHeads) * 4 + rows * (kStage + 8) * 2 + (rows + stages * kStage) * ld * 2;
}

// Rows per run: one stage for windows up to a wave of CTAs, whole stages beyond.
uint32_t run_rows(const LatentSpec& s, uint32_t rows) {
  const uint32_t groups = head_groups(s.heads);
  const uint32_t ctas = sm_count() / groups ? sm_count() / groups : 1u;
  const uint32_t per = (rows + ctas - 1) / ctas;
  return (per + kStage - 1) / kStage * kStage;
}

}  // namespace

bool latent_decode_mma_supported(const LatentSpec& s) {
  // rows of whole MMA steps; the scratch arrays of the query kernel
  return s.rank % 16 == 0 && s.rot % 16 == 0 && s.rank <= 512 && s.rank + s.rot <= 8 * kMT && s.dim + s.rot <= 1024 &&
         window_smem(s, 2) <= 227 * 1024 && s.heads <= 65535;
}

// Bytes of the operand tiles (zero-filled once: unused rows stay zero) and of the partials for a cache of ctx rows.
size_t latent_decode_mma_scratch(const LatentSpec& s, uint32_t ctx, size_t* tiles_bytes) {
  const uint32_t rows = s.window && s.window < ctx ? s.window : ctx;
  const size_t tiles = ((size_t)head_groups(s.heads) * kTerms * kHeads * (s.rank + s.rot) * 2 + 255) / 256 * 256;
  const uint32_t run = run_rows(s, rows), runs = (rows + run - 1) / run;
  if (tiles_bytes) *tiles_bytes = tiles;
  return tiles + (size_t)runs * s.heads * (s.rank + 4) * 4;
}

cudaError_t launch_latent_decode_mma(cudaStream_t s, const LatentParams& p, uint32_t rows, bool pdl, int* launches) {
  const LatentSpec& sp = p.spec;
  if (!p.scratch) return cudaErrorInvalidValue;
  size_t tiles = 0;
  latent_decode_mma_scratch(sp, p.ctx, &tiles);
  T* qs = reinterpret_cast<T*>(p.scratch);
  float* part = reinterpret_cast<float*>(reinterpret_cast<char*>(p.scratch) + tiles);
  const uint32_t slices = (sp.rank / 8 + kSlice - 1) / kSlice;
  const uint32_t run = run_rows(sp, rows), runs = (rows + run - 1) / run;
  cudaError_t e = launch_pdl(latent_query_kernel, dim3(sp.heads * slices + 1), dim3(kMT), 0, s, pdl, p, qs, slices);
  if (e != cudaSuccess) return e;
  const size_t smem = window_smem(sp, run > kStage ? 2 : 1);
  if ((e = cudaFuncSetAttribute(latent_window_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem)) != cudaSuccess) return e;
  if ((e = launch_pdl(latent_window_kernel, dim3(runs, head_groups(sp.heads)), dim3(kMT), smem, s, pdl, p, (const T*)qs, part, run)) != cudaSuccess)
    return e;
  // a cluster per head, about one CTA per SM in all
  uint32_t C = 8;
  while (C > 1 && C * sp.heads > sm_count()) C >>= 1;
  const size_t vsmem = ((size_t)sp.rank + kMT * 4 + runs) * 4;
  if (vsmem > 48 * 1024) {
    if ((e = cudaFuncSetAttribute(latent_value_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)vsmem)) != cudaSuccess) return e;
  }
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(C, sp.heads);
  cfg.blockDim = dim3(kMT);
  cfg.dynamicSmemBytes = vsmem;
  cfg.stream = s;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = pdl ? 1 : 0;
  attr[1].id = cudaLaunchAttributeClusterDimension;
  attr[1].val.clusterDim.x = C;
  attr[1].val.clusterDim.y = 1;
  attr[1].val.clusterDim.z = 1;
  cfg.attrs = attr;
  cfg.numAttrs = 2;
  if (launches) *launches += 3;
  return cudaLaunchKernelEx(&cfg, latent_value_kernel, p, (const float*)part, run, runs, C);
}

}  // namespace nfai
