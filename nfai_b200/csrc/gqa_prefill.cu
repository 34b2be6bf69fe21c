// Grouped-query attention of a prompt portion with head norms, distance bias and head gates.
//
//   gqa_prep           divides what the projection left by its root mean square, head by head: queries (times scale * log2 e)
//                      become operands, keys and values cache rows. Lanes of a warp share a head in quads of elements.
//   gqa_prefill_mma    flash attention on the warp-level tensor cores (bfloat16 operands, float32 accumulators) straight over
//                      the cache: a CTA owns 64 tokens of one head and walks the key tiles from the causal edge back to the
//                      reach of the head's distance bias (gqa_common.cuh). Two groups of four warps take alternate tiles and
//                      are merged at the end: heads reach differently far, and the time of the launch is that of the longest
//                      walk. Newest first: with a bias the running
//                      maximum is then found early and the sums hardly ever have to be rescaled. A constant per query changes
//                      nothing in its softmax, so the bias of a key is taken relative to the warp's first token: the part
//                      inside a tile is what the score accumulators start from, the part of the tile itself goes into the
//                      subtraction of the maximum. Scores, exponentials and sums are float32, the weights enter the second
//                      product as a bfloat16 head and remainder (relative error ~2^-17).
//   gqa_prefill_simt   the same for true float32 and for head sizes the former does not take.
// A portion may start anywhere: earlier positions are read from the cache.
#include <algorithm>

#include "gqa_common.cuh"

namespace nfai {

namespace {

using namespace gqa_detail;
using attn_detail::kNegBig;

// ---- norms ----------------------------------------------------------------------------------------------------------------
constexpr int kPrepThreads = 256;

template <typename CT>
__device__ __forceinline__ void put4(CT* p, const float (&f)[4], uint32_t n, bool quad) {
  if (quad) {
    if constexpr (sizeof(CT) == 4) {
      *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
    } else {
      __nv_bfloat162 b[2] = {__floats2bfloat162_rn(f[0], f[1]), __floats2bfloat162_rn(f[2], f[3])};
      *reinterpret_cast<uint2*>(p) = *reinterpret_cast<uint2*>(b);
    }
    return;
  }
#pragma unroll
  for (int e = 0; e < 4; ++e)
    if ((uint32_t)e < n) store_as(p + e, f[e]);
}

// NQ quads per lane; LPH lanes per head
template <typename CT, int LPH, int NQ>
__global__ void __launch_bounds__(kPrepThreads) gqa_prep_kernel(const GqaParams p, const int quads) {
  const GqaSpec& s = p.spec;
  const uint32_t t = blockIdx.x, lane = threadIdx.x & 31, sub = lane % LPH;
  const uint32_t heads_at_once = kPrepThreads / LPH, H = s.heads, G = s.own_kv() ? s.kv_heads : 0;
  pdl_launch_dependents();
  pdl_wait();
  const float* in = p.in + (size_t)t * p.in_ld;
  const float qs = s.scale * kLog2e;
  const uint32_t total = H + 2 * G;
  for (uint32_t i0 = 0; i0 < total; i0 += heads_at_once) {  // (uniform: the shuffles below need every lane)
    const uint32_t i = i0 + threadIdx.x / LPH;
    const bool live = i < total;
    const uint32_t kind = !live || i < H ? 0u : i < H + G ? 1u : 2u, j = kind == 0 ? i : kind == 1 ? i - H : i - H - G;
    const uint32_t len = kind == 2 ? s.vdim : s.dim;
    const float* src = in + (kind == 0 ? 0 : kind == 1 ? s.q_rows() : s.q_rows() + s.k_cols()) + (live ? (size_t)j * len : 0);
    float f[NQ][4], ss = 0.f;
#pragma unroll
    for (int q = 0; q < NQ; ++q) {
      const uint32_t e0 = (q * LPH + sub) * 4;
      if (quads) {
        const float4 v = live && e0 < len ? __ldcg(reinterpret_cast<const float4*>(src + e0)) : make_float4(0.f, 0.f, 0.f, 0.f);
        f[q][0] = v.x; f[q][1] = v.y; f[q][2] = v.z; f[q][3] = v.w;
      } else {
#pragma unroll
        for (int e = 0; e < 4; ++e) f[q][e] = live && e0 + e < len ? __ldcg(src + e0 + e) : 0.f;
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) ss = fmaf(f[q][e], f[q][e], ss);
    }
#pragma unroll
    for (int o = 1; o < LPH; o <<= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    const bool normed = kind == 2 ? s.v_norm : s.qk_norm;
    const float rms = normed ? sqrtf(__fdiv_rn(ss, (float)len) + p.eps) : 1.0f;
    if (!live) continue;
    CT* dst = kind == 0 ? reinterpret_cast<CT*>(p.q) + (size_t)t * s.q_rows() + (size_t)j * len
              : kind == 1 ? reinterpret_cast<CT*>(p.k_cache) + (size_t)(p.pos0 + t) * s.k_cols() + (size_t)j * len
                          : reinterpret_cast<CT*>(p.v_cache) + (size_t)(p.pos0 + t) * s.v_cols() + (size_t)j * len;
#pragma unroll
    for (int q = 0; q < NQ; ++q) {
      const uint32_t e0 = (q * LPH + sub) * 4;
      if (e0 >= len) continue;
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        f[q][e] = __fdiv_rn(f[q][e], rms);
        if (kind == 0) f[q][e] *= qs;
      }
      put4(dst + e0, f[q], len - e0, quads != 0);
    }
  }
}

template <typename CT>
cudaError_t launch_prep(cudaStream_t s, const GqaParams& p, uint32_t T) {
  const uint32_t D = p.spec.dim > p.spec.vdim ? p.spec.dim : p.spec.vdim;
  const int quads = p.spec.dim % 4 == 0 && p.spec.vdim % 4 == 0 && p.in_ld % 4 == 0;
  const dim3 grid(T), block(kPrepThreads);
  if (D <= 32) return launch_pdl(gqa_prep_kernel<CT, 8, 1>, grid, block, 0, s, prefill_pdl(), p, quads);
  if (D <= 64) return launch_pdl(gqa_prep_kernel<CT, 16, 1>, grid, block, 0, s, prefill_pdl(), p, quads);
  if (D <= 128) return launch_pdl(gqa_prep_kernel<CT, 32, 1>, grid, block, 0, s, prefill_pdl(), p, quads);
  return launch_pdl(gqa_prep_kernel<CT, 32, 4>, grid, block, 0, s, prefill_pdl(), p, quads);
}

// ---- tensor cores -----------------------------------------------------------------------------------------------------------
__device__ __forceinline__ uint32_t pack_bf(float a, float b) {
  __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<uint32_t*>(&h);
}
__device__ __forceinline__ void mma_bf16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldsm4(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm4t(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr));
}
__device__ __forceinline__ void cpa16(uint32_t dst, const void* src, uint32_t bytes) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(bytes) : "memory");
}

constexpr int kPGroups = 2, kPW = 4;                              // groups of warps, warps of a group
constexpr int kPM = kPW * 16, kPThr = kPGroups * kPW * 32;        // tokens and threads of a CTA
constexpr int kPBuf = 2 * kPGroups;                               // tile buffers: a tile per group, and the next ones in flight

// DQ > 0: dim padded to it, query fragments stay in registers; DQ = 0: any dim, the query is read from shared memory per tile.
template <int DQ, int DV, int kN>
__global__ void __launch_bounds__(kPThr, DV <= 64 && DQ == 64 ? 2 : 1) gqa_prefill_mma_kernel(const GqaParams p, const uint32_t T, const uint32_t dq_rt,
                                                                                              const int vec) {
  extern __shared__ __align__(16) unsigned char pm_smem[];
  const GqaSpec& s = p.spec;
  const uint32_t dim = s.dim, vdim = s.vdim;
  const uint32_t DQr = DQ ? DQ : dq_rt, LQ = DQr + 8;
  constexpr uint32_t LV = DV + 8;
  __nv_bfloat16* const Qs = reinterpret_cast<__nv_bfloat16*>(pm_smem);  // [kPM][LQ]
  __nv_bfloat16* const Ks = Qs + kPM * LQ;                              // [kPBuf][kN][LQ]
  __nv_bfloat16* const Vs = Ks + kPBuf * kN * LQ;                       // [kPBuf][kN][LV]
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, qr = lane >> 2, qc = (lane & 3) * 2;
  pdl_launch_dependents();
  pdl_wait();
  // the last tiles of tokens of the heads that reach farthest start first
  const uint32_t h = s.heads - 1 - blockIdx.x % s.heads, tile = gridDim.x / s.heads - 1 - blockIdx.x / s.heads, g = h / (s.heads / s.kv_heads);
  const uint32_t t0 = tile * kPM, rows_end = min(T, t0 + kPM);
  const uint32_t first_pos = p.pos0 + t0, k_hi = p.pos0 + rows_end;  // one past the last visible position
  const float sl = slope2(s, h);
  const uint32_t far = reach(s, sl);
  const uint32_t k_lo = (first_pos > far ? first_pos - far : 0u) & ~7u;
  const __nv_bfloat16* const Q = reinterpret_cast<const __nv_bfloat16*>(p.q) + (size_t)h * dim;
  const __nv_bfloat16* const K = reinterpret_cast<const __nv_bfloat16*>(p.k_cache) + (size_t)g * dim;
  const __nv_bfloat16* const Vc = reinterpret_cast<const __nv_bfloat16*>(p.v_cache) + (size_t)g * vdim;
  const size_t q_ld = s.q_rows(), k_ld = s.k_cols(), v_ld = s.v_cols();
  const __nv_bfloat16 zero = __float2bfloat16_rn(0.f);

  // rows [r0, r0 + n) of a matrix into shared rows of `ld_s` elements; rows at or beyond `end` and columns at or beyond
  // `cols` (up to `width`) become zero
  auto stage = [&](__nv_bfloat16* dst, uint32_t ld_s, const __nv_bfloat16* src, size_t ld_g, uint32_t r0, uint32_t n, uint32_t end, uint32_t cols,
                   uint32_t width) {
    if (vec) {
      const uint32_t per = width / 8;
      for (uint32_t i = tid; i < n * per; i += kPThr) {
        const uint32_t r = i / per, c = (i - r * per) * 8;
        const bool in = r0 + r < end && c < cols;
        cpa16((uint32_t)__cvta_generic_to_shared(dst + r * ld_s + c), in ? src + (size_t)(r0 + r) * ld_g + c : src, in ? 16u : 0u);
      }
    } else {
      for (uint32_t i = tid; i < n * width; i += kPThr) {
        const uint32_t r = i / width, c = i - r * width;
        dst[r * ld_s + c] = r0 + r < end && c < cols ? src[(size_t)(r0 + r) * ld_g + c] : zero;
      }
    }
  };
  auto issue = [&](uint32_t buf, uint32_t kb) {
    stage(Ks + buf * kN * LQ, LQ, K, k_ld, kb, kN, k_hi, dim, DQr);
    stage(Vs + buf * kN * LV, LV, Vc, v_ld, kb, kN, k_hi, vdim, DV);
  };
  stage(Qs, LQ, Q, q_ld, t0, kPM, T, dim, DQr);
  const uint32_t ntiles = (k_hi - k_lo + kN - 1) / kN;
  auto tile_pos = [&](uint32_t it) { return k_lo + (ntiles - 1 - it) * kN; };  // newest first
  auto issue_round = [&](uint32_t round) {  // a tile for each group
#pragma unroll
    for (int i = 0; i < kPGroups; ++i)
      if (round * kPGroups + i < ntiles) issue((round & 1u) * kPGroups + i, tile_pos(round * kPGroups + i));
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  issue_round(0);  // with the query rows

  const int group = warp / kPW, wq = warp % kPW;  // this warp's group, and its place among the tokens
  const uint32_t row_a = t0 + wq * 16 + qr, row_b = row_a + 8;
  const uint32_t pos_a = p.pos0 + row_a, pos_b = p.pos0 + row_b;
  const uint32_t w_first = first_pos + wq * 16, w_last = w_first + 15;
  float o[DV / 8][4];
#pragma unroll
  for (int j = 0; j < DV / 8; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
  float m_a = kNegBig, m_b = kNegBig, l_a = 0.f, l_b = 0.f;
  const int lm = lane >> 3, lr = lane & 7;
  const uint32_t q_s = (uint32_t)__cvta_generic_to_shared(Qs) + (uint32_t)((wq * 16 + (lm & 1) * 8 + lr) * LQ + (lm >> 1) * 8) * 2;
  const uint32_t k_off = (uint32_t)(((lm >> 1) * 8 + lr) * LQ + (lm & 1) * 8) * 2;
  const uint32_t v_off = (uint32_t)(((lm & 1) * 8 + lr) * LV + (lm >> 1) * 8) * 2;
  const uint32_t ks_b = (uint32_t)__cvta_generic_to_shared(Ks), vs_b = (uint32_t)__cvta_generic_to_shared(Vs);
  uint32_t qf[DQ ? DQ / 16 : 1][4];
  const float b_lane = sl * (float)qc;

  for (uint32_t round = 0; round * kPGroups < ntiles; ++round) {
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();  // this round's tiles are there for every warp, and every warp has left the last round's
    if ((round + 1) * kPGroups < ntiles) issue_round(round + 1);
    const uint32_t it = round * kPGroups + group, buf = (round & 1u) * kPGroups + group, kb = tile_pos(it < ntiles ? it : 0);
    if constexpr (DQ > 0) {
      if (round == 0) {
#pragma unroll
        for (int kk = 0; kk < DQ / 16; ++kk) ldsm4(q_s + kk * 32, qf[kk]);
      }
    }
    if (it >= ntiles || kb > w_last) continue;  // (warp-uniform)
    const uint32_t ks = ks_b + buf * (uint32_t)(kN * LQ * 2), vs = vs_b + buf * (uint32_t)(kN * LV * 2);
    float c[kN / 8][4];
#pragma unroll
    for (int j = 0; j < kN / 8; ++j) {  // (without a bias sl is zero)
      c[j][0] = c[j][2] = fmaf(sl, (float)(j * 8), b_lane);
      c[j][1] = c[j][3] = fmaf(sl, (float)(j * 8 + 1), b_lane);
    }
    auto scores = [&](const uint32_t (&a)[4], uint32_t kk) {
#pragma unroll
      for (int j = 0; j < kN / 8; j += 2) {
        uint32_t b[4];
        ldsm4(ks + (uint32_t)(j * 8) * LQ * 2 + kk * 32 + k_off, b);
        mma_bf16(c[j], a, b[0], b[1]);
        mma_bf16(c[j + 1], a, b[2], b[3]);
      }
    };
    if constexpr (DQ > 0) {
#pragma unroll
      for (int kk = 0; kk < DQ / 16; ++kk) scores(qf[kk], kk);
    } else {
      for (uint32_t kk = 0; kk < DQr / 16; ++kk) {
        uint32_t a[4];
        ldsm4(q_s + kk * 32, a);
        scores(a, kk);
      }
    }
    if (kb + kN - 1 > w_first) {  // not every row of the warp sees the whole tile
#pragma unroll
      for (int j = 0; j < kN / 8; ++j) {
        const uint32_t k = kb + j * 8 + qc;
        if (k > pos_a) c[j][0] = -INFINITY;
        if (k + 1 > pos_a) c[j][1] = -INFINITY;
        if (k > pos_b) c[j][2] = -INFINITY;
        if (k + 1 > pos_b) c[j][3] = -INFINITY;
      }
    }
    float mx_a = c[0][0], mx_b = c[0][2];
#pragma unroll
    for (int j = 0; j < kN / 8; ++j) {
      mx_a = fmaxf(mx_a, fmaxf(c[j][0], c[j][1]));
      mx_b = fmaxf(mx_b, fmaxf(c[j][2], c[j][3]));
    }
    mx_a = fmaxf(mx_a, __shfl_xor_sync(0xffffffffu, mx_a, 1));
    mx_a = fmaxf(mx_a, __shfl_xor_sync(0xffffffffu, mx_a, 2));
    mx_b = fmaxf(mx_b, __shfl_xor_sync(0xffffffffu, mx_b, 1));
    mx_b = fmaxf(mx_b, __shfl_xor_sync(0xffffffffu, mx_b, 2));
    const float tile_bias = sl * (float)((int)kb - (int)w_first);
    const float new_a = fmaxf(m_a, mx_a + tile_bias), new_b = fmaxf(m_b, mx_b + tile_bias);
    if (__any_sync(0xffffffffu, new_a > m_a || new_b > m_b)) {
      const float al_a = gqa_ex2(m_a - new_a), al_b = gqa_ex2(m_b - new_b);
      m_a = new_a;
      m_b = new_b;
      l_a *= al_a;
      l_b *= al_b;
#pragma unroll
      for (int j = 0; j < DV / 8; ++j) {
        o[j][0] *= al_a;
        o[j][1] *= al_a;
        o[j][2] *= al_b;
        o[j][3] *= al_b;
      }
    }
    const float mn_a = m_a - tile_bias, mn_b = m_b - tile_bias;
    float sum_a = 0.f, sum_b = 0.f;
    uint32_t ph[kN / 16][4], pl[kN / 16][4];
#pragma unroll
    for (int j = 0; j < kN / 8; ++j) {
      const float e0 = gqa_ex2(c[j][0] - mn_a), e1 = gqa_ex2(c[j][1] - mn_a), e2 = gqa_ex2(c[j][2] - mn_b), e3 = gqa_ex2(c[j][3] - mn_b);
      sum_a += e0 + e1;
      sum_b += e2 + e3;
      const uint32_t ha = pack_bf(e0, e1), hb = pack_bf(e2, e3);
      const int i = j >> 1, w = (j & 1) * 2;
      ph[i][w] = ha;
      ph[i][w + 1] = hb;
      pl[i][w] = pack_bf(e0 - __uint_as_float(ha << 16), e1 - __uint_as_float(ha & 0xffff0000u));
      pl[i][w + 1] = pack_bf(e2 - __uint_as_float(hb << 16), e3 - __uint_as_float(hb & 0xffff0000u));
    }
    l_a += sum_a;
    l_b += sum_b;
#pragma unroll
    for (int kk = 0; kk < kN / 16; ++kk) {
#pragma unroll
      for (int j = 0; j < DV / 8; j += 2) {
        uint32_t b[4];
        ldsm4t(vs + (uint32_t)(kk * 16 * LV + j * 8) * 2 + v_off, b);
        mma_bf16(o[j], ph[kk], b[0], b[1]);
        mma_bf16(o[j + 1], ph[kk], b[2], b[3]);
        mma_bf16(o[j], pl[kk], b[0], b[1]);
        mma_bf16(o[j + 1], pl[kk], b[2], b[3]);
      }
    }
  }
  // the second group's sums join the first's (the buffers are free: nothing is in flight any more)
  static_assert(kPGroups == 2, "one group hands over to the other");
  __syncthreads();
  float* const hand = reinterpret_cast<float*>(Ks);  // [DV/8 + 1][kPW * 32] quads
  const int slot = (wq * 32 + lane) * 4;
  if (group == 1) {
#pragma unroll
    for (int j = 0; j < DV / 8; ++j) *reinterpret_cast<float4*>(hand + j * (kPW * 128) + slot) = make_float4(o[j][0], o[j][1], o[j][2], o[j][3]);
    *reinterpret_cast<float4*>(hand + DV / 8 * (kPW * 128) + slot) = make_float4(m_a, m_b, l_a, l_b);
  }
  __syncthreads();
  if (group == 1) return;
  {
    const float4 r = *reinterpret_cast<const float4*>(hand + DV / 8 * (kPW * 128) + slot);
    const float M_a = fmaxf(m_a, r.x), M_b = fmaxf(m_b, r.y);
    const float x_a = gqa_ex2(m_a - M_a), x_b = gqa_ex2(m_b - M_b), y_a = gqa_ex2(r.x - M_a), y_b = gqa_ex2(r.y - M_b);
    l_a = l_a * x_a + r.z * y_a;
    l_b = l_b * x_b + r.w * y_b;
#pragma unroll
    for (int j = 0; j < DV / 8; ++j) {
      const float4 v = *reinterpret_cast<const float4*>(hand + j * (kPW * 128) + slot);
      o[j][0] = o[j][0] * x_a + v.x * y_a;
      o[j][1] = o[j][1] * x_a + v.y * y_a;
      o[j][2] = o[j][2] * x_b + v.z * y_b;
      o[j][3] = o[j][3] * x_b + v.w * y_b;
    }
  }
  l_a += __shfl_xor_sync(0xffffffffu, l_a, 1);
  l_a += __shfl_xor_sync(0xffffffffu, l_a, 2);
  l_b += __shfl_xor_sync(0xffffffffu, l_b, 1);
  l_b += __shfl_xor_sync(0xffffffffu, l_b, 2);
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    const uint32_t row = half ? row_b : row_a;
    if (row >= T) continue;
    const float f = __fdiv_rn(1.0f, half ? l_b : l_a) * (s.head_gate ? head_sigmoid(p.in[(size_t)row * p.in_ld + s.gate_row0() + h]) : 1.0f);
    __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(p.ao) + (size_t)row * s.out_cols() + (size_t)h * vdim;
#pragma unroll
    for (int j = 0; j < DV / 8; ++j) {
      const uint32_t c = j * 8 + qc;
      const float a = o[j][half * 2] * f, b = o[j][half * 2 + 1] * f;
      if (vec) {
        if (c < vdim) *reinterpret_cast<__nv_bfloat162*>(out + c) = __floats2bfloat162_rn(a, b);
      } else {
        if (c < vdim) store_as(out + c, a);
        if (c + 1 < vdim) store_as(out + c + 1, b);
      }
    }
  }
}

size_t prefill_smem(uint32_t DQ, uint32_t DV, uint32_t kN) {
  const size_t q = (size_t)kPM * (DQ + 8) * 2, tiles = (size_t)kPBuf * kN * (DQ + DV + 16) * 2, hand = (size_t)(DV / 8 + 1) * kPW * 128 * 4;
  return q + std::max(tiles, hand);
}
uint32_t value_width(uint32_t vdim) { return vdim <= 32 ? 32 : vdim <= 64 ? 64 : vdim <= 128 ? 128 : vdim <= 256 ? 256 : 0; }

template <int DQ, int DV, int kN>
cudaError_t launch_mma(cudaStream_t s, const GqaParams& p, uint32_t T) {
  const uint32_t dq = DQ ? DQ : (p.spec.dim + 15u) & ~15u;
  const size_t smem = prefill_smem(dq, DV, kN);
  auto kern = gqa_prefill_mma_kernel<DQ, DV, kN>;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) return e;
  const int vec = p.spec.dim % 8 == 0 && p.spec.vdim % 8 == 0;
  return launch_pdl(kern, dim3((T + kPM - 1) / kPM * p.spec.heads), dim3(kPThr), smem, s, prefill_pdl(), p, T, dq, vec);
}

bool mma_supported(const GqaSpec& s) {
  const uint32_t dv = value_width(s.vdim);
  return dv && prefill_smem((s.dim + 15u) & ~15u, dv, 32) <= 227 * 1024;
}

// ---- any sizes, any type ------------------------------------------------------------------------------------------------------
constexpr int kSW = 8;        // tokens (one warp each) per CTA
constexpr uint32_t kSB = 32;  // keys per block, one per lane

// A warp works on one token of head blockIdx.y; lanes are keys in the first product and elements of the value in the second.
template <typename CT, int NE>
__global__ void __launch_bounds__(kSW * 32) gqa_prefill_simt_kernel(const GqaParams p, const uint32_t T) {
  extern __shared__ __align__(16) float ssm_f[];
  const GqaSpec& s = p.spec;
  const uint32_t dim = s.dim, vdim = s.vdim, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, tid = threadIdx.x;
  const uint32_t LK = dim | 1u;               // odd row stride: lanes read a column without conflicts
  float* const qs = ssm_f;                    // [kSW][dim]
  float* const ks = qs + kSW * dim;           // [kSB][LK]
  float* const vs = ks + kSB * LK;            // [kSB][vdim]
  float* const ws = vs + kSB * vdim;          // [kSW][kSB]
  const uint32_t h = blockIdx.y, g = h / (s.heads / s.kv_heads);
  pdl_launch_dependents();
  pdl_wait();
  const uint32_t ta = (gridDim.x - 1 - blockIdx.x) * kSW, t = ta + warp;
  const bool live = t < T;
  const uint32_t pos = p.pos0 + (live ? t : T - 1), last = p.pos0 + min(T, ta + kSW) - 1;
  const float sl = slope2(s, h);
  const uint32_t far = reach(s, sl), first = p.pos0 + ta;
  const uint32_t lo = first > far ? first - far : 0u;
  const CT* const K = reinterpret_cast<const CT*>(p.k_cache) + (size_t)g * dim;
  const CT* const Vc = reinterpret_cast<const CT*>(p.v_cache) + (size_t)g * vdim;
  const size_t k_ld = s.k_cols(), v_ld = s.v_cols();
  const CT* q = reinterpret_cast<const CT*>(p.q) + (size_t)(live ? t : T - 1) * s.q_rows() + (size_t)h * dim;
  for (uint32_t i = lane; i < dim; i += 32) qs[warp * dim + i] = to_float(q[i]);
  float o[NE];
#pragma unroll
  for (int e = 0; e < NE; ++e) o[e] = 0.f;
  float m = kNegBig, l = 0.f;
  for (uint32_t kb = lo; kb <= last; kb += kSB) {
    const uint32_t nk = min(kSB, last - kb + 1);
    __syncthreads();
    for (uint32_t i = tid; i < nk * dim; i += kSW * 32) {
      const uint32_t r = i / dim, c = i - r * dim;
      ks[r * LK + c] = to_float(K[(size_t)(kb + r) * k_ld + c]);
    }
    for (uint32_t i = tid; i < nk * vdim; i += kSW * 32) {
      const uint32_t r = i / vdim, c = i - r * vdim;
      vs[i] = to_float(Vc[(size_t)(kb + r) * v_ld + c]);
    }
    __syncthreads();
    const uint32_t key = kb + lane;
    float sc = -INFINITY;
    if (lane < nk && key <= pos) {
      float a = 0.f;
      for (uint32_t i = 0; i < dim; ++i) a = fmaf(qs[warp * dim + i], ks[lane * LK + i], a);
      sc = fmaf(-sl, (float)(pos - key), a);
    }
    const float mn = fmaxf(m, warp_max(sc)), alpha = gqa_ex2(m - mn), w = gqa_ex2(sc - mn);
    m = mn;
    l = l * alpha + warp_sum(w);
    ws[warp * kSB + lane] = w;
    __syncwarp();
#pragma unroll
    for (int e = 0; e < NE; ++e) {
      const uint32_t c = e * 32 + lane;
      if (c >= vdim) continue;
      float a = o[e] * alpha;
      for (uint32_t k = 0; k < nk; ++k) a = fmaf(ws[warp * kSB + k], vs[k * vdim + c], a);
      o[e] = a;
    }
    __syncwarp();
  }
  if (!live) return;
  const float f = __fdiv_rn(1.0f, l) * (s.head_gate ? head_sigmoid(p.in[(size_t)t * p.in_ld + s.gate_row0() + h]) : 1.0f);
  CT* out = reinterpret_cast<CT*>(p.ao) + (size_t)t * s.out_cols() + (size_t)h * vdim;
#pragma unroll
  for (int e = 0; e < NE; ++e) {
    const uint32_t c = e * 32 + lane;
    if (c < vdim) store_as(out + c, o[e] * f);
  }
}

template <typename CT, int NE>
cudaError_t launch_simt_ne(cudaStream_t s, const GqaParams& p, uint32_t T) {
  const GqaSpec& sp = p.spec;
  const size_t smem = ((size_t)kSW * sp.dim + kSB * (sp.dim | 1u) + (size_t)kSB * sp.vdim + kSW * kSB) * 4;
  auto kern = gqa_prefill_simt_kernel<CT, NE>;
  if (smem > 40 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return e;
  }
  return launch_pdl(kern, dim3((T + kSW - 1) / kSW, sp.heads), dim3(kSW * 32), smem, s, prefill_pdl(), p, T);
}
template <typename CT>
cudaError_t launch_simt(cudaStream_t s, const GqaParams& p, uint32_t T) {
  if (p.spec.vdim <= 64) return launch_simt_ne<CT, 2>(s, p, T);
  if (p.spec.vdim <= 128) return launch_simt_ne<CT, 4>(s, p, T);
  return launch_simt_ne<CT, 16>(s, p, T);
}

}  // namespace

cudaError_t launch_gqa_prep(cudaStream_t s, const GqaParams& p, uint32_t T) {
  if (!T || !p.in || !p.q || !p.k_cache || !p.v_cache || (uint64_t)p.pos0 + T > p.ctx) return cudaErrorInvalidValue;
  return p.dtype == 0 ? launch_prep<float>(s, p, T) : launch_prep<__nv_bfloat16>(s, p, T);
}

cudaError_t launch_gqa_prefill(cudaStream_t s, const GqaParams& p, uint32_t T) {
  if (!T || !p.in || !p.q || !p.ao || (uint64_t)p.pos0 + T > p.ctx) return cudaErrorInvalidValue;
  static const bool tensor_cores = env_int("NFAI_PREFILL_ATTN", 1) != 0;
  if (p.dtype == 2 && tensor_cores && mma_supported(p.spec)) {
    const uint32_t dim = p.spec.dim, dv = value_width(p.spec.vdim);
    if (dim > 32 && dim <= 64 && dv == 64) return launch_mma<64, 64, 64>(s, p, T);
    if (dim > 64 && dim <= 128 && dv == 128) return launch_mma<128, 128, 64>(s, p, T);
    switch (dv) {
      case 32: return launch_mma<0, 32, 32>(s, p, T);
      case 64: return launch_mma<0, 64, 32>(s, p, T);
      case 128: return launch_mma<0, 128, 32>(s, p, T);
      default: return launch_mma<0, 256, 32>(s, p, T);
    }
  }
  return p.dtype == 0 ? launch_simt<float>(s, p, T) : launch_simt<__nv_bfloat16>(s, p, T);
}

}  // namespace nfai
