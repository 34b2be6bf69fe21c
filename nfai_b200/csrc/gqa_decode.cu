// Grouped-query attention of one new token over cached, normed keys and values (the layout and the split-KV scheme of
// attn.cu, for any head sizes up to 512, equal or not), with everything this attention does around it in the same launch:
//   * query heads and, in a layer with keys of its own, the new key and value heads are divided by their root mean square
//     where the projection left them; the new rows go into the cache and into this token's own attention as cached;
//   * the distance bias is taken off the scores, and keys it puts out of reach (gqa_common.cuh) are not read;
//   * a head's output is multiplied by the sigmoid of its gate.
// A CTA of 16 warps owns up to GH query heads of one KV head and one range of positions; LPP lanes own one position (eight
// elements each, NV times), so no shared memory and no barrier in the loop. Rows of earlier positions are requested before the
// dependency wait. Splits are merged by the CTA that draws the last ticket of its heads; no CTA waits for another.
#include <algorithm>

#include "gqa_common.cuh"

namespace nfai {

namespace {

using namespace gqa_detail;
using attn_detail::kNegBig;

constexpr int kGT = 512, kGW = kGT / 32;
constexpr uint32_t kMinChunk = 512, kSplitCap = 256;

struct DecodeShape {
  uint32_t S_max, hgroups;
  float* part;       // [heads][S_max][vdim + 2]
  uint32_t* tickets; // [kv_heads * hgroups]
};

template <typename CT, int LPP, int NV, int GH, int UNR, bool VECT>
__global__ void __launch_bounds__(kGT, 1) gqa_decode_kernel(const GqaParams p, const DecodeShape d) {
  using C8 = Cache8<CT, VECT>;
  using Raw = typename C8::Raw;
  constexpr int PPW = 32 / LPP;
  extern __shared__ __align__(16) float gsm[];  // [kGW][GH][vdim + 2]
  __shared__ float fin_w[kGW][GH], fin_ML[GH][2], mw[GH][kSplitCap], gates[GH];
  __shared__ uint32_t is_last;
  const GqaSpec& s = p.spec;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, grp = lane / LPP, sub = lane % LPP;
  const uint32_t dim = s.dim, vdim = s.vdim, G = s.heads / s.kv_heads;
  const uint32_t g = blockIdx.x / d.hgroups, hg = blockIdx.x % d.hgroups, h0 = g * G + hg * GH;
  const uint32_t nh = min((uint32_t)GH, G - hg * GH);
  const size_t k_ld = s.k_cols(), v_ld = s.v_cols();
  const CT* const kc = reinterpret_cast<const CT*>(p.k_cache) + (size_t)g * dim;
  const CT* const vc = reinterpret_cast<const CT*>(p.v_cache) + (size_t)g * vdim;
  pdl_launch_dependents();
  uint32_t pos = p.state ? p.state->pos : p.pos0;  // (advanced by the previous step, which has completed)
  const bool full = pos >= p.ctx;
  if (full) pos = p.ctx - 1;
  // the head with the smallest slope of the CTA reaches farthest
  const uint32_t far = reach(s, slope2(s, h0 + nh - 1));
  const uint32_t lo = pos > far ? pos - far : 0u, n = pos - lo + 1;
  uint32_t chunk = max((n + d.S_max - 1) / d.S_max, kMinChunk);
  chunk = (chunk + 63) / 64 * 64;
  const uint32_t S_eff = (n + chunk - 1) / chunk, sp = blockIdx.y;
  if (sp >= S_eff) return;  // the whole CTA
  const uint32_t t0 = lo + sp * chunk, t1 = min(pos + 1, t0 + chunk);

  int kn[NV], vn[NV];  // how many of this lane's elements exist
#pragma unroll
  for (int v = 0; v < NV; ++v) {
    const int e0 = (v * LPP + sub) * 8;
    kn[v] = (int)dim - e0;
    vn[v] = (int)vdim - e0;
  }
  auto load_rows = [&](uint32_t t, bool live, Raw (&kr)[NV], Raw (&vr)[NV]) {
#pragma unroll
    for (int v = 0; v < NV; ++v) {
      const int e0 = (v * LPP + sub) * 8;
      kr[v] = C8::ld(kc + (live ? (size_t)t * k_ld + e0 : 0), live ? kn[v] : 0);
      vr[v] = C8::ld(vc + (live ? (size_t)t * v_ld + e0 : 0), live ? vn[v] : 0);
    }
  };
  uint32_t base = t0 + warp * PPW;
  Raw kr[UNR][NV], vr[UNR][NV];
#pragma unroll
  for (int u = 0; u < UNR; ++u) {
    const uint32_t t = base + u * (kGW * PPW) + grp;
    load_rows(t, t < t1 && t != pos, kr[u], vr[u]);
  }
  pdl_wait();
  if (full && p.state && tid == 0) atomicOr(&p.state->err, 2u);

  // Eight elements (NV times) of a vector of `len` floats held by the lanes of a position, and the vector's division by its
  // root mean square. Every lane of the warp takes part. All loads of the set-up are issued before the first sum.
  auto fetch = [&](const float* src, uint32_t len, float (&f)[NV][8]) {
#pragma unroll
    for (int v = 0; v < NV; ++v) {
      const int e0 = (v * LPP + sub) * 8;
      if constexpr (VECT) {
        const bool in = e0 < (int)len;
        const float4 z = make_float4(0.f, 0.f, 0.f, 0.f);
        const float4 a = in ? __ldcg(reinterpret_cast<const float4*>(src + e0)) : z, b = in ? __ldcg(reinterpret_cast<const float4*>(src + e0) + 1) : z;
        f[v][0] = a.x; f[v][1] = a.y; f[v][2] = a.z; f[v][3] = a.w;
        f[v][4] = b.x; f[v][5] = b.y; f[v][6] = b.z; f[v][7] = b.w;
      } else {
#pragma unroll
        for (int e = 0; e < 8; ++e) f[v][e] = e0 + e < (int)len ? __ldcg(src + e0 + e) : 0.f;
      }
    }
  };
  auto unit = [&](uint32_t len, float factor, float (&f)[NV][8]) {  // f / rms(f) * factor
    float ss = 0.f;
#pragma unroll
    for (int v = 0; v < NV; ++v)
#pragma unroll
      for (int e = 0; e < 8; ++e) ss = fmaf(f[v][e], f[v][e], ss);
#pragma unroll
    for (int o = 1; o < LPP; o <<= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    const float c = __fdiv_rn(factor, sqrtf(__fdiv_rn(ss, (float)len) + p.eps));
#pragma unroll
    for (int v = 0; v < NV; ++v)
#pragma unroll
      for (int e = 0; e < 8; ++e) f[v][e] *= c;
  };
  const bool newest = t1 == pos + 1;  // this CTA's range ends with the new position
  float q[GH][NV][8], sl[GH], m[GH], l[GH], acc[GH][NV][8], fk[NV][8], fv[NV][8];
  Raw new_k[NV], new_v[NV];
#pragma unroll
  for (int j = 0; j < GH; ++j) fetch(p.in + (size_t)(h0 + min((uint32_t)j, nh - 1)) * dim, dim, q[j]);  // (heads past the group repeat the last)
  float gate_z = 0.f;
  if (s.head_gate && (uint32_t)tid < nh) gate_z = __ldcg(p.in + s.gate_row0() + h0 + tid);
  if (newest) {
    if (s.own_kv()) {
      fetch(p.in + s.q_rows() + (size_t)g * dim, dim, fk);
      fetch(p.in + s.q_rows() + s.k_cols() + (size_t)g * vdim, vdim, fv);
      if (s.qk_norm) unit(dim, 1.0f, fk);
      if (s.v_norm) unit(vdim, 1.0f, fv);
#pragma unroll
      for (int v = 0; v < NV; ++v) {
        new_k[v] = C8::pack(fk[v]);
        new_v[v] = C8::pack(fv[v]);
      }
      if (hg == 0 && warp == 0 && grp == 0) {  // one CTA per KV head keeps the new rows
        CT* ko = reinterpret_cast<CT*>(p.k_cache) + (size_t)pos * k_ld + (size_t)g * dim;
        CT* vo = reinterpret_cast<CT*>(p.v_cache) + (size_t)pos * v_ld + (size_t)g * vdim;
#pragma unroll
        for (int v = 0; v < NV; ++v) {
          const int e0 = (v * LPP + sub) * 8;
          C8::st(ko + e0, new_k[v], kn[v]);
          C8::st(vo + e0, new_v[v], vn[v]);
        }
      }
    } else {
      load_rows(pos, true, new_k, new_v);  // the source layer of this step has written them
    }
  }
  if (tid < GH) gates[tid] = s.head_gate ? head_sigmoid(gate_z) : 1.0f;  // (read behind the barriers of the merge)
#pragma unroll
  for (int j = 0; j < GH; ++j) {
    if (s.qk_norm) {
      unit(dim, s.scale * kLog2e, q[j]);
    } else {
#pragma unroll
      for (int v = 0; v < NV; ++v)
#pragma unroll
        for (int e = 0; e < 8; ++e) q[j][v][e] *= s.scale * kLog2e;
    }
    sl[j] = slope2(s, h0 + min((uint32_t)j, nh - 1));
    m[j] = kNegBig;
    l[j] = 0.f;
#pragma unroll
    for (int v = 0; v < NV; ++v)
#pragma unroll
      for (int e = 0; e < 8; ++e) acc[j][v][e] = 0.f;
  }

  while (base < t1) {
#pragma unroll
    for (int u = 0; u < UNR; ++u)
      if (newest && base + u * (kGW * PPW) + grp == pos) {
#pragma unroll
        for (int v = 0; v < NV; ++v) {
          kr[u][v] = new_k[v];
          vr[u][v] = new_v[v];
        }
      }
#pragma unroll
    for (int j = 0; j < GH; ++j) {
      float sc[UNR], mx = m[j];
#pragma unroll
      for (int u = 0; u < UNR; ++u) {
        float dot = 0.f;
#pragma unroll
        for (int v = 0; v < NV; ++v) {
          float kf[8];
          C8::unpack(kr[u][v], kf);
#pragma unroll
          for (int e = 0; e < 8; ++e) dot = fmaf(q[j][v][e], kf[e], dot);
        }
#pragma unroll
        for (int o = 1; o < LPP; o <<= 1) dot += __shfl_xor_sync(0xffffffffu, dot, o);
        const uint32_t t = base + u * (kGW * PPW) + grp;
        sc[u] = t < t1 ? fmaf(-sl[j], (float)(pos - t), dot) : -INFINITY;
        mx = fmaxf(mx, sc[u]);
      }
      const float alpha = gqa_ex2(m[j] - mx);
      m[j] = mx;
      l[j] *= alpha;
#pragma unroll
      for (int v = 0; v < NV; ++v)
#pragma unroll
        for (int e = 0; e < 8; ++e) acc[j][v][e] *= alpha;
#pragma unroll
      for (int u = 0; u < UNR; ++u) {
        const float w = gqa_ex2(sc[u] - mx);
        l[j] += w;
#pragma unroll
        for (int v = 0; v < NV; ++v) {
          float vf[8];
          C8::unpack(vr[u][v], vf);
#pragma unroll
          for (int e = 0; e < 8; ++e) acc[j][v][e] = fmaf(w, vf[e], acc[j][v][e]);
        }
      }
    }
    base += kGW * PPW * UNR;
    if (base >= t1) break;
#pragma unroll
    for (int u = 0; u < UNR; ++u) {
      const uint32_t t = base + u * (kGW * PPW) + grp;
      load_rows(t, t < t1 && t != pos, kr[u], vr[u]);
    }
  }

  // ---- lanes of a warp -> warps -> (if the range was split) CTAs
#pragma unroll
  for (int o = LPP; o < 32; o <<= 1) {
#pragma unroll
    for (int j = 0; j < GH; ++j) {
      const float m_o = __shfl_xor_sync(0xffffffffu, m[j], o), l_o = __shfl_xor_sync(0xffffffffu, l[j], o);
      const float m_new = fmaxf(m[j], m_o), a = gqa_ex2(m[j] - m_new), b = gqa_ex2(m_o - m_new);
      l[j] = l[j] * a + l_o * b;
#pragma unroll
      for (int v = 0; v < NV; ++v)
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          const float acc_o = __shfl_xor_sync(0xffffffffu, acc[j][v][e], o);
          acc[j][v][e] = acc[j][v][e] * a + acc_o * b;
        }
      m[j] = m_new;
    }
  }
  const uint32_t str = vdim + 2;
  if (grp == 0) {
#pragma unroll
    for (int j = 0; j < GH; ++j) {
      float* w = gsm + (size_t)(warp * GH + j) * str;
#pragma unroll
      for (int v = 0; v < NV; ++v)
#pragma unroll
        for (int e = 0; e < 8; ++e)
          if (e < vn[v]) w[(v * LPP + sub) * 8 + e] = acc[j][v][e];
      if (sub == 0) {
        w[vdim] = m[j];
        w[vdim + 1] = l[j];
      }
    }
  }
  __syncthreads();
  if (warp < GH) {  // a warp per head, lanes along the warps' partials
    const float* w = gsm + (size_t)((lane % kGW) * GH + warp) * str + vdim;
    const float mw_l = lane < kGW ? w[0] : kNegBig, lw = lane < kGW ? w[1] : 0.f;
    const float M = warp_max(mw_l), f = gqa_ex2(mw_l - M), L = warp_sum(lw * f);
    if (lane < kGW) fin_w[lane][warp] = f;
    if (lane == 0) {
      fin_ML[warp][0] = M;
      fin_ML[warp][1] = L;
    }
  }
  __syncthreads();
  for (uint32_t i = tid; i < nh * vdim; i += kGT) {
    const uint32_t j = i / vdim, e = i - j * vdim;
    float o = 0.f;
#pragma unroll
    for (int w = 0; w < kGW; ++w) o = fmaf(gsm[(size_t)(w * GH + j) * str + e], fin_w[w][j], o);
    if (S_eff == 1) p.out[(size_t)(h0 + j) * vdim + e] = o * __fdiv_rn(1.0f, fin_ML[j][1]) * gates[j];
    else d.part[((size_t)(h0 + j) * d.S_max + sp) * str + e] = o;
  }
  if (S_eff == 1) return;
  if ((uint32_t)tid < nh) {
    float* w = d.part + ((size_t)(h0 + tid) * d.S_max + sp) * str + vdim;
    w[0] = fin_ML[tid][0];
    w[1] = fin_ML[tid][1];
  }
  __syncthreads();
  if (tid == 0) {
    __threadfence();  // the block's stores, ordered before by the barrier, are out before the ticket ...
    is_last = atomicAdd(&d.tickets[blockIdx.x], 1u) == S_eff - 1 ? 1u : 0u;
    __threadfence();  // ... and the other blocks' are seen after it
  }
  __syncthreads();
  if (!is_last) return;
  constexpr uint32_t kAhead = 8;  // partials a thread asks for before it uses one
  float first[kAhead];            // those of its first output element, on their way while the weights are made
  auto partial = [&](uint32_t i, uint32_t k) { return __ldcg(d.part + ((size_t)(h0 + i / vdim) * d.S_max + k) * str + i % vdim); };
#pragma unroll
  for (uint32_t k = 0; k < kAhead; ++k) first[k] = (uint32_t)tid < nh * vdim && k < S_eff ? partial(tid, k) : 0.f;
  for (uint32_t j = warp; j < nh; j += kGW) {
    const float* b = d.part + (size_t)(h0 + j) * d.S_max * str + vdim;
    constexpr int kPer = kSplitCap / 32;
    float mk[kPer], lk[kPer], M = kNegBig, L = 0.f;
#pragma unroll
    for (int u = 0; u < kPer; ++u) {
      const uint32_t k = lane + 32 * u;
      mk[u] = k < S_eff ? __ldcg(b + (size_t)k * str) : kNegBig;
      lk[u] = k < S_eff ? __ldcg(b + (size_t)k * str + 1) : 0.f;
    }
#pragma unroll
    for (int u = 0; u < kPer; ++u) M = fmaxf(M, mk[u]);
    M = warp_max(M);
#pragma unroll
    for (int u = 0; u < kPer; ++u) {
      const float w = gqa_ex2(mk[u] - M);
      if (lane + 32 * u < S_eff) mw[j][lane + 32 * u] = w;
      L = fmaf(lk[u], w, L);
    }
    L = warp_sum(L);
    if (lane == 0) fin_ML[j][1] = L;
  }
  __syncthreads();
  for (uint32_t i = tid; i < nh * vdim; i += kGT) {
    const uint32_t j = i / vdim, e = i - j * vdim;
    float o = 0.f;
    uint32_t k = 0;
    if (i == (uint32_t)tid) {
#pragma unroll
      for (; k < kAhead; ++k) o = fmaf(first[k], k < S_eff ? mw[j][k] : 0.f, o);
    }
#pragma unroll 8
    for (; k < S_eff; ++k) o = fmaf(partial(i, k), mw[j][k], o);
    p.out[(size_t)(h0 + j) * vdim + e] = o * __fdiv_rn(1.0f, fin_ML[j][1]) * gates[j];
  }
  if (tid == 0) d.tickets[blockIdx.x] = 0;
}

// Query heads per CTA: one while all of a short cache is in flight at once, up to four of a group to share a long one.
uint32_t heads_per_cta(const GqaSpec& s, uint32_t ctx) {
  const uint32_t G = s.heads / s.kv_heads;
  if (ctx <= 4096 || G == 1 || s.dim > 128 || s.vdim > 128) return 1;
  return G <= 2 ? 2 : 4;
}
// As many splits of kMinChunk positions as a full cache needs, unless the CTAs with work would not fit the GPU at once; heads
// whose bias keeps them near use fewer of them.
DecodeShape decode_shape(const GqaSpec& s, uint32_t ctx, float* part) {
  DecodeShape d;
  const uint32_t GH = heads_per_cta(s, ctx), G = s.heads / s.kv_heads;
  d.hgroups = (G + GH - 1) / GH;
  uint32_t S = std::min((ctx + kMinChunk - 1) / kMinChunk, kSplitCap);
  for (; S > 1; --S) {
    const uint32_t chunk = std::max((ctx + S - 1) / S, kMinChunk);
    uint64_t busy = 0;
    for (uint32_t g = 0; g < s.kv_heads; ++g)
      for (uint32_t i = 0; i < d.hgroups; ++i)
        busy += (std::min<uint64_t>(ctx, (uint64_t)reach(s, slope2(s, g * G + std::min((i + 1) * GH, G) - 1)) + 1) + chunk - 1) / chunk;
    if (busy <= sm_count()) break;
  }
  d.S_max = S < 1 ? 1 : S;
  d.part = part;
  d.tickets = reinterpret_cast<uint32_t*>(part + (size_t)s.heads * d.S_max * (s.vdim + 2));
  return d;
}

template <typename CT, int LPP, int NV, int GH, int UNR, bool VECT>
cudaError_t launch_shape(cudaStream_t s, const GqaParams& p, const DecodeShape& d, bool pdl) {
  const size_t smem = (size_t)kGW * GH * (p.spec.vdim + 2) * 4;
  auto kern = gqa_decode_kernel<CT, LPP, NV, GH, UNR, VECT>;
  if (smem > 40 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return e;
  }
  return launch_pdl(kern, dim3(p.spec.kv_heads * d.hgroups, d.S_max), dim3(kGT), smem, s, pdl, p, d);
}

template <typename CT, bool VECT>
cudaError_t launch_ct(cudaStream_t s, const GqaParams& p, const DecodeShape& d, uint32_t GH, bool pdl) {
  constexpr int W = sizeof(CT) == 4 ? 2 : 1;  // float32 rows take twice the registers
  const uint32_t D = p.spec.dim > p.spec.vdim ? p.spec.dim : p.spec.vdim;
  if (D > 256) return launch_shape<CT, 32, 2, 1, 2 / W, VECT>(s, p, d, pdl);
  if (D > 128) return launch_shape<CT, 32, 1, 1, 4 / W, VECT>(s, p, d, pdl);
  if constexpr (VECT) {  // sharing a long cache between heads is worth its instances only for the sizes models use
    if (GH == 4) return D > 64 ? launch_shape<CT, 16, 1, 4, 2 / W, VECT>(s, p, d, pdl) : launch_shape<CT, 8, 1, 4, 2 / W, VECT>(s, p, d, pdl);
    if (GH == 2) return D > 64 ? launch_shape<CT, 16, 1, 2, 4 / W, VECT>(s, p, d, pdl) : launch_shape<CT, 8, 1, 2, 4 / W, VECT>(s, p, d, pdl);
  } else if (GH != 1) {
    return GH == 4 ? launch_shape<CT, 16, 1, 4, 2, VECT>(s, p, d, pdl) : launch_shape<CT, 16, 1, 2, 2, VECT>(s, p, d, pdl);
  }
  if (D > 64) return launch_shape<CT, 16, 1, 1, 8 / W, VECT>(s, p, d, pdl);
  if (D > 32) return launch_shape<CT, 8, 1, 1, 8 / W, VECT>(s, p, d, pdl);
  return launch_shape<CT, 4, 1, 1, 4 / W, VECT>(s, p, d, pdl);
}

}  // namespace

bool gqa_supported(const GqaSpec& s, std::string* why) {
  if (s.dim > kMaxHeadDim || s.vdim > kMaxHeadDim) return *why = "attention head sizes go up to 512", false;
  if (s.heads > 65535) return *why = "too many attention heads", false;
  return true;
}

size_t gqa_decode_scratch(const GqaSpec& s, uint32_t ctx) {
  const DecodeShape d = decode_shape(s, ctx, nullptr);
  return ((size_t)s.heads * d.S_max * (s.vdim + 2) + (size_t)s.kv_heads * d.hgroups) * 4;
}

uint64_t gqa_rows_read(const GqaSpec& s, uint32_t pos) {
  uint64_t n = 0;
  for (uint32_t g = 0; g < s.kv_heads; ++g)  // the last head of a group has the smallest slope
    n += (pos > reach(s, slope2(s, (g + 1) * (s.heads / s.kv_heads) - 1)) ? reach(s, slope2(s, (g + 1) * (s.heads / s.kv_heads) - 1)) : pos) + 1ull;
  return n;
}

cudaError_t launch_gqa_decode(cudaStream_t s, const GqaParams& p, bool pdl) {
  if (!p.in || !p.k_cache || !p.v_cache || !p.out || !p.part || !p.ctx) return cudaErrorInvalidValue;
  const DecodeShape d = decode_shape(p.spec, p.ctx, p.part);
  const uint32_t GH = heads_per_cta(p.spec, p.ctx);
  const bool vect = p.spec.dim % 8 == 0 && p.spec.vdim % 8 == 0;
  if (p.dtype == 0) return vect ? launch_ct<float, true>(s, p, d, GH, pdl) : launch_ct<float, false>(s, p, d, GH, pdl);
  if (p.dtype == 2) return vect ? launch_ct<__nv_bfloat16, true>(s, p, d, GH, pdl) : launch_ct<__nv_bfloat16, false>(s, p, d, GH, pdl);
  return cudaErrorInvalidValue;
}

}  // namespace nfai
