// Latent attention: per position one RMS-normed latent c (rank values) and one rotated key part shared by all heads are
// cached; a head's keys and values are linear maps of c. Sliding window, per-element sigmoid gate on the output.
//
// Decode (latent_decode_kernel here for true float32 and any sizes; latent_decode_mma.cu for bfloat16 caches) never expands a key or a value. A head's query is pulled back through its key map
// (q_lat = W_uk^T q), scores are q_lat . c + q_rot . k_rot, the weighted sum is taken over the latents themselves and only
// the finished sum goes through the value map. One thread-block cluster works on one head; its CTAs
//   1. each make a slice of q_lat and write it into every CTA of the cluster (distributed shared memory),
//   2. each take a share of the window: cache rows staged by cp.async, online softmax, sum of latents,
//   3. merge the shares through distributed shared memory and each map a slice of the merged sum to values, times the gate.
// So projection of q, attention and value map are one launch. The new position's latent is normed and its key part rotated
// by every CTA for itself (the cache row written by one CTA is read by later launches only).
//
// Prompt path: latent_prep_kernel norms and rotates the portion's rows, a GEMM expands keys and values of every latent the
// portion's windows reach, and latent_prefill_mma_kernel (bfloat16, warp-level tensor cores) or latent_prefill_simt_kernel
// (float32, and head sizes the former does not take) run causal windowed attention over them.
#include <string>

#include "latent_common.cuh"

namespace nfai {

namespace {

using namespace latent_detail;

// ---- decode -------------------------------------------------------------------------------------------------------------
constexpr int kDT = 256;   // threads per CTA
constexpr int kKB = 32;    // cache rows per stage, one per lane in the softmax
constexpr int kSlots = 4;  // vectors of the latent sum per thread, at most

struct DecodeLayout {  // float offsets into dynamic shared memory; the staged rows follow at `stage` (bytes)
  uint32_t q, cur, om, opart, ml, part, sc, raw, stage, row_bytes, nbuf, total;
};
__host__ __device__ inline DecodeLayout decode_layout(const LatentSpec& s, uint32_t elem, uint32_t vec) {
  DecodeLayout l;
  const uint32_t D = s.rank + s.rot;
  uint32_t o = 0;
  auto take = [&](uint32_t n) { const uint32_t at = o; o += (n + 3u) & ~3u; return at; };
  l.q = take(D);            // [q_lat | q_rot]
  l.cur = take(D);          // the new position's [c | k_rot]
  l.raw = take((s.dim + s.rot > D ? s.dim + s.rot : D));
  l.om = take(s.rank);
  l.opart = take(s.rank);
  l.ml = take(4);
  l.part = take(kDT * vec);
  l.sc = take(kKB + 8);
  l.stage = o * 4;
  l.row_bytes = (D * elem + 15u) & ~15u;
  l.nbuf = 2;
  l.total = l.stage + 2 * kKB * l.row_bytes;
  if (l.total > 200u * 1024u) {
    l.nbuf = 1;
    l.total = l.stage + kKB * l.row_bytes;
  }
  return l;
}

template <typename CT, int VEC>
__global__ void __launch_bounds__(kDT) latent_decode_kernel(const LatentParams p, const uint32_t C) {
  extern __shared__ __align__(16) unsigned char ldsm_raw[];
  float* const sm = reinterpret_cast<float*>(ldsm_raw);
  const LatentSpec& s = p.spec;
  const DecodeLayout L = decode_layout(s, sizeof(CT), VEC);
  const uint32_t rank = s.rank, rot = s.rot, dim = s.dim, D = rank + rot, nv = rank / VEC;
  const uint32_t tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const uint32_t h = blockIdx.y, cr = C > 1 ? cluster_rank() : 0u;
  float* const q = sm + L.q;
  float* const cur = sm + L.cur;
  float* const raw = sm + L.raw;
  const CT* const Wuk = reinterpret_cast<const CT*>(p.Wkv) + (size_t)h * dim * rank;
  const CT* const Wuv = reinterpret_cast<const CT*>(p.Wkv) + ((size_t)s.heads * dim + (size_t)h * s.vdim) * rank;
  const CT* const cc = reinterpret_cast<const CT*>(p.c_cache);
  const CT* const kc = reinterpret_cast<const CT*>(p.kr_cache);
  uint32_t pos = p.state ? p.state->pos : p.pos0;
  const bool full = pos >= p.ctx;
  if (full) pos = p.ctx - 1;
  const uint32_t lo = s.window && pos + 1 > s.window ? pos + 1 - s.window : 0u;
  const uint32_t n = pos - lo + 1;
  const uint32_t k0 = lo + (uint32_t)((uint64_t)cr * n / C), k1 = lo + (uint32_t)((uint64_t)(cr + 1) * n / C);
  const uint32_t sv0 = (uint32_t)((uint64_t)cr * nv / C), sv1 = (uint32_t)((uint64_t)(cr + 1) * nv / C);
  const uint32_t o0 = (uint32_t)((uint64_t)cr * s.vdim / C), o1 = (uint32_t)((uint64_t)(cr + 1) * s.vdim / C);

  // copy cache rows [kb, kb + nk) into stage `buf`; the new position's row comes from shared memory
  unsigned char* const stage0 = ldsm_raw + L.stage;
  auto stage = [&](uint32_t buf, uint32_t kb, uint32_t nk) {
    unsigned char* const st = stage0 + buf * kKB * L.row_bytes;
    if constexpr (VEC > 1) {
      const uint32_t cv = nv, rv = rot / VEC, per = cv + rv;
      for (uint32_t i = tid; i < nk * per; i += kDT) {
        const uint32_t k = i / per, v = i - k * per, key = kb + k;
        CT* dst = reinterpret_cast<CT*>(st + k * L.row_bytes) + v * VEC;
        if (key == pos) {
#pragma unroll
          for (int e = 0; e < VEC; ++e) dst[e] = cast_to<CT>(cur[v * VEC + e]);
        } else {
          const CT* src = v < cv ? cc + (size_t)key * rank + v * VEC : kc + (size_t)key * rot + (v - cv) * VEC;
          cp16((uint32_t)__cvta_generic_to_shared(dst), src, 16);
        }
      }
    } else {
      for (uint32_t i = tid; i < nk * D; i += kDT) {
        const uint32_t k = i / D, v = i - k * D, key = kb + k;
        CT* dst = reinterpret_cast<CT*>(st + k * L.row_bytes) + v;
        *dst = key == pos ? cast_to<CT>(cur[v]) : v < rank ? cc[(size_t)key * rank + v] : kc[(size_t)key * rot + v - rank];
      }
    }
    cp_commit();
  };

  if (C > 1) cluster_arrive();  // "this CTA runs": waited for before the first access to a peer's shared memory
  // Weights and rows of earlier positions do not depend on the step's previous kernel: ask the L2 for this CTA's share.
  {
    const char* a = reinterpret_cast<const char*>(Wuk);
    const uint32_t slice = (sv1 - sv0) * VEC * (uint32_t)sizeof(CT), lines = (slice + 127) / 128;
    for (uint32_t i = tid; i < dim * lines; i += kDT) {
      const uint32_t d = i / lines, l = i - d * lines;
      asm volatile("prefetch.global.L2 [%0];" ::"l"(a + ((size_t)d * rank + (size_t)sv0 * VEC) * sizeof(CT) + (size_t)l * 128));
    }
    const char* b = reinterpret_cast<const char*>(Wuv + (size_t)o0 * rank);
    for (size_t i = (size_t)tid * 128; i < (size_t)(o1 - o0) * rank * sizeof(CT); i += kDT * 128)
      asm volatile("prefetch.global.L2 [%0];" ::"l"(b + i));
  }
  pdl_launch_dependents();
  pdl_wait();

  // ---- the new position's latent and key part, this head's query
  {
    const float* kvrow = p.in + s.q_rows();
    float ss = 0.f;
    for (uint32_t i = tid; i < D; i += kDT) {
      const float v = __ldcg(kvrow + i);
      raw[i] = v;
      if (i < rank) ss = fmaf(v, v, ss);
    }
    ss = warp_sum(ss);
    if (lane == 0) sm[L.part + warp] = ss;
    __syncthreads();
    float tot = 0.f;
#pragma unroll
    for (int w = 0; w < kDT / 32; ++w) tot += sm[L.part + w];
    const float rms = sqrtf(__fdiv_rn(tot, (float)rank) + p.eps);
    const float2* cs = p.rope_cs + (size_t)pos * (s.rope_dims / 2);
    for (uint32_t i = tid; i < D; i += kDT) {
      float v = i < rank ? __fmul_rn(__fdiv_rn(raw[i], rms), p.lat_gain[i]) : rotated(raw + rank, i - rank, s.rope_dims, cs);
      const CT t = cast_to<CT>(v);
      cur[i] = to_float(t);
      if (h == 0 && cr == 0 && !full) {
        if (i < rank) reinterpret_cast<CT*>(p.c_cache)[(size_t)pos * rank + i] = t;
        else reinterpret_cast<CT*>(p.kr_cache)[(size_t)pos * rot + i - rank] = t;
      }
    }
    if (full && h == 0 && cr == 0 && tid == 0 && p.state) atomicOr(&p.state->err, 2u);
    __syncthreads();
    const float* qrow = p.in + (size_t)h * (dim + rot);
    for (uint32_t i = tid; i < dim + rot; i += kDT) raw[i] = __ldcg(qrow + i);
    __syncthreads();
    for (uint32_t i = tid; i < rot; i += kDT) q[rank + i] = rotated(raw + dim, i, s.rope_dims, cs);
  }
  // first rows of the share are on their way while q_lat is made
  uint32_t nk = min((uint32_t)kKB, k1 - k0);
  stage(0, k0, nk);

  // ---- a slice of q_lat = W_uk^T q, written into every CTA of the cluster
  if (C > 1) cluster_wait();
  for (uint32_t base = sv0; base < sv1; base += kDT) {
    const uint32_t ns = min((uint32_t)kDT, sv1 - base), groups = kDT / ns, gi = tid / ns, vi = tid - gi * ns;
    if (gi < groups) {
      float acc[VEC];
#pragma unroll
      for (int e = 0; e < VEC; ++e) acc[e] = 0.f;
      const CT* w = Wuk + (size_t)(base + vi) * VEC;
#pragma unroll 4
      for (uint32_t d = gi; d < dim; d += groups) {
        float f[VEC];
        load_vec<CT, VEC>(w + (size_t)d * rank, f);
        const float qd = raw[d];
#pragma unroll
        for (int e = 0; e < VEC; ++e) acc[e] = fmaf(qd, f[e], acc[e]);
      }
#pragma unroll
      for (int e = 0; e < VEC; ++e) sm[L.part + (gi * ns + vi) * VEC + e] = acc[e];
    }
    __syncthreads();
    for (uint32_t i = tid; i < ns * VEC; i += kDT) {
      float a = 0.f;
      for (uint32_t g = 0; g < groups; ++g) a += sm[L.part + g * ns * VEC + i];
      float* dst = q + base * VEC + i;
      if (C == 1) *dst = a;
      else
        for (uint32_t c = 0; c < C; ++c) st_peer(peer_addr(dst, c), a);
    }
    __syncthreads();
  }
  if (C > 1) {
    cluster_arrive();
    cluster_wait();
  } else {
    __syncthreads();
  }

  // ---- this share of the window
  float m = kNeg, l = 0.f;
  float acc[kSlots][VEC];
#pragma unroll
  for (int j = 0; j < kSlots; ++j)
#pragma unroll
    for (int e = 0; e < VEC; ++e) acc[j][e] = 0.f;
  const uint32_t nvc = min(nv, (uint32_t)kDT), kgroups = kDT / nvc, kg = tid / nvc, vi = tid - kg * nvc;
  const uint32_t iters = (kKB + kgroups - 1) / kgroups;
  uint32_t buf = 0;
  for (uint32_t kb = k0; kb < k1; kb += kKB) {
    const uint32_t nk_next = kb + kKB < k1 ? min((uint32_t)kKB, k1 - kb - kKB) : 0u;
    if (L.nbuf == 2) {
      if (nk_next) stage(buf ^ 1u, kb + kKB, nk_next);
      else cp_commit();
      cp_wait<1>();
    } else {
      cp_wait<0>();
    }
    __syncthreads();
    const unsigned char* st = stage0 + buf * kKB * L.row_bytes;
    // scores: four rows per warp
    {
      float a[4] = {0.f, 0.f, 0.f, 0.f};
      for (uint32_t v = lane; v < D / VEC; v += 32) {
        float qf[VEC];
#pragma unroll
        for (int e = 0; e < VEC; ++e) qf[e] = q[v * VEC + e];
#pragma unroll
        for (int r = 0; r < 4; ++r) {
          if (warp * 4 + r < nk) {
            float f[VEC];
            load_vec<CT, VEC>(reinterpret_cast<const CT*>(st + (warp * 4 + r) * L.row_bytes) + v * VEC, f);
#pragma unroll
            for (int e = 0; e < VEC; ++e) a[r] = fmaf(qf[e], f[e], a[r]);
          }
        }
      }
#pragma unroll
      for (int r = 0; r < 4; ++r) {
        a[r] = warp_sum(a[r]);
        if (lane == 0) sm[L.sc + warp * 4 + r] = warp * 4 + r < nk ? a[r] * s.scale : -INFINITY;
      }
    }
    __syncthreads();
    // every warp repeats the small softmax for itself: lane = row
    const float sc = sm[L.sc + lane];
    const float mn = fmaxf(m, warp_max(sc));
    const float alpha = expf(m - mn), pr = expf(sc - mn);
    l = l * alpha + warp_sum(pr);
    m = mn;
#pragma unroll
    for (int j = 0; j < kSlots; ++j)
#pragma unroll
      for (int e = 0; e < VEC; ++e) acc[j][e] *= alpha;
    for (uint32_t it = 0; it < iters; ++it) {
      const uint32_t k = kg + it * kgroups;
      const float pk = __shfl_sync(0xffffffffu, pr, k & 31u);
      if (kg < kgroups && k < nk) {
        const CT* rowp = reinterpret_cast<const CT*>(st + k * L.row_bytes);
#pragma unroll
        for (int j = 0; j < kSlots; ++j) {
          const uint32_t v = vi + j * kDT;
          if (v < nv) {
            float f[VEC];
            load_vec<CT, VEC>(rowp + v * VEC, f);
#pragma unroll
            for (int e = 0; e < VEC; ++e) acc[j][e] = fmaf(pk, f[e], acc[j][e]);
          }
        }
      }
    }
    __syncthreads();  // everybody is done with this stage and with the scores
    if (L.nbuf == 2) buf ^= 1u;
    else if (nk_next) stage(0, kb + kKB, nk_next);
    nk = nk_next;
  }
  cp_wait<0>();
  // ---- the CTA's sum of latents
  float* const opart = sm + L.opart;
  if (kgroups > 1) {
    if (kg < kgroups) {
#pragma unroll
      for (int e = 0; e < VEC; ++e) sm[L.part + (kg * nv + vi) * VEC + e] = acc[0][e];
    }
    __syncthreads();
    for (uint32_t i = tid; i < rank; i += kDT) {
      float a = 0.f;
      for (uint32_t g = 0; g < kgroups; ++g) a += sm[L.part + g * rank + i];
      opart[i] = a;
    }
  } else {
#pragma unroll
    for (int j = 0; j < kSlots; ++j) {
      const uint32_t v = vi + j * kDT;
      if (kg == 0 && v < nv) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) opart[v * VEC + e] = acc[j][e];
      }
    }
  }
  if (tid == 0) {
    sm[L.ml] = m;
    sm[L.ml + 1] = l;
  }
  // ---- merge the shares (in rank order, the same in every CTA)
  float* const om = sm + L.om;
  if (C > 1) {
    cluster_arrive();
    cluster_wait();
    float M = kNeg, Lsum = 0.f, w[8];
#pragma unroll
    for (int c = 0; c < 8; ++c)
      if (c < (int)C) {
        const float lc = ld_peer(peer_addr(sm + L.ml + 1, c));
        w[c] = lc > 0.f ? ld_peer(peer_addr(sm + L.ml, c)) : kNeg;
        M = fmaxf(M, w[c]);
      }
#pragma unroll
    for (int c = 0; c < 8; ++c)
      if (c < (int)C) {
        const float lc = ld_peer(peer_addr(sm + L.ml + 1, c));
        w[c] = lc > 0.f ? expf(w[c] - M) : 0.f;
        Lsum = fmaf(w[c], lc, Lsum);
      }
    const float inv = 1.0f / Lsum;
    for (uint32_t i = tid; i < rank; i += kDT) {
      float a = 0.f;
#pragma unroll
      for (int c = 0; c < 8; ++c)
        if (c < (int)C) a = fmaf(w[c], ld_peer(peer_addr(opart + i, c)), a);
      om[i] = a * inv;
    }
    cluster_arrive();  // this CTA reads no peer any more; waited for before it leaves
  } else {
    __syncthreads();
    const float inv = 1.0f / sm[L.ml + 1];
    for (uint32_t i = tid; i < rank; i += kDT) om[i] = opart[i] * inv;
  }
  __syncthreads();
  // ---- a slice of the values, gated
  const float* gate = p.in + s.q_rows() + s.kv_rows() + (size_t)h * s.vdim;
  for (uint32_t o = o0 + warp; o < o1; o += kDT / 32) {
    const CT* w = Wuv + (size_t)o * rank;
    float a = 0.f;
#pragma unroll 2
    for (uint32_t v = lane; v < nv; v += 32) {
      float f[VEC];
      load_vec<CT, VEC>(w + v * VEC, f);
#pragma unroll
      for (int e = 0; e < VEC; ++e) a = fmaf(f[e], om[v * VEC + e], a);
    }
    a = warp_sum(a);
    if (lane == 0) p.out[(size_t)h * s.vdim + o] = a * sigmoid_f(__ldcg(gate + o));
  }
  if (C > 1) cluster_wait();  // no CTA leaves while another may still read its shared memory
}

template <typename CT, int VEC>
cudaError_t launch_decode_t(cudaStream_t s, const LatentParams& p, uint32_t C, bool pdl) {
  const DecodeLayout L = decode_layout(p.spec, sizeof(CT), VEC);
  auto kern = latent_decode_kernel<CT, VEC>;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)L.total);
  if (e != cudaSuccess) return e;
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(C, p.spec.heads);
  cfg.blockDim = dim3(kDT);
  cfg.dynamicSmemBytes = L.total;
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
  return cudaLaunchKernelEx(&cfg, kern, p, C);
}

uint32_t vec_of(const LatentSpec& s, int dtype) {
  const uint32_t ve = dtype == 0 ? 4 : 8;
  return s.rank % ve == 0 && s.rot % ve == 0 ? ve : 1;
}

// ---- prompt path: norm, rotate, cache rows ---------------------------------------------------------------------------------
template <typename CT>
__global__ void __launch_bounds__(256) latent_prep_kernel(const LatentParams p) {
  __shared__ float red[8];
  const LatentSpec& s = p.spec;
  pdl_launch_dependents();
  pdl_wait();
  const uint32_t t = blockIdx.x, pos = p.pos0 + t, rank = s.rank, rot = s.rot, hd = s.dim + rot;
  const float* row = p.in + (size_t)t * p.in_ld;
  const float* kv = row + s.q_rows();
  const float2* cs = p.rope_cs + (size_t)pos * (s.rope_dims / 2);
  float ss = 0.f;
  for (uint32_t i = threadIdx.x; i < rank; i += 256) ss = fmaf(kv[i], kv[i], ss);
  ss = warp_sum(ss);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
  __syncthreads();
  float tot = 0.f;
#pragma unroll
  for (int w = 0; w < 8; ++w) tot += red[w];
  const float rms = sqrtf(__fdiv_rn(tot, (float)rank) + p.eps);
  CT* c = reinterpret_cast<CT*>(p.c_cache) + (size_t)pos * rank;
  for (uint32_t i = threadIdx.x; i < rank; i += 256) store_as(c + i, __fmul_rn(__fdiv_rn(kv[i], rms), p.lat_gain[i]));
  CT* k = reinterpret_cast<CT*>(p.kr_cache) + (size_t)pos * rot;
  for (uint32_t i = threadIdx.x; i < rot; i += 256) store_as(k + i, rotated(kv + rank, i, s.rope_dims, cs));
  // a warp per head: four values a lane where the layout allows it
  const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const bool quads = s.dim % 4 == 0 && hd % 4 == 0 && p.in_ld % 4 == 0;
  for (uint32_t h = warp; h < s.heads; h += 8) {
    const float* src = row + (size_t)h * hd;
    CT* q = reinterpret_cast<CT*>(p.q) + (size_t)t * s.q_rows() + (size_t)h * hd;
    if (quads) {
      for (uint32_t i = lane * 4; i < s.dim; i += 128) {
        const float4 v = *reinterpret_cast<const float4*>(src + i);
        if constexpr (sizeof(CT) == 2) {
          __nv_bfloat162 o[2] = {__floats2bfloat162_rn(v.x, v.y), __floats2bfloat162_rn(v.z, v.w)};
          *reinterpret_cast<uint2*>(q + i) = *reinterpret_cast<uint2*>(o);
        } else {
          *reinterpret_cast<float4*>(q + i) = v;
        }
      }
    } else {
      for (uint32_t i = lane; i < s.dim; i += 32) store_as(q + i, src[i]);
    }
    for (uint32_t i = lane; i < rot; i += 32) store_as(q + s.dim + i, rotated(src + s.dim, i, s.rope_dims, cs));
  }
}

// ---- prompt path: any sizes, float32 arithmetic -------------------------------------------------------------------------------
constexpr int kST = 128, kSB = 64;
template <typename CT>
__global__ void __launch_bounds__(kST) latent_prefill_simt_kernel(const LatentParams p) {
  extern __shared__ float psm[];
  const LatentSpec& s = p.spec;
  const uint32_t t = blockIdx.x, h = blockIdx.y, dim = s.dim, rot = s.rot, hd = dim + rot, vdim = s.vdim;
  const uint32_t tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  float* q = psm;          // [hd]
  float* o = q + hd;       // [vdim]
  float* sc = o + vdim;    // [kSB]
  pdl_launch_dependents();
  pdl_wait();
  const CT* qr = reinterpret_cast<const CT*>(p.q) + (size_t)t * s.q_rows() + (size_t)h * hd;
  for (uint32_t i = tid; i < hd; i += kST) q[i] = to_float(qr[i]);
  for (uint32_t i = tid; i < vdim; i += kST) o[i] = 0.f;
  const uint32_t pos = p.pos0 + t, lo = s.window && pos + 1 > s.window ? pos + 1 - s.window : 0u;
  const uint32_t ld = s.heads * (dim + vdim);
  const CT* kv = reinterpret_cast<const CT*>(p.kv);
  const CT* kr = reinterpret_cast<const CT*>(p.kr_cache);
  float m = kNeg, l = 0.f;
  for (uint32_t kb = lo; kb <= pos; kb += kSB) {
    const uint32_t nk = min((uint32_t)kSB, pos - kb + 1);
    __syncthreads();
    for (uint32_t k = warp; k < nk; k += kST / 32) {
      const CT* row = kv + (size_t)(kb + k - p.kv_pos0) * ld + (size_t)h * dim;
      const CT* rr = kr + (size_t)(kb + k) * rot;
      float a = 0.f;
      for (uint32_t i = lane; i < dim; i += 32) a = fmaf(q[i], to_float(row[i]), a);
      for (uint32_t i = lane; i < rot; i += 32) a = fmaf(q[dim + i], to_float(rr[i]), a);
      a = warp_sum(a);
      if (lane == 0) sc[k] = a * s.scale;
    }
    __syncthreads();
    const float s0 = lane < nk ? sc[lane] : -INFINITY, s1 = lane + 32 < nk ? sc[lane + 32] : -INFINITY;
    const float mn = fmaxf(m, warp_max(fmaxf(s0, s1)));
    const float alpha = expf(m - mn);
    l = l * alpha + warp_sum(expf(s0 - mn) + expf(s1 - mn));
    m = mn;
    for (uint32_t i = tid; i < vdim; i += kST) {
      float a = o[i] * alpha;
      const CT* col = kv + (size_t)(kb - p.kv_pos0) * ld + (size_t)s.heads * dim + (size_t)h * vdim + i;
      for (uint32_t k = 0; k < nk; ++k) a = fmaf(expf(sc[k] - mn), to_float(col[(size_t)k * ld]), a);
      o[i] = a;
    }
  }
  const float inv = 1.0f / l;
  const float* gate = p.in + (size_t)t * p.in_ld + s.q_rows() + s.kv_rows() + (size_t)h * vdim;
  CT* out = reinterpret_cast<CT*>(p.ao) + (size_t)t * s.gate_rows() + (size_t)h * vdim;
  for (uint32_t i = tid; i < vdim; i += kST) store_as(out + i, o[i] * inv * sigmoid_f(gate[i]));
}

}  // namespace

bool latent_supported(const LatentSpec& s, int dtype, std::string* why) {
  const uint32_t vec = vec_of(s, dtype), elem = dtype == 0 ? 4 : 2;
  if (s.rank / vec > (uint32_t)kDT * kSlots) { *why = "kv_rank is too large for the latent attention kernel"; return false; }
  if (decode_layout(s, elem, vec).total > 227u * 1024u) { *why = "the latent attention sizes exceed shared memory"; return false; }
  if ((size_t)(s.dim + s.rot + s.vdim + kSB) * 4 > 48 * 1024) { *why = "head sizes are too large"; return false; }
  return true;
}

// latent_decode_mma.cu
bool latent_decode_mma_supported(const LatentSpec& s);
size_t latent_decode_mma_scratch(const LatentSpec& s, uint32_t ctx, size_t* tiles_bytes);
cudaError_t launch_latent_decode_mma(cudaStream_t s, const LatentParams& p, uint32_t rows, bool pdl, int* launches);

static bool decode_on_tensor_cores(const LatentSpec& s, int dtype) {
  static const bool on = env_int("NFAI_LATENT_MMA", 1) != 0;
  return dtype == 2 && on && latent_decode_mma_supported(s);
}

size_t latent_decode_scratch(const LatentSpec& s, int dtype, uint32_t ctx) {
  return decode_on_tensor_cores(s, dtype) ? latent_decode_mma_scratch(s, ctx, nullptr) : 0;
}

cudaError_t launch_latent_decode(cudaStream_t s, const LatentParams& p, bool pdl, int* launches) {
  const uint32_t rows = p.spec.window && p.spec.window < p.ctx ? p.spec.window : p.ctx;
  if (decode_on_tensor_cores(p.spec, p.dtype)) return launch_latent_decode_mma(s, p, rows, pdl, launches);
  if (launches) ++*launches;
  // CTAs per head: as many as keep the grid within one wave, but no more than there are blocks of rows to share
  uint32_t C = 8;
  while (C > 1 && (C * p.spec.heads > sm_count() || (rows + C - 1) / C < 16)) C >>= 1;
  if (p.dtype == 0) return vec_of(p.spec, 0) > 1 ? launch_decode_t<float, 4>(s, p, C, pdl) : launch_decode_t<float, 1>(s, p, C, pdl);
  if (p.dtype == 2)
    return vec_of(p.spec, 2) > 1 ? launch_decode_t<__nv_bfloat16, 8>(s, p, C, pdl) : launch_decode_t<__nv_bfloat16, 1>(s, p, C, pdl);
  return cudaErrorInvalidValue;
}

cudaError_t launch_latent_prep(cudaStream_t s, const LatentParams& p, uint32_t T) {
  if (p.dtype == 0) return launch_pdl(latent_prep_kernel<float>, dim3(T), dim3(256), 0, s, prefill_pdl(), p);
  return launch_pdl(latent_prep_kernel<__nv_bfloat16>, dim3(T), dim3(256), 0, s, prefill_pdl(), p);
}

bool latent_prefill_mma_supported(const LatentSpec& s);
cudaError_t launch_latent_prefill_mma(cudaStream_t s, const LatentParams& p, uint32_t T);

cudaError_t launch_latent_prefill(cudaStream_t s, const LatentParams& p, uint32_t T) {
  if (!T || p.spec.heads > 65535) return cudaErrorInvalidValue;
  static const bool mma_on = env_int("NFAI_PREFILL_ATTN", 1) != 0;
  if (p.dtype == 2 && mma_on && latent_prefill_mma_supported(p.spec)) return launch_latent_prefill_mma(s, p, T);
  const size_t smem = (size_t)(p.spec.dim + p.spec.rot + p.spec.vdim + kSB) * 4;
  const dim3 grid(T, p.spec.heads);
  if (p.dtype == 0) return launch_pdl(latent_prefill_simt_kernel<float>, grid, dim3(kST), smem, s, prefill_pdl(), p);
  return launch_pdl(latent_prefill_simt_kernel<__nv_bfloat16>, grid, dim3(kST), smem, s, prefill_pdl(), p);
}

}  // namespace nfai
