// Windowed causal attention of a prompt portion over expanded latents on the warp-level tensor cores (bfloat16 operands,
// float32 accumulators). A CTA owns 16 tokens per warp of one head and walks only the key tiles its tokens'
// windows reach. A key row is the head's unrotated part beside the rotated part all heads share; the two are brought
// together in shared memory. Scores, running maximum, exponentials and sums are float32; the weights go into the second
// product as a bfloat16 head and remainder (two MMAs, relative error ~2^-17), so that they keep more than the operand type.
// Head sizes are padded with zeros to the MMA's steps: any dim, rot and vdim up to the template's value width.
#include "attn_core.cuh"
#include "plan_kernels.h"

namespace nfai {

namespace {


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
__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// W warps of 16 tokens, key tiles of kN positions
template <int DV, int W, int kN>
__global__ void __launch_bounds__(W * 32, DV <= 128 ? 2 : 1) latent_prefill_mma_kernel(const LatentParams p, const uint32_t T, const uint32_t DQ,
                                                                  const int vec) {
  // DQ: dim + rot rounded up to 16
  constexpr int kM = W * 16, kThr = W * 32;
  extern __shared__ __align__(16) unsigned char lp_smem[];
  const LatentSpec& s = p.spec;
  const uint32_t dim = s.dim, rot = s.rot, hd = dim + rot, vdim = s.vdim;
  const uint32_t LQ = DQ + 8;
  constexpr uint32_t LV = DV + 8;
  __nv_bfloat16* const Qs = reinterpret_cast<__nv_bfloat16*>(lp_smem);
  __nv_bfloat16* const Ks = Qs + kM * LQ;       // two tiles
  __nv_bfloat16* const Vs = Ks + 2 * kN * LQ;   // two tiles
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, qr = lane >> 2, qc = (lane & 3) * 2;
  pdl_launch_dependents();
  pdl_wait();
  // the last tiles of tokens start first: without a window their work is the longest
  const uint32_t h = blockIdx.x % s.heads, tile = gridDim.x / s.heads - 1 - blockIdx.x / s.heads;
  const uint32_t t0 = tile * kM, rows_end = min(T, t0 + kM);
  const uint32_t first_pos = p.pos0 + t0;
  const uint32_t k_lo = s.window && first_pos + 1 > s.window ? first_pos + 1 - s.window : 0u;  // first position any row sees
  const uint32_t k_hi = p.pos0 + rows_end;                                                      // one past the last
  const __nv_bfloat16* const Q = reinterpret_cast<const __nv_bfloat16*>(p.q);
  const __nv_bfloat16* const KV = reinterpret_cast<const __nv_bfloat16*>(p.kv);
  const __nv_bfloat16* const KR = reinterpret_cast<const __nv_bfloat16*>(p.kr_cache);
  const size_t kv_ld = (size_t)s.heads * (dim + vdim), q_ld = (size_t)s.heads * hd;
  const __nv_bfloat16 zero = __float2bfloat16_rn(0.f);

  if (vec) {
    const uint32_t per = DQ / 8;
    for (uint32_t i = tid; i < kM * per; i += kThr) {
      const uint32_t r = i / per, c = (i - r * per) * 8, t = t0 + r;
      const bool in = t < T && c < hd;
      cpa16((uint32_t)__cvta_generic_to_shared(Qs + r * LQ + c), in ? Q + t * q_ld + (size_t)h * hd + c : Q, in ? 16u : 0u);
    }
  } else {
    for (uint32_t i = tid; i < kM * DQ; i += kThr) {
      const uint32_t r = i / DQ, c = i - r * DQ, t = t0 + r;
      Qs[r * LQ + c] = t < T && c < hd ? Q[t * q_ld + (size_t)h * hd + c] : zero;
    }
  }
  auto issue = [&](uint32_t buf, uint32_t kb) {
    __nv_bfloat16* const kd = Ks + buf * kN * LQ;
    __nv_bfloat16* const vd = Vs + buf * kN * LV;
    if (vec) {
      const uint32_t per = DQ / 8, dv8 = dim / 8, rv8 = hd / 8;
      for (uint32_t i = tid; i < kN * per; i += kThr) {
        const uint32_t r = i / per, c = i - r * per, pos = kb + r;
        const bool in = pos < k_hi && c < rv8;
        const __nv_bfloat16* src = !in ? KV : c < dv8 ? KV + (size_t)(pos - p.kv_pos0) * kv_ld + (size_t)h * dim + c * 8
                                                     : KR + (size_t)pos * rot + (c - dv8) * 8;
        cpa16((uint32_t)__cvta_generic_to_shared(kd + r * LQ + c * 8), src, in ? 16u : 0u);
      }
      constexpr uint32_t pv = DV / 8;
      for (uint32_t i = tid; i < kN * pv; i += kThr) {
        const uint32_t r = i / pv, c = (i - r * pv) * 8, pos = kb + r;
        const bool in = pos < k_hi && c < vdim;
        cpa16((uint32_t)__cvta_generic_to_shared(vd + r * LV + c),
              in ? KV + (size_t)(pos - p.kv_pos0) * kv_ld + (size_t)s.heads * dim + (size_t)h * vdim + c : KV, in ? 16u : 0u);
      }
    } else {
      for (uint32_t i = tid; i < kN * DQ; i += kThr) {
        const uint32_t r = i / DQ, c = i - r * DQ, pos = kb + r;
        kd[r * LQ + c] = pos >= k_hi || c >= hd ? zero
                         : c < dim ? KV[(size_t)(pos - p.kv_pos0) * kv_ld + (size_t)h * dim + c] : KR[(size_t)pos * rot + c - dim];
      }
      for (uint32_t i = tid; i < kN * DV; i += kThr) {
        const uint32_t r = i / DV, c = i - r * DV, pos = kb + r;
        vd[r * LV + c] = pos >= k_hi || c >= vdim ? zero : KV[(size_t)(pos - p.kv_pos0) * kv_ld + (size_t)s.heads * dim + (size_t)h * vdim + c];
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };

  const uint32_t row_a = t0 + warp * 16 + qr, row_b = row_a + 8;
  const uint32_t pos_a = p.pos0 + row_a, pos_b = p.pos0 + row_b;
  const uint32_t win = s.window ? s.window : 0xffffffffu;
  const float qs = s.scale * 1.4426950408889634f;
  float o[DV / 8][4];
#pragma unroll
  for (int j = 0; j < DV / 8; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
  float m_a = attn_detail::kNegBig, m_b = attn_detail::kNegBig, l_a = 0.f, l_b = 0.f;
  const int lm = lane >> 3, lr = lane & 7;
  const uint32_t q_s = (uint32_t)__cvta_generic_to_shared(Qs) + (uint32_t)((warp * 16 + (lm & 1) * 8 + lr) * LQ + (lm >> 1) * 8) * 2;
  const uint32_t k_off = (uint32_t)(((lm >> 1) * 8 + lr) * LQ + (lm & 1) * 8) * 2;
  const uint32_t v_off = (uint32_t)(((lm & 1) * 8 + lr) * LV + (lm >> 1) * 8) * 2;
  const uint32_t ks_b = (uint32_t)__cvta_generic_to_shared(Ks), vs_b = (uint32_t)__cvta_generic_to_shared(Vs);
  // rows of this warp see positions [w_lo, w_hi]
  const uint32_t w_first = p.pos0 + t0 + warp * 16, w_hi = w_first + 15;
  const uint32_t w_lo = w_first + 1 > win ? w_first + 1 - win : 0u;

  issue(0, k_lo);
  uint32_t buf = 0;
  for (uint32_t kb = k_lo; kb < k_hi; kb += kN, buf ^= 1u) {
    if (kb + kN < k_hi) issue(buf ^ 1u, kb + kN);
    else asm volatile("cp.async.commit_group;" ::: "memory");
    asm volatile("cp.async.wait_group 1;" ::: "memory");
    __syncthreads();
    if (kb <= w_hi && kb + kN > w_lo) {
      const uint32_t ks = ks_b + buf * (uint32_t)(kN * LQ * 2), vs = vs_b + buf * (uint32_t)(kN * LV * 2);
      float c[kN / 8][4];
#pragma unroll
      for (int j = 0; j < kN / 8; ++j) c[j][0] = c[j][1] = c[j][2] = c[j][3] = 0.f;
      for (uint32_t kk = 0; kk < DQ / 16; ++kk) {
        uint32_t a[4];
        ldsm4(q_s + kk * 32, a);
#pragma unroll
        for (int j = 0; j < kN / 8; j += 2) {
          uint32_t b[4];
          ldsm4(ks + (uint32_t)(j * 8 * LQ) * 2 + kk * 32 + k_off, b);
          mma_bf16(c[j], a, b[0], b[1]);
          mma_bf16(c[j + 1], a, b[2], b[3]);
        }
      }
#pragma unroll
      for (int j = 0; j < kN / 8; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) c[j][e] *= qs;
      // not every row of the warp sees the whole tile: mask
      if (kb + kN - 1 > w_first || kb < (w_hi + 1 > win ? w_hi + 1 - win : 0u)) {
#pragma unroll
        for (int j = 0; j < kN / 8; ++j) {
          const uint32_t k = kb + j * 8 + qc;
          if (k > pos_a || pos_a - k >= win) c[j][0] = -INFINITY;
          if (k + 1 > pos_a || pos_a - (k + 1) >= win) c[j][1] = -INFINITY;
          if (k > pos_b || pos_b - k >= win) c[j][2] = -INFINITY;
          if (k + 1 > pos_b || pos_b - (k + 1) >= win) c[j][3] = -INFINITY;
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
      const float mn_a = fmaxf(m_a, mx_a), mn_b = fmaxf(m_b, mx_b);
      const float al_a = ex2(m_a - mn_a), al_b = ex2(m_b - mn_b);
      m_a = mn_a;
      m_b = mn_b;
      float sum_a = 0.f, sum_b = 0.f;
      uint32_t ph[kN / 16][4], pl[kN / 16][4];
#pragma unroll
      for (int j = 0; j < kN / 8; ++j) {
        const float e0 = ex2(c[j][0] - mn_a), e1 = ex2(c[j][1] - mn_a), e2 = ex2(c[j][2] - mn_b), e3 = ex2(c[j][3] - mn_b);
        sum_a += e0 + e1;
        sum_b += e2 + e3;
        const uint32_t ha = pack_bf(e0, e1), hb = pack_bf(e2, e3);
        const int i = j >> 1, w = (j & 1) * 2;
        ph[i][w] = ha;
        ph[i][w + 1] = hb;
        pl[i][w] = pack_bf(e0 - __uint_as_float(ha << 16), e1 - __uint_as_float(ha & 0xffff0000u));
        pl[i][w + 1] = pack_bf(e2 - __uint_as_float(hb << 16), e3 - __uint_as_float(hb & 0xffff0000u));
      }
      l_a = l_a * al_a + sum_a;
      l_b = l_b * al_b + sum_b;
#pragma unroll
      for (int j = 0; j < DV / 8; ++j) {
        o[j][0] *= al_a;
        o[j][1] *= al_a;
        o[j][2] *= al_b;
        o[j][3] *= al_b;
      }
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
    __syncthreads();  // the other buffer's tile may be overwritten in the next iteration
  }
  l_a += __shfl_xor_sync(0xffffffffu, l_a, 1);
  l_a += __shfl_xor_sync(0xffffffffu, l_a, 2);
  l_b += __shfl_xor_sync(0xffffffffu, l_b, 1);
  l_b += __shfl_xor_sync(0xffffffffu, l_b, 2);
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    const uint32_t row = half ? row_b : row_a;
    if (row >= T) continue;
    const float inv = 1.0f / (half ? l_b : l_a);
    const float* gate = p.in + (size_t)row * p.in_ld + s.q_rows() + s.kv_rows() + (size_t)h * vdim;
    __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(p.ao) + (size_t)row * s.gate_rows() + (size_t)h * vdim;
#pragma unroll
    for (int j = 0; j < DV / 8; ++j)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const uint32_t c = j * 8 + qc + e;
        if (c < vdim) store_as(out + c, o[j][half * 2 + e] * inv * (1.0f / (1.0f + expf(-gate[c]))));
      }
  }
}

size_t mma_smem(uint32_t DQ, uint32_t DV, uint32_t kM, uint32_t kN) { return ((size_t)(kM + 2 * kN) * (DQ + 8) + (size_t)2 * kN * (DV + 8)) * 2; }
uint32_t value_width(uint32_t vdim) { return vdim <= 32 ? 32 : vdim <= 64 ? 64 : vdim <= 128 ? 128 : vdim <= 256 ? 256 : 0; }

// 8 warps and tiles of 32 positions: two CTAs per SM share the tensor cores, and 128 tokens share a tile (measured against
// 4 and 8 warps with 32 and 64 positions).
constexpr int kWarpsPerCta = 8, kTilePositions = 32;

template <int DV>
cudaError_t launch_dv(cudaStream_t s, const LatentParams& p, uint32_t T) {
  const LatentSpec& sp = p.spec;
  constexpr uint32_t kM = kWarpsPerCta * 16;
  const uint32_t DQ = (sp.dim + sp.rot + 15u) & ~15u;
  const size_t smem = mma_smem(DQ, DV, kM, kTilePositions);
  auto kern = latent_prefill_mma_kernel<DV, kWarpsPerCta, kTilePositions>;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) return e;
  const int vec = sp.dim % 8 == 0 && sp.rot % 8 == 0 && sp.vdim % 8 == 0;
  return launch_pdl(kern, dim3((T + kM - 1) / kM * sp.heads), dim3(kWarpsPerCta * 32), smem, s, prefill_pdl(), p, T, DQ, vec);
}

}  // namespace

bool latent_prefill_mma_supported(const LatentSpec& s) {
  const uint32_t dv = value_width(s.vdim);
  return dv && mma_smem((s.dim + s.rot + 15u) & ~15u, dv, kWarpsPerCta * 16, kTilePositions) <= 227 * 1024;
}

cudaError_t launch_latent_prefill_mma(cudaStream_t s, const LatentParams& p, uint32_t T) {
  switch (value_width(p.spec.vdim)) {
    case 32: return launch_dv<32>(s, p, T);
    case 64: return launch_dv<64>(s, p, T);
    case 128: return launch_dv<128>(s, p, T);
    case 256: return launch_dv<256>(s, p, T);
    default: return cudaErrorInvalidValue;
  }
}

}  // namespace nfai
