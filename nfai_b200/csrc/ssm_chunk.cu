// The recurrence of a state space layer over a prompt portion, in chunks of 128 tokens on the warp-level tensor cores.
//
// Inside a chunk, with c_i the running sum of the log decays -exp(A_log) dt (inclusive), S0 the state before the chunk:
//   y_i = exp(c_i) C_i S0 + sum_{j<=i} (C_i . B_j) exp(c_i - c_j) dt_j x_j          and after it
//   S1  = exp(c_last) S0 + sum_j exp(c_last - c_j) dt_j x_j B_j^T
// Three kernels: ssm_chunk_state (what each chunk adds to the state, all chunks in parallel), ssm_chunk_pass (the states
// before every chunk, a short serial walk per element, float32), ssm_chunk_out (the outputs).
//
// Precision: x, B and C are bfloat16 results of projection and convolution and enter the products as they are. Everything
// float32 that has to be an operand (decay times step times x, the decayed weights of a chunk, the state) is split into
// three bfloat16 terms that together carry its 24 bits; products accumulate in float32. The sums c_i are formed in double and kept
// as two floats, so that differences of large sums stay exact.
#include "common.cuh"
#include "plan_kernels.h"

namespace nfai {

namespace {

constexpr uint32_t kQ = 128;  // tokens per chunk
constexpr int kThr = 256;

__device__ __forceinline__ uint32_t pack2(float a, float b) {
  __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<uint32_t*>(&h);
}
__device__ __forceinline__ float lo_f(uint32_t w) { return __uint_as_float(w << 16); }
__device__ __forceinline__ float hi_f(uint32_t w) { return __uint_as_float(w & 0xffff0000u); }
// (a, b) as three packed bfloat16 pairs whose sum is (a, b) to float32 accuracy
__device__ __forceinline__ void split3(float a, float b, uint32_t& p0, uint32_t& p1, uint32_t& p2) {
  p0 = pack2(a, b);
  a -= lo_f(p0);
  b -= hi_f(p0);
  p1 = pack2(a, b);
  p2 = pack2(a - lo_f(p1), b - hi_f(p1));
}
__device__ __forceinline__ void mma_bf(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldsm(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm_t(uint32_t addr, uint32_t (&r)[4]) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr));
}
__device__ __forceinline__ uint32_t s32(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }

// rows [0, kQ) of `cols` bfloat16 columns (padded with zeros to `pad`) from global rows t0 + r (zero past T)
__device__ __forceinline__ void load_tile(__nv_bfloat16* dst, uint32_t ld, const __nv_bfloat16* src, size_t src_ld, uint32_t t0,
                                          uint32_t T, uint32_t cols, uint32_t pad, bool vec) {
  if (vec) {
    const uint32_t per = pad / 8;
    for (uint32_t i = threadIdx.x; i < kQ * per; i += kThr) {
      const uint32_t r = i / per, c = (i - r * per) * 8, t = t0 + r;
      const bool in = t < T && c < cols;
      asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(s32(dst + r * ld + c)),
                   "l"(in ? src + (size_t)t * src_ld + c : src), "r"(in ? 16u : 0u)
                   : "memory");
    }
  } else {
    for (uint32_t i = threadIdx.x; i < kQ * pad; i += kThr) {
      const uint32_t r = i / pad, c = i - r * pad, t = t0 + r;
      dst[r * ld + c] = t < T && c < cols ? src[(size_t)t * src_ld + c] : __float2bfloat16_rn(0.f);
    }
  }
  asm volatile("cp.async.commit_group;" ::: "memory");
}
__device__ __forceinline__ void wait_copies() { asm volatile("cp.async.wait_group 0;" ::: "memory"); }

// Step sizes and running log-decay sums of this chunk (warp 0): c as head and remainder, dt (zero past T).
__device__ __forceinline__ void chunk_sums(const SsmParams& p, uint32_t h, uint32_t t0, uint32_t T, float* ch, float* cl, float* dts) {
  if (threadIdx.x >= 32) return;
  const int lane = threadIdx.x;
  const double A = -(double)expf(p.A_log[h]);
  double loc[kQ / 32], run = 0.0;
#pragma unroll
  for (int j = 0; j < (int)kQ / 32; ++j) {
    const uint32_t i = lane * (kQ / 32) + j, t = t0 + i;
    const float dt = t < T ? p.dt[(size_t)t * p.spec.heads + h] : 0.f;
    dts[i] = dt;
    run += A * (double)dt;
    loc[j] = run;
  }
  double incl = run;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const double v = __shfl_up_sync(0xffffffffu, incl, o);
    if (lane >= o) incl += v;
  }
  const double before = incl - run;
#pragma unroll
  for (int j = 0; j < (int)kQ / 32; ++j) {
    const uint32_t i = lane * (kQ / 32) + j;
    const double c = before + loc[j];
    ch[i] = (float)c;
    cl[i] = (float)(c - (double)ch[i]);
  }
}

// The chunk workspace: decays [chunks][heads], running sums (head, remainder, step size) [chunks][heads][3][kQ], then what
// every chunk adds to the state [chunks][heads][vdim][state].
__host__ __device__ inline size_t sums_offset(uint32_t heads, uint32_t nchunks) { return ((size_t)nchunks * heads + 3) & ~(size_t)3; }
__host__ __device__ inline size_t added_offset(uint32_t heads, uint32_t nchunks) {
  return sums_offset(heads, nchunks) + (size_t)nchunks * heads * 3 * kQ;
}

__host__ __device__ inline uint32_t pad16(uint32_t n) { return (n + 15u) & ~15u; }

// ---- what a chunk adds to the state: [V][N] = sum_j (exp(c_last - c_j) dt_j x_j) B_j^T ----------------------------------------
__global__ void __launch_bounds__(kThr) ssm_chunk_state_kernel(const SsmParams p, const uint32_t T, const int vec) {
  extern __shared__ __align__(16) unsigned char cs_smem[];
  const SsmSpec& sp = p.spec;
  const uint32_t V = sp.vdim, N = sp.state, Vp = pad16(V), Np = pad16(N), LX = Vp + 8, LB = Np + 8;
  const uint32_t chunk = blockIdx.x, h = blockIdx.y, g = h / (sp.heads / sp.groups), t0 = chunk * kQ, CH = sp.channels();
  __nv_bfloat16* const Xs = reinterpret_cast<__nv_bfloat16*>(cs_smem);
  __nv_bfloat16* const Bs = Xs + kQ * LX;
  float* const ch = reinterpret_cast<float*>(Bs + kQ * LB);
  float* const cl = ch + kQ;
  float* const wt = cl + kQ;
  pdl_launch_dependents();
  pdl_wait();
  const __nv_bfloat16* xbc = reinterpret_cast<const __nv_bfloat16*>(p.xbc);
  load_tile(Xs, LX, xbc + (size_t)h * V, CH, t0, T, V, Vp, vec);
  load_tile(Bs, LB, xbc + sp.inner() + (size_t)g * N, CH, t0, T, N, Np, vec);
  chunk_sums(p, h, t0, T, ch, cl, wt);
  __syncthreads();
  float* const sums = p.chunk + sums_offset(sp.heads, gridDim.x) + ((size_t)chunk * sp.heads + h) * 3 * kQ;
  for (uint32_t i = threadIdx.x; i < 3 * kQ; i += kThr) sums[i] = ch[i];  // for the output kernel (ch, cl and wt are contiguous)
  __syncthreads();
  const float cend_h = ch[kQ - 1], cend_l = cl[kQ - 1];
  if (threadIdx.x < kQ) wt[threadIdx.x] *= expf((cend_h - ch[threadIdx.x]) + (cend_l - cl[threadIdx.x]));
  const size_t per_head = (size_t)V * N;
  float* const decays = p.chunk;  // [chunks][heads]
  const uint32_t nchunks = gridDim.x;
  if (threadIdx.x == 0) decays[(size_t)chunk * sp.heads + h] = expf(cend_h + cend_l);
  wait_copies();
  __syncthreads();
  float* const out = p.chunk + added_offset(sp.heads, nchunks) + ((size_t)chunk * sp.heads + h) * per_head;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, lm = lane >> 3, lr = lane & 7, qr = lane >> 2, qc = (lane & 3) * 2;
  const uint32_t ntiles = (Np + 63) / 64, tiles = Vp / 16 * ntiles;
  for (uint32_t tile = warp; tile < tiles; tile += kThr / 32) {
    const uint32_t v0 = tile / ntiles * 16, n0 = tile % ntiles * 64;
    const int nj = (int)min(8u, (Np - n0) / 8);  // even
    float acc[8][4];
#pragma unroll
    for (int j = 0; j < 8; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
    for (uint32_t k0 = 0; k0 < kQ; k0 += 16) {
      uint32_t a[4], a0[4], a1[4], a2[4];
      ldsm_t(s32(Xs + (k0 + (lm >> 1) * 8 + lr) * LX + v0 + (lm & 1) * 8), a);
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float w0 = wt[k0 + (i >> 1) * 8 + qc], w1 = wt[k0 + (i >> 1) * 8 + qc + 1];
        split3(w0 * lo_f(a[i]), w1 * hi_f(a[i]), a0[i], a1[i], a2[i]);
      }
#pragma unroll
      for (int j = 0; j < 8; j += 2) {
        if (j < nj) {
          uint32_t b[4];
          ldsm_t(s32(Bs + (k0 + (lm & 1) * 8 + lr) * LB + n0 + j * 8 + (lm >> 1) * 8), b);
          mma_bf(acc[j], a0, b[0], b[1]);
          mma_bf(acc[j + 1], a0, b[2], b[3]);
          mma_bf(acc[j], a1, b[0], b[1]);
          mma_bf(acc[j + 1], a1, b[2], b[3]);
          mma_bf(acc[j], a2, b[0], b[1]);
          mma_bf(acc[j + 1], a2, b[2], b[3]);
        }
      }
    }
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const uint32_t n = n0 + j * 8 + qc;
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const uint32_t v = v0 + qr + (e >> 1) * 8;
        if (v < V && n + (e & 1) < N) out[(size_t)v * N + n + (e & 1)] = acc[j][e];
      }
    }
  }
}

// ---- states before every chunk, in place of what the chunks add; the state after the last one into p.S -------------------------
__global__ void __launch_bounds__(128) ssm_chunk_pass_kernel(const SsmParams p, const uint32_t nchunks) {
  pdl_launch_dependents();
  pdl_wait();
  const size_t per_head = (size_t)p.spec.vdim * p.spec.state, total = per_head * p.spec.heads;
  const float* decays = p.chunk;
  float* add = p.chunk + added_offset(p.spec.heads, nchunks);
  auto walk = [&](auto* s_ptr, auto* a_ptr, size_t stride, uint32_t h, auto&& step) {
    auto s = *s_ptr;
    if (p.pos0 == 0) step(s, 0.f, s, true);
    for (uint32_t c0 = 0; c0 < nchunks; c0 += 8) {
      decltype(s) a[8];
      float d[8];
#pragma unroll
      for (int j = 0; j < 8; ++j)
        if (c0 + j < nchunks) {
          a[j] = a_ptr[(size_t)(c0 + j) * stride];
          d[j] = decays[(size_t)(c0 + j) * p.spec.heads + h];
        }
#pragma unroll
      for (int j = 0; j < 8; ++j)
        if (c0 + j < nchunks) {
          a_ptr[(size_t)(c0 + j) * stride] = s;
          step(s, d[j], a[j], false);
        }
    }
    *s_ptr = s;
  };
  const size_t i = (size_t)blockIdx.x * 128 + threadIdx.x;
  if (per_head % 4 == 0) {
    if (i * 4 >= total) return;
    walk(reinterpret_cast<float4*>(p.S) + i, reinterpret_cast<float4*>(add) + i, total / 4, (uint32_t)(i * 4 / per_head),
         [](float4& s, float d, const float4& a, bool zero) {
           if (zero) s = make_float4(0.f, 0.f, 0.f, 0.f);
           else s = make_float4(fmaf(d, s.x, a.x), fmaf(d, s.y, a.y), fmaf(d, s.z, a.z), fmaf(d, s.w, a.w));
         });
  } else {
    if (i >= total) return;
    walk(p.S + i, add + i, total, (uint32_t)(i / per_head), [](float& s, float d, const float& a, bool zero) { s = zero ? 0.f : fmaf(d, s, a); });
  }
}

// ---- outputs ---------------------------------------------------------------------------------------------------------------------
// VT: values of a head, padded (multiple of 16). Eight warps of 16 tokens.
template <int VT>
__global__ void __launch_bounds__(kThr, VT <= 64 ? 2 : 1) ssm_chunk_out_kernel(const SsmParams p, const uint32_t T, const int vec) {
  extern __shared__ __align__(16) unsigned char co_smem[];
  const SsmSpec& sp = p.spec;
  const uint32_t V = sp.vdim, N = sp.state, Np = pad16(N), LB = Np + 8;
  constexpr uint32_t LX = VT + 8;
  const uint32_t chunk = blockIdx.x, h = blockIdx.y, g = h / (sp.heads / sp.groups), t0 = chunk * kQ, CH = sp.channels(), inner = sp.inner();
  __nv_bfloat16* const Cs = reinterpret_cast<__nv_bfloat16*>(co_smem);
  __nv_bfloat16* const Xs = Cs + kQ * LB;
  __nv_bfloat16* const Bs = Xs + kQ * LX;    // first the state's three terms [3][VT][LB], then B [kQ][LB]
  const uint32_t bs_elems = (3u * VT > kQ ? 3u * VT : kQ) * LB;
  float* const ch = reinterpret_cast<float*>(Bs + bs_elems);
  float* const cl = ch + kQ;
  float* const dts = cl + kQ;
  pdl_launch_dependents();
  pdl_wait();
  const __nv_bfloat16* xbc = reinterpret_cast<const __nv_bfloat16*>(p.xbc);
  // the gate's rows are needed last: have them on their way from memory
  for (uint32_t i = threadIdx.x; i < kQ * ((V * 4 + 127) / 128); i += kThr) {
    const uint32_t lines = (V * 4 + 127) / 128, r = i / lines, l = i - r * lines;
    if (t0 + r < T) asm volatile("prefetch.global.L2 [%0];" ::"l"(p.in + (size_t)(t0 + r) * sp.in_rows() + (size_t)h * V + l * 32));
  }
  load_tile(Cs, LB, xbc + inner + (size_t)(sp.groups + g) * N, CH, t0, T, N, Np, vec);
  load_tile(Xs, LX, xbc + (size_t)h * V, CH, t0, T, V, VT, vec);
  const float* sums = p.chunk + sums_offset(sp.heads, gridDim.x) + ((size_t)chunk * sp.heads + h) * 3 * kQ;
  for (uint32_t i = threadIdx.x; i < 3 * kQ; i += kThr) ch[i] = sums[i];  // ch, cl and dts are contiguous
  const size_t per_head = (size_t)V * N;
  const float* S0 = p.chunk + added_offset(sp.heads, gridDim.x) + ((size_t)chunk * sp.heads + h) * per_head;
#pragma unroll 4
  for (uint32_t i = threadIdx.x; i < VT * (Np / 2); i += kThr) {
    const uint32_t v = i / (Np / 2), n = (i - v * (Np / 2)) * 2;
    const float a = v < V && n < N ? S0[(size_t)v * N + n] : 0.f, b = v < V && n + 1 < N ? S0[(size_t)v * N + n + 1] : 0.f;
    uint32_t w0, w1, w2;
    split3(a, b, w0, w1, w2);
    *reinterpret_cast<uint32_t*>(Bs + v * LB + n) = w0;
    *reinterpret_cast<uint32_t*>(Bs + (VT + v) * LB + n) = w1;
    *reinterpret_cast<uint32_t*>(Bs + (2 * VT + v) * LB + n) = w2;
  }
  wait_copies();
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, lm = lane >> 3, lr = lane & 7, qr = lane >> 2, qc = (lane & 3) * 2;
  const uint32_t ia = warp * 16 + qr, ib = ia + 8;  // this thread's two tokens of the chunk
  const uint32_t c_addr = s32(Cs + (warp * 16 + (lm & 1) * 8 + lr) * LB + (lm >> 1) * 8);
  float o[VT / 8][4];
#pragma unroll
  for (int j = 0; j < VT / 8; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
  // from the state before the chunk
  for (uint32_t k0 = 0; k0 < Np; k0 += 16) {
    uint32_t a[4];
    ldsm(c_addr + k0 * 2, a);
#pragma unroll
    for (int term = 0; term < 3; ++term)
#pragma unroll
      for (int j = 0; j < VT / 8; j += 2) {
        uint32_t b[4];
        ldsm(s32(Bs + (term * VT + j * 8 + (lm >> 1) * 8 + lr) * LB + k0 + (lm & 1) * 8), b);
        mma_bf(o[j], a, b[0], b[1]);
        mma_bf(o[j + 1], a, b[2], b[3]);
      }
  }
  const float ea = expf(ch[ia] + cl[ia]), eb = expf(ch[ib] + cl[ib]);
#pragma unroll
  for (int j = 0; j < VT / 8; ++j) {
    o[j][0] *= ea;
    o[j][1] *= ea;
    o[j][2] *= eb;
    o[j][3] *= eb;
  }
  __syncthreads();  // everybody has read the state
  load_tile(Bs, LB, xbc + inner + (size_t)g * N, CH, t0, T, N, Np, vec);
  wait_copies();
  __syncthreads();
  // from the chunk itself: blocks of 32 earlier tokens
  const float cha = ch[ia], cla = cl[ia], chb = ch[ib], clb = cl[ib];
  for (uint32_t j0 = 0; j0 <= (uint32_t)warp * 16 + 15; j0 += 32) {
    float c[4][4];
#pragma unroll
    for (int j = 0; j < 4; ++j) c[j][0] = c[j][1] = c[j][2] = c[j][3] = 0.f;
    for (uint32_t k0 = 0; k0 < Np; k0 += 16) {
      uint32_t a[4];
      ldsm(c_addr + k0 * 2, a);
#pragma unroll
      for (int j = 0; j < 4; j += 2) {
        uint32_t b[4];
        ldsm(s32(Bs + (j0 + j * 8 + (lm >> 1) * 8 + lr) * LB + k0 + (lm & 1) * 8), b);
        mma_bf(c[j], a, b[0], b[1]);
        mma_bf(c[j + 1], a, b[2], b[3]);
      }
    }
    uint32_t w[3][2][4];
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      float m[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const uint32_t jj = j0 + j * 8 + qc + (e & 1), i = e < 2 ? ia : ib;
        const float d = e < 2 ? (cha - ch[jj]) + (cla - cl[jj]) : (chb - ch[jj]) + (clb - cl[jj]);
        m[e] = jj <= i ? c[j][e] * expf(d) * dts[jj] : 0.f;
      }
      const int q = j >> 1, s = (j & 1) * 2;
      split3(m[0], m[1], w[0][q][s], w[1][q][s], w[2][q][s]);
      split3(m[2], m[3], w[0][q][s + 1], w[1][q][s + 1], w[2][q][s + 1]);
    }
#pragma unroll
    for (int q = 0; q < 2; ++q)
#pragma unroll
      for (int j = 0; j < VT / 8; j += 2) {
        uint32_t b[4];
        ldsm_t(s32(Xs + (j0 + q * 16 + (lm & 1) * 8 + lr) * LX + j * 8 + (lm >> 1) * 8), b);
#pragma unroll
        for (int term = 0; term < 3; ++term) {
          mma_bf(o[j], w[term][q], b[0], b[1]);
          mma_bf(o[j + 1], w[term][q], b[2], b[3]);
        }
      }
  }
  // skip and gate
  const float D = p.D[h];
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    const uint32_t i = half ? ib : ia, t = t0 + i;
    if (t >= T) continue;
    const float* z = p.in + (size_t)t * sp.in_rows() + (size_t)h * V;
    float* y = p.y + (size_t)t * inner + (size_t)h * V;
#pragma unroll
    for (int j = 0; j < VT / 8; ++j)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const uint32_t v = j * 8 + qc + e;
        if (v < V) {
          const float x = to_float(Xs[i * LX + v]), zz = z[v];
          y[v] = fmaf(D, x, o[j][half * 2 + e]) * (zz / (1.0f + expf(-zz)));
        }
      }
  }
}

size_t state_smem(const SsmSpec& s) { return (size_t)kQ * (pad16(s.vdim) + 8 + pad16(s.state) + 8) * 2 + 3 * kQ * 4; }
uint32_t out_width(uint32_t v) { return v <= 32 ? 32 : v <= 64 ? 64 : v <= 128 ? 128 : 0; }
size_t out_smem(const SsmSpec& s) {
  const uint32_t VT = out_width(s.vdim), LB = pad16(s.state) + 8;
  return ((size_t)kQ * LB + (size_t)kQ * (VT + 8) + (size_t)(3 * VT > kQ ? 3 * VT : kQ) * LB) * 2 + 3 * kQ * 4;
}

template <int VT>
cudaError_t launch_out(cudaStream_t s, const SsmParams& p, uint32_t T, uint32_t nchunks, int vec) {
  const size_t smem = out_smem(p.spec);
  cudaError_t e = cudaFuncSetAttribute(ssm_chunk_out_kernel<VT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) return e;
  return launch_pdl(ssm_chunk_out_kernel<VT>, dim3(nchunks, p.spec.heads), dim3(kThr), smem, s, prefill_pdl(), p, T, vec);
}

}  // namespace

bool ssm_chunk_supported(const SsmSpec& s) {
  return out_width(s.vdim) && out_smem(s) <= 227 * 1024 && state_smem(s) <= 227 * 1024 && s.heads <= 65535;
}

size_t ssm_chunk_floats(const SsmSpec& s, uint32_t T) {
  if (!ssm_chunk_supported(s)) return 0;
  const size_t n = (T + kQ - 1) / kQ;
  return added_offset(s.heads, (uint32_t)n) + n * s.heads * s.vdim * s.state;
}

cudaError_t launch_ssm_chunked(cudaStream_t s, const SsmParams& p, uint32_t T) {
  const uint32_t nchunks = (T + kQ - 1) / kQ;
  if (p.chunk_floats < ssm_chunk_floats(p.spec, T)) return cudaErrorInvalidValue;
  const SsmSpec& sp = p.spec;
  // 16-byte copies: every head's and group's columns start on a multiple of eight elements
  const int vec = sp.vdim % 8 == 0 && sp.state % 8 == 0;
  const size_t smem = state_smem(sp);
  cudaError_t e = cudaFuncSetAttribute(ssm_chunk_state_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e != cudaSuccess) return e;
  e = launch_pdl(ssm_chunk_state_kernel, dim3(nchunks, sp.heads), dim3(kThr), smem, s, prefill_pdl(), p, T, vec);
  if (e != cudaSuccess) return e;
  const size_t total = (size_t)sp.heads * sp.vdim * sp.state;
  e = launch_pdl(ssm_chunk_pass_kernel, dim3((unsigned)(((sp.vdim * sp.state % 4 ? total : total / 4) + 127) / 128)), dim3(128), 0, s, prefill_pdl(), p, nchunks);
  if (e != cudaSuccess) return e;
  switch (out_width(sp.vdim)) {
    case 32: return launch_out<32>(s, p, T, nchunks, vec);
    case 64: return launch_out<64>(s, p, T, nchunks, vec);
    case 128: return launch_out<128>(s, p, T, nchunks, vec);
    default: return cudaErrorInvalidValue;
  }
}

}  // namespace nfai
