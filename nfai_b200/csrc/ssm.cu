// Selective state space layers (Mamba-2 form): per head h with a scalar decay, state S [vdim][N] in float32,
//   dt = softplus(raw + bias),  S <- exp(-exp(A_log) dt) S + dt x B^T,  y = S C + D x,  then y silu(z).
// x, B and C come out of a causal convolution over the last `taps` projected rows. Those rows live in a ring indexed by
// position, which the projection writes directly; nothing is ever shifted, and position 0 starts from a zero state without
// anything having to be cleared (rows of negative positions are not read, the old state is ignored).
//
// Decode (ssm_step_kernel): a CTA owns 32 rows of one head's state. The state does not depend on the previous kernel of the
// step, so a warp has its rows in registers before the dependency wait; the kernel is one read and one write of the state.
#include "plan_kernels.h"
#include "common.cuh"

namespace nfai {

// ssm_chunk.cu
bool ssm_chunk_supported(const SsmSpec& s);
cudaError_t launch_ssm_chunked(cudaStream_t s, const SsmParams& p, uint32_t T);

namespace {

constexpr int kStepV = 32;  // state rows (values of one head) per CTA

__device__ __forceinline__ float softplus_f(float v) { return v > 20.f ? v : log1pf(expf(v)); }
__device__ __forceinline__ float silu_f(float v) { return v / (1.0f + expf(-v)); }

// One convolved channel at position pos, input rows from the ring
__device__ __forceinline__ float conv_ring(const SsmParams& p, uint32_t pos, uint32_t ch) {
  const uint32_t K = p.spec.taps, ld = p.spec.in_rows();
  const float* col = p.ring + p.spec.inner() + ch;
  float a = p.conv_b[ch];
  uint32_t slot = (pos + 1) % K;  // row of the oldest tap's position
  for (uint32_t j0 = 0; j0 < K; j0 += 4) {  // four taps' loads in flight together
    float v[4], w[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const uint32_t j = j0 + i;
      const bool in = j < K && K - 1 - j <= pos;
      v[i] = in ? __ldcg(col + (size_t)slot * ld) : 0.f;
      w[i] = in ? p.conv_w[ch * K + j] : 0.f;
      slot = slot + 1 == K ? 0 : slot + 1;
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) a = fmaf(w[i], v[i], a);
  }
  return silu_f(a);
}

// NJ state columns per lane (32 NJ >= N); NJ = 0: any N, nothing held in registers
template <int NJ>
__global__ void __launch_bounds__(256) ssm_step_kernel(const SsmParams p) {
  extern __shared__ float ssm_sm[];
  const SsmSpec& sp = p.spec;
  const uint32_t N = sp.state, V = sp.vdim, h = blockIdx.x, v0 = blockIdx.y * kStepV;
  float* Bs = ssm_sm;
  float* Cs = Bs + N;
  float* xs = Cs + N;  // [kStepV]
  float* sc = xs + kStepV;  // decay, dt
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  constexpr int VR = kStepV / 8;  // rows per warp
  const uint32_t pos = p.state ? p.state->pos : p.pos0;
  float st[VR][NJ > 0 ? NJ : 1];
  float* const Sh = p.S + (size_t)h * V * N;
  if constexpr (NJ > 0) {
#pragma unroll
    for (int r = 0; r < VR; ++r) {
      const uint32_t v = v0 + warp * VR + r;
#pragma unroll
      for (int j = 0; j < NJ; ++j) {
        const uint32_t n = lane + 32 * j;
        st[r][j] = pos > 0 && v < V && n < N ? Sh[(size_t)v * N + n] : 0.f;
      }
    }
  }
  pdl_launch_dependents();
  pdl_wait();
  const uint32_t g = h / (sp.heads / sp.groups), inner = sp.inner();
  const float* row = p.ring + (size_t)(pos % sp.taps) * sp.in_rows();
  for (uint32_t i = threadIdx.x; i < 2 * N + kStepV; i += 256) {
    if (i < N) Bs[i] = conv_ring(p, pos, inner + g * N + i);
    else if (i < 2 * N) Cs[i - N] = conv_ring(p, pos, inner + sp.groups * N + g * N + i - N);
    else if (v0 + i - 2 * N < V) xs[i - 2 * N] = conv_ring(p, pos, h * V + v0 + i - 2 * N);
  }
  if (threadIdx.x == 0) {
    const float dt = softplus_f(__ldcg(row + inner + sp.channels() + h) + p.dt_bias[h]);
    sc[0] = expf(-expf(p.A_log[h]) * dt);
    sc[1] = dt;
  }
  __syncthreads();
  const float decay = sc[0], dt = sc[1], D = p.D[h];
#pragma unroll
  for (int r = 0; r < VR; ++r) {
    const uint32_t v = v0 + warp * VR + r;
    if (v >= V) break;  // uniform in the warp
    const float x = xs[warp * VR + r], dx = dt * x;
    float acc = 0.f;
    if constexpr (NJ > 0) {
#pragma unroll
      for (int j = 0; j < NJ; ++j) {
        const uint32_t n = lane + 32 * j;
        if (n < N) {
          const float s = fmaf(decay, st[r][j], dx * Bs[n]);
          Sh[(size_t)v * N + n] = s;
          acc = fmaf(s, Cs[n], acc);
        }
      }
    } else {
      for (uint32_t n = lane; n < N; n += 32) {
        const float s = fmaf(decay, pos > 0 ? Sh[(size_t)v * N + n] : 0.f, dx * Bs[n]);
        Sh[(size_t)v * N + n] = s;
        acc = fmaf(s, Cs[n], acc);
      }
    }
    acc = warp_sum(acc);
    if (lane == 0) p.y[h * V + v] = fmaf(D, x, acc) * silu_f(__ldcg(row + h * V + v));
  }
}

// ---- prompt path ------------------------------------------------------------------------------------------------------
// One channel per thread over kConvTB tokens. KT taps known at compile time: the inputs are requested together.
constexpr uint32_t kConvTB = 16;
template <typename XT, int KT>
__global__ void __launch_bounds__(256) ssm_conv_kernel(const SsmParams p, uint32_t T) {
  const SsmSpec& sp = p.spec;
  const uint32_t ch = blockIdx.x * 256 + threadIdx.x, CH = sp.channels(), ld = sp.in_rows(), K = KT ? KT : sp.taps, inner = sp.inner();
  pdl_launch_dependents();
  pdl_wait();
  if (ch >= CH + sp.heads) return;
  const uint32_t t0 = blockIdx.y * kConvTB, t1 = min(T, t0 + kConvTB);
  if (ch >= CH) {
    const uint32_t h = ch - CH;
    for (uint32_t t = t0; t < t1; ++t) p.dt[(size_t)t * sp.heads + h] = softplus_f(p.in[(size_t)t * ld + inner + ch] + p.dt_bias[h]);
    return;
  }
  XT* out = reinterpret_cast<XT*>(p.xbc) + ch;
  const float* in = p.in + inner + ch;
  const float b = p.conv_b[ch];
  auto past = [&](uint32_t t, uint32_t back) -> float {  // input `back` tokens before token t of the portion
    if (back <= t) return in[(size_t)(t - back) * ld];
    if (back <= p.pos0 + t) return p.ring[(size_t)((p.pos0 + t - back) % K) * ld + inner + ch];
    return 0.f;
  };
  if constexpr (KT > 0) {
    float v[kConvTB + KT - 1], w[KT];
#pragma unroll
    for (int j = 0; j < KT; ++j) w[j] = p.conv_w[ch * KT + j];
#pragma unroll
    for (int j = 0; j < KT - 1; ++j) v[j] = past(t0, KT - 1 - j);
#pragma unroll
    for (uint32_t i = 0; i < kConvTB; ++i) v[KT - 1 + i] = t0 + i < T ? in[(size_t)(t0 + i) * ld] : 0.f;
#pragma unroll
    for (uint32_t i = 0; i < kConvTB; ++i) {
      float a = b;
#pragma unroll
      for (int j = 0; j < KT; ++j) a = fmaf(w[j], v[i + j], a);
      if (t0 + i < T) store_as(out + (size_t)(t0 + i) * CH, silu_f(a));
    }
  } else {
    for (uint32_t t = t0; t < t1; ++t) {
      float a = b;
      for (uint32_t j = 0; j < K; ++j) a = fmaf(p.conv_w[ch * K + j], past(t, K - 1 - j), a);
      store_as(out + (size_t)t * CH, silu_f(a));
    }
  }
}

template <typename XT>
cudaError_t launch_conv(cudaStream_t s, const SsmParams& p, uint32_t T) {
  const dim3 grid((p.spec.channels() + p.spec.heads + 255) / 256, (T + kConvTB - 1) / kConvTB);
  auto kern = p.spec.taps == 2 ? ssm_conv_kernel<XT, 2> : p.spec.taps == 3 ? ssm_conv_kernel<XT, 3> : p.spec.taps == 4 ? ssm_conv_kernel<XT, 4>
              : ssm_conv_kernel<XT, 0>;
  return launch_pdl(kern, grid, dim3(256), 0, s, prefill_pdl(), p, T);
}

// the last rows of the portion into the ring, where decoding would have put them
__global__ void __launch_bounds__(256) ssm_ring_kernel(const SsmParams p, uint32_t T) {
  pdl_launch_dependents();
  pdl_wait();
  const uint32_t ld = p.spec.in_rows(), K = p.spec.taps, n = min(T, K), t = T - 1 - blockIdx.y;
  if (blockIdx.y >= n) return;
  const uint32_t c = blockIdx.x * 256 + threadIdx.x;
  if (c < ld) p.ring[(size_t)((p.pos0 + t) % K) * ld + c] = p.in[(size_t)t * ld + c];
}

// The recurrence token by token: 32 values of one head per CTA, eight lanes share the N columns of one value's state row.
// NJ columns per lane in registers (8 NJ >= N); NJ = 0: any N, the state stays in memory.
constexpr int kScanTB = 16;
template <typename XT, int NJ>
__global__ void __launch_bounds__(256) ssm_scan_kernel(const SsmParams p, uint32_t T) {
  extern __shared__ float scan_sm[];
  const SsmSpec& sp = p.spec;
  const uint32_t N = sp.state, V = sp.vdim, h = blockIdx.x, v0 = blockIdx.y * 32, CH = sp.channels(), inner = sp.inner();
  const uint32_t g = h / (sp.heads / sp.groups);
  float* Bs = scan_sm;                 // [TB][N]
  float* Cs = Bs + kScanTB * N;        // [TB][N]
  float* xs = Cs + kScanTB * N;        // [TB][32]
  float* ds = xs + kScanTB * 32;       // [TB] decay, [TB] dt
  const uint32_t vi = threadIdx.x >> 3, ln = threadIdx.x & 7, v = v0 + vi;
  const bool live = v < V;
  pdl_launch_dependents();
  pdl_wait();
  const XT* xbc = reinterpret_cast<const XT*>(p.xbc);
  float* Sv = p.S + ((size_t)h * V + (live ? v : 0)) * N;
  float st[NJ > 0 ? NJ : 1];
  if constexpr (NJ > 0) {
#pragma unroll
    for (int j = 0; j < NJ; ++j) st[j] = live && p.pos0 > 0 && ln + 8 * j < N ? Sv[ln + 8 * j] : 0.f;
  } else if (live && p.pos0 == 0) {
    for (uint32_t n = ln; n < N; n += 8) Sv[n] = 0.f;
  }
  const float A = -expf(p.A_log[h]), D = p.D[h];
  for (uint32_t t0 = 0; t0 < T; t0 += kScanTB) {
    const uint32_t nt = min((uint32_t)kScanTB, T - t0);
    __syncthreads();
    for (uint32_t i = threadIdx.x; i < nt * N; i += 256) {
      const uint32_t t = i / N, n = i - t * N;
      const XT* r = xbc + (size_t)(t0 + t) * CH + inner + g * N + n;
      Bs[i] = to_float(r[0]);
      Cs[i] = to_float(r[sp.groups * N]);
    }
    for (uint32_t i = threadIdx.x; i < nt * 32; i += 256) {
      const uint32_t t = i >> 5, vv = v0 + (i & 31);
      xs[i] = vv < V ? to_float(xbc[(size_t)(t0 + t) * CH + h * V + vv]) : 0.f;
    }
    if (threadIdx.x < nt) {
      const float dt = p.dt[(size_t)(t0 + threadIdx.x) * sp.heads + h];
      ds[threadIdx.x] = expf(A * dt);
      ds[kScanTB + threadIdx.x] = dt;
    }
    __syncthreads();
    for (uint32_t t = 0; t < nt; ++t) {
      const float decay = ds[t], x = xs[t * 32 + vi], dx = ds[kScanTB + t] * x;
      float acc = 0.f;
      if constexpr (NJ > 0) {
#pragma unroll
        for (int j = 0; j < NJ; ++j) {
          const uint32_t n = ln + 8 * j;
          if (n < N) {
            st[j] = fmaf(decay, st[j], dx * Bs[t * N + n]);
            acc = fmaf(st[j], Cs[t * N + n], acc);
          }
        }
      } else if (live) {
        for (uint32_t n = ln; n < N; n += 8) {
          const float s = fmaf(decay, Sv[n], dx * Bs[t * N + n]);
          Sv[n] = s;
          acc = fmaf(s, Cs[t * N + n], acc);
        }
      }
      acc += __shfl_xor_sync(0xffffffffu, acc, 1);
      acc += __shfl_xor_sync(0xffffffffu, acc, 2);
      acc += __shfl_xor_sync(0xffffffffu, acc, 4);
      if (ln == 0 && live) {
        const float z = p.in[(size_t)(t0 + t) * sp.in_rows() + h * V + v];
        p.y[(size_t)(t0 + t) * inner + h * V + v] = fmaf(D, x, acc) * silu_f(z);
      }
    }
  }
  if constexpr (NJ > 0) {
#pragma unroll
    for (int j = 0; j < NJ; ++j)
      if (live && ln + 8 * j < N) Sv[ln + 8 * j] = st[j];
  }
}

// A warp per (token, part). NQ > 0: parts of up to 128 NQ values in quads, kept in registers between the two passes.
template <typename OT, int NQ>
__global__ void __launch_bounds__(256) group_norm_rows_kernel(const float* __restrict__ y, const float* __restrict__ gain, float eps,
                                                              uint32_t groups, uint32_t T, uint32_t K, OT* __restrict__ out) {
  pdl_launch_dependents();
  pdl_wait();
  const uint32_t part = K / groups, lane = threadIdx.x & 31;
  const size_t item = (size_t)blockIdx.x * 8 + (threadIdx.x >> 5);
  if (item >= (size_t)T * groups) return;
  const uint32_t g = (uint32_t)(item % groups);
  const float* yr = y + item * part;
  const float* gr = gain + (size_t)g * part;
  OT* o = out + item * part;
  float ss = 0.f;
  if constexpr (NQ > 0) {
    float4 v[NQ];
#pragma unroll
    for (int i = 0; i < NQ; ++i) {
      const uint32_t at = (lane + 32 * i) * 4;
      v[i] = at < part ? *reinterpret_cast<const float4*>(yr + at) : make_float4(0.f, 0.f, 0.f, 0.f);
      ss = fmaf(v[i].x, v[i].x, ss);
      ss = fmaf(v[i].y, v[i].y, ss);
      ss = fmaf(v[i].z, v[i].z, ss);
      ss = fmaf(v[i].w, v[i].w, ss);
    }
    const float rms = sqrtf(__fdiv_rn(warp_sum(ss), (float)part) + eps);
#pragma unroll
    for (int i = 0; i < NQ; ++i) {
      const uint32_t at = (lane + 32 * i) * 4;
      if (at < part) {
        const float4 w = *reinterpret_cast<const float4*>(gr + at);
        const float r[4] = {__fmul_rn(__fdiv_rn(v[i].x, rms), w.x), __fmul_rn(__fdiv_rn(v[i].y, rms), w.y),
                            __fmul_rn(__fdiv_rn(v[i].z, rms), w.z), __fmul_rn(__fdiv_rn(v[i].w, rms), w.w)};
        if constexpr (sizeof(OT) == 2) {
          __nv_bfloat162 b[2] = {__floats2bfloat162_rn(r[0], r[1]), __floats2bfloat162_rn(r[2], r[3])};
          *reinterpret_cast<uint2*>(o + at) = *reinterpret_cast<uint2*>(b);
        } else {
          *reinterpret_cast<float4*>(o + at) = make_float4(r[0], r[1], r[2], r[3]);
        }
      }
    }
  } else {
    for (uint32_t i = lane; i < part; i += 32) ss = fmaf(yr[i], yr[i], ss);
    const float rms = sqrtf(__fdiv_rn(warp_sum(ss), (float)part) + eps);
    for (uint32_t i = lane; i < part; i += 32) store_as(o + i, __fmul_rn(__fdiv_rn(yr[i], rms), gr[i]));
  }
}

template <typename OT>
cudaError_t launch_norm(cudaStream_t s, const float* y, const float* gain, float eps, uint32_t groups, uint32_t T, uint32_t K, OT* out) {
  const uint32_t part = K / groups;
  auto kern = part % 4 || part > 1024 ? group_norm_rows_kernel<OT, 0> : part <= 512 ? group_norm_rows_kernel<OT, 4> : group_norm_rows_kernel<OT, 8>;
  return launch_pdl(kern, dim3((unsigned)(((size_t)T * groups + 7) / 8)), dim3(256), 0, s, prefill_pdl(), y, gain, eps, groups, T, K, out);
}

template <typename XT>
cudaError_t launch_scan(cudaStream_t s, const SsmParams& p, uint32_t T) {
  const uint32_t N = p.spec.state;
  const size_t smem = ((size_t)kScanTB * (2 * N + 32) + 2 * kScanTB) * 4;
  if (smem > 227 * 1024) return cudaErrorInvalidValue;
  auto kern = N <= 32 ? ssm_scan_kernel<XT, 4> : N <= 64 ? ssm_scan_kernel<XT, 8> : N <= 128 ? ssm_scan_kernel<XT, 16>
              : N <= 256 ? ssm_scan_kernel<XT, 32> : ssm_scan_kernel<XT, 0>;
  if (smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return e;
  }
  return launch_pdl(kern, dim3(p.spec.heads, (p.spec.vdim + 31) / 32), dim3(256), smem, s, prefill_pdl(), p, T);
}

}  // namespace

cudaError_t launch_ssm_step(cudaStream_t s, const SsmParams& p, bool pdl) {
  const uint32_t N = p.spec.state;
  const size_t smem = ((size_t)2 * N + kStepV + 2) * 4;
  if (smem > 48 * 1024) return cudaErrorInvalidValue;
  auto kern = N <= 64 ? ssm_step_kernel<2> : N <= 128 ? ssm_step_kernel<4> : N <= 256 ? ssm_step_kernel<8> : ssm_step_kernel<0>;
  return launch_pdl(kern, dim3(p.spec.heads, (p.spec.vdim + kStepV - 1) / kStepV), dim3(256), smem, s, pdl, p);
}

cudaError_t launch_ssm_prefill(cudaStream_t s, const SsmParams& p, uint32_t T) {
  if (!T) return cudaErrorInvalidValue;
  cudaError_t e = p.xbc_dtype == 2 ? launch_conv<__nv_bfloat16>(s, p, T) : launch_conv<float>(s, p, T);
  if (e != cudaSuccess) return e;
  const uint32_t n = T < p.spec.taps ? T : p.spec.taps;
  e = launch_pdl(ssm_ring_kernel, dim3((p.spec.in_rows() + 255) / 256, n), dim3(256), 0, s, prefill_pdl(), p, T);
  if (e != cudaSuccess) return e;
  // portions long enough to fill the tensor cores' tiles: chunk by chunk (NFAI_SSM_CHUNK=0 keeps the token-by-token scan)
  static const bool chunked = env_int("NFAI_SSM_CHUNK", 1) != 0;
  if (p.xbc_dtype == 2 && chunked && T >= 32 && p.chunk && ssm_chunk_supported(p.spec)) return launch_ssm_chunked(s, p, T);
  return p.xbc_dtype == 2 ? launch_scan<__nv_bfloat16>(s, p, T) : launch_scan<float>(s, p, T);
}

cudaError_t launch_group_norm_rows(cudaStream_t s, const float* y, const float* gain, float eps, uint32_t groups, uint32_t T,
                                   uint32_t K, void* out, int out_dtype) {
  if (!groups || K % groups || !T) return cudaErrorInvalidValue;
  if (out_dtype == 2) return launch_norm(s, y, gain, eps, groups, T, K, (__nv_bfloat16*)out);
  if (out_dtype == 0) return launch_norm(s, y, gain, eps, groups, T, K, (float*)out);
  return cudaErrorInvalidValue;
}

}  // namespace nfai
