// Fused epilogues of the prompt GEMMs (gemm_tc.cu, gemm_simt.cu): what happens to two adjacent output columns.
#pragma once
#include "common.cuh"
#include "gemm_tc.h"

namespace nfai {

// element `at` of the epilogue's activation output, in its type
__device__ __forceinline__ void store_operand(const GemmEpilogue& ep, size_t at, float v) {
  if (ep.out_dtype == 1) store_as(reinterpret_cast<__half*>(ep.out_act) + at, v);
  else if (ep.out_dtype == 2) store_as(reinterpret_cast<__nv_bfloat16*>(ep.out_act) + at, v);
  else reinterpret_cast<float*>(ep.out_act)[at] = v;
}

// ---- epilogues: two adjacent output columns (n, n+1) of row m; n is even -----------------------------------------
// What the epilogue of a pair reads from memory: the residual pair of a plain store, the (cos, sin) of a rotated Q/K
// pair. The callers fetch it for a whole block of pairs before they touch the accumulators: a loop of load -> add ->
// store per pair runs at one memory round trip per pair (the store may alias the next load as far as the compiler
// knows), which cost more than the tile's MMAs.
// KIND >= 0 fixes the epilogue at compile time (the persistent kernel dispatches once per tile); -1 reads ep.kind.
template <int KIND = -1>
__device__ __forceinline__ float2 epilogue_aux(const GemmEpilogue& ep, uint32_t m, uint32_t n, uint32_t N) {
  switch (KIND >= 0 ? KIND : (int)ep.kind) {
    case GEMM_EPI_STORE: {
      float2 r = make_float2(0.f, 0.f);
      if (ep.resid) {
        const float* res = ep.resid + (size_t)m * N;
        if ((N & 1u) == 0) r = __ldcg(reinterpret_cast<const float2*>(res + n));
        else r = make_float2(__ldcg(res + n), n + 1 < N ? __ldcg(res + n + 1) : 0.f);
      }
      if (ep.bias) {
        r.x += __ldg(ep.bias + n);
        if (n + 1 < N) r.y += __ldg(ep.bias + n + 1);
      }
      return r;
    }
    case GEMM_EPI_GATED:
    case GEMM_EPI_STORE_ACT:
      if (ep.bias) return make_float2(__ldg(ep.bias + n), n + 1 < N ? __ldg(ep.bias + n + 1) : 0.f);
      break;
    case GEMM_EPI_QKV_ROPE: {
      if (n < ep.qDim + ep.kvDim) {
        const uint32_t local = n < ep.qDim ? n : n - ep.qDim;
        const uint32_t e = local % ep.d;
        if (e < ep.ropeDim) return ep.rope_cs[(size_t)(ep.pos0 + m) * (ep.ropeDim / 2) + (e >> 1)];
      }
      break;
    }
    default: break;
  }
  return make_float2(0.f, 0.f);
}

template <int KIND = -1>
__device__ __forceinline__ void epilogue_pair(const GemmEpilogue& ep, uint32_t m, uint32_t n, uint32_t N, float a, float b,
                                              const float2 aux) {
  switch (KIND >= 0 ? KIND : (int)ep.kind) {
    case GEMM_EPI_STORE: {
      float* out = ep.out_f32 + (size_t)m * N;
      if ((N & 1u) == 0) {  // rows start on an 8-byte boundary: one store per pair
        *reinterpret_cast<float2*>(out + n) = make_float2(aux.x + a, aux.y + b);
      } else {
        out[n] = aux.x + a;
        if (n + 1 < N) out[n + 1] = aux.y + b;
      }
      break;
    }
    case GEMM_EPI_GATED: {  // columns (2j, 2j+1) = (gate_j, up_j); h_j = up * act(gate)
      if (n + 1 < N) store_operand(ep, (size_t)m * (N / 2) + (n >> 1), gated(ep.act, a + aux.x, b + aux.y));
      break;
    }
    case GEMM_EPI_GATED_CLAMPED: {
      const uint32_t cols = ep.gated_cols ? ep.gated_cols : N;
      if (n < cols) store_operand(ep, (size_t)m * (cols / 2) + (n >> 1), gated_clamped(a, b, ep.act_limit));
      else *reinterpret_cast<float2*>(ep.out_f32 + (size_t)m * (N - cols) + (n - cols)) = make_float2(a, b);
      break;
    }
    case GEMM_EPI_STORE_ACT: {  // plain store in the operand type of the next product
      const size_t at = (size_t)m * N + n;
      if ((N & 1u) == 0 && ep.out_dtype == 2) {
        *reinterpret_cast<__nv_bfloat162*>(reinterpret_cast<__nv_bfloat16*>(ep.out_act) + at) =
            __floats2bfloat162_rn(a + aux.x, b + aux.y);
      } else {
        store_operand(ep, at, a + aux.x);
        if (n + 1 < N) store_operand(ep, at + 1, b + aux.y);
      }
      break;
    }
    case GEMM_EPI_QKV_ROPE: {  // columns [Q | K | V]; RoPE on adjacent pairs at position pos0 + m
      const uint32_t pos = ep.pos0 + m;
      if (n < ep.qDim + ep.kvDim) {
        const uint32_t local = n < ep.qDim ? n : n - ep.qDim;
        const uint32_t e = local % ep.d;
        if (e < ep.ropeDim) {
          const float2 cs = aux;
          const float v1 = __fsub_rn(__fmul_rn(cs.x, a), __fmul_rn(cs.y, b));
          const float v2 = __fadd_rn(__fmul_rn(cs.y, a), __fmul_rn(cs.x, b));
          a = v1;
          b = v2;
        }
        if (n < ep.qDim) {
          // (n, local and the row lengths are even: pairs are naturally aligned)
          *reinterpret_cast<float2*>(ep.out_f32 + (size_t)m * ep.qDim + n) = make_float2(a, b);
        } else if (ep.kv_f16) {
          __half* kc = reinterpret_cast<__half*>(ep.kcache) + (size_t)pos * ep.kvDim + local;
          *reinterpret_cast<__half2*>(kc) = __floats2half2_rn(a, b);
        } else {
          float* kc = reinterpret_cast<float*>(ep.kcache) + (size_t)pos * ep.kvDim + local;
          kc[0] = a;
          kc[1] = b;
        }
      } else {
        const uint32_t local = n - ep.qDim - ep.kvDim;
        if (ep.kv_f16) {
          __half* vc = reinterpret_cast<__half*>(ep.vcache) + (size_t)pos * ep.kvDim + local;
          *reinterpret_cast<__half2*>(vc) = __floats2half2_rn(a, b);
        } else {
          float* vc = reinterpret_cast<float*>(ep.vcache) + (size_t)pos * ep.kvDim + local;
          vc[0] = a;
          vc[1] = b;
        }
      }
      break;
    }
  }
}

}  // namespace nfai
