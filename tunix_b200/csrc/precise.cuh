// Scalar helpers of the kernels that serve both bf16 and 32-bit models. Files that include this header are compiled
// without fast-math (see _build.py): their 32-bit results must hold to rounding.
#pragma once
#include "common.cuh"

namespace tb {

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T>
__device__ __forceinline__ T from_f(float v);
template <>
__device__ __forceinline__ float from_f<float>(float v) { return v; }
template <>
__device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16(v); }

__device__ __forceinline__ float sigmoid(float z) { return 1.f / (1.f + expf(-z)); }
// e^z for z <= 0 that is raised to high powers by a recurrence: near 1 the error of expf (up to one unit in the last place,
// always to the same side for a slowly varying z) would add up over a thousand steps, so the sum is rounded once.
__device__ __forceinline__ float decay_exp(float z) { return z > -0.6f ? 1.f + expm1f(z) : expf(z); }
// log(1 + e^z), without overflow
__device__ __forceinline__ float softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float log_sigmoid(float z) { return -softplus(-z); }
__device__ __forceinline__ float gelu_tanh(float z) {
  return 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}

// A ragged batch: entry e holds tokens cu[e] .. cu[e+1]-1 of the flat token list, which continue the sequence in slot
// slot[e] at position pos0[e] (negative: an idle slot, nothing is read or written for it).
struct Ragged {
  const int* cu;      // [E + 1]
  const int* slot;    // [E]
  const int* pos0;    // [E]
  const int* ent;     // [n] entry of every token
  int E, n;
};

}  // namespace tb
