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

// V consecutive elements as floats; p is aligned to V elements.
template <int V>
__device__ __forceinline__ void load_v(const float* p, float (&v)[V]) {
  if constexpr (V % 4 == 0) {
#pragma unroll
    for (int i = 0; i < V; i += 4) {
      const float4 u = *reinterpret_cast<const float4*>(p + i);
      v[i] = u.x; v[i + 1] = u.y; v[i + 2] = u.z; v[i + 3] = u.w;
    }
  } else {
#pragma unroll
    for (int i = 0; i < V; ++i) v[i] = p[i];
  }
}
template <int V>
__device__ __forceinline__ void store_v(float* p, const float (&v)[V]) {
  if constexpr (V % 4 == 0) {
#pragma unroll
    for (int i = 0; i < V; i += 4) *reinterpret_cast<float4*>(p + i) = make_float4(v[i], v[i + 1], v[i + 2], v[i + 3]);
  } else {
#pragma unroll
    for (int i = 0; i < V; ++i) p[i] = v[i];
  }
}
template <int V>
__device__ __forceinline__ void load_v(const __nv_bfloat16* p, float (&v)[V]) {
  if constexpr (V == 8) {
    const uint4 u = *reinterpret_cast<const uint4*>(p);
    v[0] = bf16_lo(u.x); v[1] = bf16_hi(u.x); v[2] = bf16_lo(u.y); v[3] = bf16_hi(u.y);
    v[4] = bf16_lo(u.z); v[5] = bf16_hi(u.z); v[6] = bf16_lo(u.w); v[7] = bf16_hi(u.w);
  } else if constexpr (V == 4) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    v[0] = bf16_lo(u.x); v[1] = bf16_hi(u.x); v[2] = bf16_lo(u.y); v[3] = bf16_hi(u.y);
  } else {
#pragma unroll
    for (int i = 0; i < V; ++i) v[i] = __bfloat162float(p[i]);
  }
}
template <int V>
__device__ __forceinline__ void store_v(__nv_bfloat16* p, const float (&v)[V]) {
  if constexpr (V == 8) {
    *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]), pack_bf16(v[4], v[5]), pack_bf16(v[6], v[7]));
  } else if constexpr (V == 4) {
    *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]));
  } else {
#pragma unroll
    for (int i = 0; i < V; ++i) p[i] = __float2bfloat16(v[i]);
  }
}

// The same functions for kernels that only bf16 models run: hardware exponential and division (relative error of a few
// units in the last place), which is far below the rounding of their bf16 inputs and outputs. quick_expm1 keeps its relative
// accuracy near zero (Taylor series there), as the decays of a recurrence need it.
constexpr float LOG2_E = 1.4426950408889634f;
__device__ __forceinline__ float quick_exp2(float z) {
  float r;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(z));
  return r;
}
__device__ __forceinline__ float quick_log2(float z) {
  float r;
  asm("lg2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(z));
  return r;
}
__device__ __forceinline__ float quick_rcp(float z) {
  float r;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(z));
  return r;
}
__device__ __forceinline__ float quick_exp(float z) { return quick_exp2(z * LOG2_E); }
__device__ __forceinline__ float quick_sigmoid(float z) { return quick_rcp(1.f + quick_exp(-z)); }
// log2(1 - k) for 0 <= k < 1, f = 1 - k: relative accuracy near k = 0 by -2 atanh(k / (2 - k)), whose series is short there
__device__ __forceinline__ float quick_log2_decay(float k, float f) {
  const float s = k * quick_rcp(2.f - k), s2 = s * s;
  const float series = s * fmaf(s2, fmaf(s2, fmaf(s2, fmaf(s2, 1.f / 9.f, 1.f / 7.f), 0.2f), 1.f / 3.f), 1.f);
  return k < 0.5f ? -2.f * LOG2_E * series : quick_log2(fmaxf(f, 1e-30f));
}
__device__ __forceinline__ float quick_expm1(float z) {
  const float t = z * fmaf(z, fmaf(z, fmaf(z, fmaf(z, fmaf(z, fmaf(z, 1.f / 5040.f, 1.f / 720.f), 1.f / 120.f), 1.f / 24.f), 1.f / 6.f), 0.5f), 1.f);
  return fabsf(z) < 0.3f ? t : quick_exp(z) - 1.f;
}
__device__ __forceinline__ float quick_sqrt(float z) {
  float r;
  asm("sqrt.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(z));
  return r;
}
__device__ __forceinline__ float quick_gelu_tanh(float z) {
  // 0.5 z (1 + tanh(y)) = z sigmoid(2 y)
  return z * quick_sigmoid(1.5957691216057308f * (z + 0.044715f * z * z * z));
}

// First visible position of a query at position i: a sliding window of `window` keys and / or chunks of `chunk` positions
// counted from the start of the sequence (<= 0: none).
__device__ __forceinline__ int first_visible(int i, int window, int chunk) {
  const int w = window > 0 ? max(0, i - window + 1) : 0;
  return chunk > 0 ? max(w, i - i % chunk) : w;
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
