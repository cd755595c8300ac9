// Single-query attention over paged keys whose context is split over CTAs: which tiles of keys a query walks, what the heads add
// to the sum of their weights and to their output, and the kernel that merges the splits.
#pragma once
#include "common.cuh"

namespace tb {

constexpr int TILE_KEYS = 64;   // keys staged per pipeline stage

// A sink is one more score without a value in the sum of a head's weights (-inf: none); gates are rows of logits, one per head.
struct HeadExtras {
  float sink;
  const float* sinks;           // [N] or null: a sink per head instead
  const __nv_bfloat16* gate;    // rows ldg apart, or null
  long long ldg;
  __device__ __forceinline__ float sink_of(int n) const { return sinks ? sinks[n] : sink; }
  __device__ __forceinline__ float gate_of(long long row, int n) const {
    return gate ? 1.f / (1.f + __expf(-__bfloat162float(gate[row * ldg + n]))) : 1.f;
  }
};

// The key tiles a single query at position len - 1 walks: the tiles that hold kept first tokens, then those of the window.
struct KeyTiles {
  int w_lo, first, n_sink, total;
  __device__ __forceinline__ KeyTiles(int len, int window, int chunk, int keep) {
    w_lo = window > 0 ? max(0, len - window) : 0;
    if (chunk > 0 && len > 0) w_lo = max(w_lo, len - 1 - (len - 1) % chunk);
    first = w_lo / TILE_KEYS;
    n_sink = min((min(keep, len) + TILE_KEYS - 1) / TILE_KEYS, first);
    total = n_sink + (len + TILE_KEYS - 1) / TILE_KEYS - first;
  }
  __device__ __forceinline__ int start(int tile) const { return (tile < n_sink ? tile : first + tile - n_sink) * TILE_KEYS; }
};

// out[b, n, :vd] = out_scale * sum_s acc_s * exp(m_s - M) / (exp(sink - M) + sum_s l_s * exp(m_s - M))
static __global__ void paged_decode_combine_kernel(const float* __restrict__ part_acc, const float* __restrict__ part_ml,
                                            const int* __restrict__ seq_lens, int N, int H, int num_splits, int split_tokens,
                                            int window, int chunk, int keep, float out_scale, int vd, const HeadExtras ex,
                                            __nv_bfloat16* __restrict__ out, long long ldo) {
  pdl_trigger();
  pdl_wait();
  const int b = blockIdx.x, n = blockIdx.y;
  const int len = seq_lens[b];
  const int tps = split_tokens / TILE_KEYS;
  const int used = len > 0 ? min(num_splits, (KeyTiles(len, window, chunk, keep).total + tps - 1) / tps) : 0;
  const long long base = ((long long)b * N + n) * num_splits;
  float M = -INFINITY;
  for (int s = 0; s < used; ++s) M = fmaxf(M, part_ml[(base + s) * 2]);
  float L = used > 0 ? __expf(ex.sink_of(n) - M) : 0.f;
  for (int s = 0; s < used; ++s) {
    const float ms = part_ml[(base + s) * 2];
    if (ms != -INFINITY) L += part_ml[(base + s) * 2 + 1] * __expf(ms - M);
  }
  const float inv = L > 0.f ? out_scale * ex.gate_of(b, n) / L : 0.f;
  __nv_bfloat16* to = out + (long long)b * ldo + (long long)n * vd;
  for (int d = threadIdx.x * 4; d < vd; d += blockDim.x * 4) {          // H is a multiple of 4
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int s = 0; s < used; ++s) {
      const float ms = part_ml[(base + s) * 2];
      if (ms == -INFINITY) continue;
      const float w = __expf(ms - M) * inv;
      const float4 v = *reinterpret_cast<const float4*>(part_acc + (base + s) * H + d);
      a.x += v.x * w; a.y += v.y * w; a.z += v.z * w; a.w += v.w * w;
    }
    if (d + 4 <= vd && (((uintptr_t)to) & 7) == 0) {
      *reinterpret_cast<uint2*>(to + d) = make_uint2(pack_bf16(a.x, a.y), pack_bf16(a.z, a.w));
    } else {
      const float v[4] = {a.x, a.y, a.z, a.w};
      for (int k = 0; k < 4 && d + k < vd; ++k) to[d + k] = __float2bfloat16(v[k]);
    }
  }
}

}  // namespace tb
