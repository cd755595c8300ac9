// Kernels around the sublayers of layer-stack models (models/stack.py): parallel residual streams with their
// hyper-connection matrices, the norms at their ends, gated activations for any width. The streams and everything
// computed on them are fp32; T is the activation type of the model (bf16 or float).
//
//   stream_step : one launch between two sublayers. It closes the sublayer before it (streams <- mix^T streams +
//                 out * y) and opens the one after it (u = in . streams, h = RMS norm(u) * w), so that the streams are
//                 read and written once per sublayer. y is one tensor, or half the sum of two tensors that are
//                 RMS-normed first (two mixers side by side). The first launch of a forward pass takes the embedding
//                 rows instead of streams, the last one has no successor but the final norm.
//
// This file is compiled without fast-math: the same kernels serve the 32-bit mode.
#include "precise.cuh"

using namespace tb;

namespace {

constexpr int MAX_STREAMS = 8;

struct StreamArgs {
  float* x;                   // [n, S, D]
  int D;
  float eps;
  // the sublayer that just ended
  const void* y;              // T [n, D] or null
  const void* y2;             // T [n, D] or null: y and y2 are normed, weighted and averaged
  const void* wy;             // T [D]
  const void* wy2;            // T [D]
  const void* mix;            // T [S, S], row = from, column = to
  const void* out;            // T [S]
  // the start of a forward pass (instead of the above)
  const long long* tokens;    // [n] or null
  const void* embed;          // T [V, D]
  int vocab;
  // the sublayer that follows
  const void* in;             // T [S]; null = all ones (the sum of the streams)
  const void* w;              // T [D] norm weight
  void* h;                    // T [n, D]
  float* sum_out;             // fp32 [n, D] or null: the sum of the streams
};

// V elements of a row per thread and iteration (4, or 1 for widths that are no multiple of 4)
template <typename T, int S, int V>
__global__ void __launch_bounds__(512) stream_step_kernel(const StreamArgs a) {
  extern __shared__ float u_s[];          // [D]
  __shared__ float red[33];
  pdl_trigger();
  pdl_wait();
  const long long row = blockIdx.x;
  const int D = a.D, step = blockDim.x * V;
  float* x = a.x + row * S * D;
  float mix[S][S], outw[S], inw[S];
#pragma unroll
  for (int s = 0; s < S; ++s) {
    inw[s] = a.in ? to_f(static_cast<const T*>(a.in)[s]) : 1.f;
    outw[s] = a.y ? to_f(static_cast<const T*>(a.out)[s]) : 0.f;
#pragma unroll
    for (int t = 0; t < S; ++t) mix[s][t] = a.y ? to_f(static_cast<const T*>(a.mix)[s * S + t]) : 0.f;
  }
  const T* y = a.y ? static_cast<const T*>(a.y) + row * D : nullptr;
  const T* y2 = a.y2 ? static_cast<const T*>(a.y2) + row * D : nullptr;
  float r1 = 1.f, r2 = 0.f;
  if (y2) {
    float s1 = 0.f, s2 = 0.f;
    for (int d = threadIdx.x * V; d < D; d += step) {
      float v1[V], v2[V];
      load_v<V>(y + d, v1);
      load_v<V>(y2 + d, v2);
#pragma unroll
      for (int i = 0; i < V; ++i) { s1 += v1[i] * v1[i]; s2 += v2[i] * v2[i]; }
    }
    s1 = block_sum(s1, red);
    s2 = block_sum(s2, red);
    r1 = 0.5f / sqrtf(s1 / (float)D + a.eps);
    r2 = 0.5f / sqrtf(s2 / (float)D + a.eps);
  }
  const T* emb = nullptr;
  if (a.tokens) {
    long long t = a.tokens[row];
    t = t < 0 ? 0 : (t >= a.vocab ? a.vocab - 1 : t);
    emb = static_cast<const T*>(a.embed) + t * D;
  }
  float ss = 0.f;
  for (int d = threadIdx.x * V; d < D; d += step) {
    float v[S][V];
    if (emb) {
      float ev[V];
      load_v<V>(emb + d, ev);
#pragma unroll
      for (int s = 0; s < S; ++s)
#pragma unroll
        for (int i = 0; i < V; ++i) v[s][i] = ev[i];
    } else {
      float o[S][V];
#pragma unroll
      for (int s = 0; s < S; ++s) load_v<V>(x + (long long)s * D + d, o[s]);
      if (y) {
        float yv[V];
        load_v<V>(y + d, yv);
        if (y2) {
          float v2[V], w1[V], w2[V];
          load_v<V>(y2 + d, v2);
          load_v<V>(static_cast<const T*>(a.wy) + d, w1);
          load_v<V>(static_cast<const T*>(a.wy2) + d, w2);
#pragma unroll
          for (int i = 0; i < V; ++i) yv[i] = yv[i] * r1 * w1[i] + v2[i] * r2 * w2[i];
        }
#pragma unroll
        for (int t = 0; t < S; ++t)
#pragma unroll
          for (int i = 0; i < V; ++i) {
            float acc = outw[t] * yv[i];
#pragma unroll
            for (int s = 0; s < S; ++s) acc += mix[s][t] * o[s][i];
            v[t][i] = acc;
          }
      } else {
#pragma unroll
        for (int t = 0; t < S; ++t)
#pragma unroll
          for (int i = 0; i < V; ++i) v[t][i] = o[t][i];
      }
    }
#pragma unroll
    for (int s = 0; s < S; ++s) store_v<V>(x + (long long)s * D + d, v[s]);
    float u[V], tot[V];
#pragma unroll
    for (int i = 0; i < V; ++i) {
      u[i] = tot[i] = 0.f;
#pragma unroll
      for (int s = 0; s < S; ++s) { u[i] += inw[s] * v[s][i]; tot[i] += v[s][i]; }
      ss += u[i] * u[i];
    }
    if (a.sum_out) store_v<V>(a.sum_out + row * D + d, tot);
    store_v<V>(u_s + d, u);
  }
  if (!a.h) return;
  ss = block_sum(ss, red);
  const float r = 1.f / sqrtf(ss / (float)D + a.eps);
  T* h = static_cast<T*>(a.h) + row * D;
  for (int d = threadIdx.x * V; d < D; d += step) {      // each thread reads back what it wrote
    float u[V], w[V];
    load_v<V>(u_s + d, u);
    load_v<V>(static_cast<const T*>(a.w) + d, w);
#pragma unroll
    for (int i = 0; i < V; ++i) u[i] = u[i] * r * w[i];
    store_v<V>(h + d, u);
  }
}

template <typename T, int S>
cudaError_t launch_stream_step(const StreamArgs& a, int n, cudaStream_t stream) {
  const bool vec = a.D % 4 == 0;
  const int per = vec ? a.D / 4 : a.D;
  int threads = n <= 296 ? 512 : 256;              // few rows: the latency of one row counts
  while (threads > 128 && threads / 2 >= per) threads /= 2;
  if (vec) return launch_pdl(stream_step_kernel<T, S, 4>, dim3(n), dim3(threads), (size_t)a.D * 4, stream, a);
  return launch_pdl(stream_step_kernel<T, S, 1>, dim3(n), dim3(threads), (size_t)a.D * 4, stream, a);
}

template <typename T>
int dispatch_stream_step(const StreamArgs& a, int S, int n, cudaStream_t stream) {
  cudaError_t err = cudaSuccess;
  switch (S) {
    case 1: err = launch_stream_step<T, 1>(a, n, stream); break;
    case 2: err = launch_stream_step<T, 2>(a, n, stream); break;
    case 3: err = launch_stream_step<T, 3>(a, n, stream); break;
    case 4: err = launch_stream_step<T, 4>(a, n, stream); break;
    case 5: err = launch_stream_step<T, 5>(a, n, stream); break;
    case 6: err = launch_stream_step<T, 6>(a, n, stream); break;
    case 7: err = launch_stream_step<T, 7>(a, n, stream); break;
    case 8: err = launch_stream_step<T, 8>(a, n, stream); break;
    default: return -2;
  }
  return err == cudaSuccess ? 0 : -5;
}

// h[r, f] = silu(gu[r, f]) * gu[r, F + f] for any F
template <typename T>
__global__ void silu_mul_kernel(const T* __restrict__ gu, T* __restrict__ h, long long rows, int F) {
  pdl_trigger();
  pdl_wait();
  const long long total = rows * F;
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const long long r = i / F;
    const int f = (int)(i - r * F);
    const float g = to_f(gu[r * 2 * F + f]), u = to_f(gu[r * 2 * F + F + f]);
    h[i] = from_f<T>(g * sigmoid(g) * u);
  }
}

// The two halves of a parallel mixer before their output projections:
//   a1[t, :] = attn[t, :] * sigmoid(g1)                                    (output gate of the attention half)
//   a2[t, head, :] = o[t, head, :] / rms(o[t, head, :]) * w[head, :] * sigmoid(g2)
// One CTA per token; a warp takes a head of the second half at a time, V columns per lane.
template <typename T, int V>
__global__ void __launch_bounds__(256)
gate_outputs_kernel(const T* __restrict__ attn, const float* __restrict__ o, const T* __restrict__ proj, long long ldp,
                    int g1_off, int g2_off, const T* __restrict__ w, float eps, int C1, int heads, int vdim,
                    T* __restrict__ a1, T* __restrict__ a2) {
  pdl_trigger();
  pdl_wait();
  const long long t = blockIdx.x;
  const T* g1 = proj + t * ldp + g1_off;
  const T* g2 = proj + t * ldp + g2_off;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
  auto gate = [](float z) { return sizeof(T) == 2 ? quick_sigmoid(z) : sigmoid(z); };
  for (int c = threadIdx.x * V; c < C1; c += blockDim.x * V) {
    float v[V], g[V];
    load_v<V>(attn + t * C1 + c, v);
    load_v<V>(g1 + c, g);
#pragma unroll
    for (int i = 0; i < V; ++i) v[i] *= gate(g[i]);
    store_v<V>(a1 + t * C1 + c, v);
  }
  for (int hd = warp; hd < heads; hd += nw) {
    const float* oh = o + (t * heads + hd) * (long long)vdim;
    float ss = 0.f;
    for (int c = lane * V; c < vdim; c += 32 * V) {
      float v[V];
      load_v<V>(oh + c, v);
#pragma unroll
      for (int i = 0; i < V; ++i) ss += v[i] * v[i];
    }
    ss = warp_sum(ss);
    const float r = 1.f / sqrtf(ss / (float)vdim + eps);
    for (int c = lane * V; c < vdim; c += 32 * V) {
      const int k = hd * vdim + c;
      float v[V], g[V], ww[V];
      load_v<V>(oh + c, v);
      load_v<V>(g2 + k, g);
      load_v<V>(w + k, ww);
#pragma unroll
      for (int i = 0; i < V; ++i) v[i] = v[i] * r * ww[i] * gate(g[i]);
      store_v<V>(a2 + t * heads * vdim + k, v);
    }
  }
}

// out[t, o] = sum_k x[t, k] w[o, k] in fp32, for a handful of outputs and few rows (gates of a decode step): one CTA per
// row, a warp per output.
__global__ void __launch_bounds__(512)
few_outputs_kernel(const __nv_bfloat16* __restrict__ x, const __nv_bfloat16* __restrict__ w, int K, int N, float* __restrict__ out) {
  pdl_trigger();
  pdl_wait();
  const long long t = blockIdx.x;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
  for (int o = warp; o < N; o += nw) {
    float acc = 0.f;
#pragma unroll 4
    for (int k = lane * 8; k < K; k += 256) {
      float a[8], b[8];
      load_v<8>(x + t * K + k, a);
      load_v<8>(w + (long long)o * K + k, b);
#pragma unroll
      for (int i = 0; i < 8; ++i) acc += a[i] * b[i];
    }
    acc = warp_sum(acc);
    if (lane == 0) out[t * N + o] = acc;
  }
}

}  // namespace

// dtype: 0 = bf16, 1 = float (activations and weights). x fp32 [n, S, D]; see StreamArgs.
TB_API int tb_stream_step(int dtype, float* x, int n, int S, int D, float eps, const void* y, const void* y2, const void* wy,
                          const void* wy2, const void* mix, const void* out, const long long* tokens, const void* embed,
                          int vocab, const void* in, const void* w, void* h, float* sum_out, cudaStream_t stream) {
  if (n <= 0) return 0;
  if (S < 1 || S > MAX_STREAMS || D <= 0 || D > 12000 || (y && tokens) || (y2 && !y)) return -2;
  StreamArgs a{x, D, eps, y, y2, wy, wy2, mix, out, tokens, embed, vocab, in, w, h, sum_out};
  return dtype == 0 ? dispatch_stream_step<__nv_bfloat16>(a, S, n, stream) : dispatch_stream_step<float>(a, S, n, stream);
}

TB_API int tb_silu_mul(int dtype, const void* gu, void* h, long long rows, int F, cudaStream_t stream) {
  if (rows <= 0 || F <= 0) return 0;
  const long long want = (rows * F + 255) / 256;
  const dim3 grid((unsigned)(want < 148 * 16 ? want : 148 * 16));
  cudaError_t err = dtype == 0
      ? launch_pdl(silu_mul_kernel<__nv_bfloat16>, grid, dim3(256), 0, stream, (const __nv_bfloat16*)gu, (__nv_bfloat16*)h, rows, F)
      : launch_pdl(silu_mul_kernel<float>, grid, dim3(256), 0, stream, (const float*)gu, (float*)h, rows, F);
  return err == cudaSuccess ? 0 : -5;
}

TB_API int tb_gate_outputs(int dtype, const void* attn, const float* o, const void* proj, long long ldp, int g1_off, int g2_off,
                           const void* w, float eps, int n, int C1, int heads, int vdim, void* a1, void* a2,
                           cudaStream_t stream) {
  if (n <= 0) return 0;
  typedef __nv_bfloat16 bf;
  const bool vec = C1 % 8 == 0 && vdim % 8 == 0 && ldp % 8 == 0 && g1_off % 8 == 0 && g2_off % 8 == 0;
#define GO(T, V)                                                                                                              \
  launch_pdl(gate_outputs_kernel<T, V>, dim3(n), dim3(256), 0, stream, (const T*)attn, o, (const T*)proj, ldp, g1_off, g2_off, \
             (const T*)w, eps, C1, heads, vdim, (T*)a1, (T*)a2)
  cudaError_t err = dtype == 0 ? (vec ? GO(bf, 8) : GO(bf, 1)) : GO(float, 1);
#undef GO
  return err == cudaSuccess ? 0 : -5;
}

// x bf16 [n, K], w bf16 [N, K] (contiguous, K a multiple of 8) -> out fp32 [n, N]
TB_API int tb_few_outputs(const void* x, const void* w, int n, int K, int N, float* out, cudaStream_t stream) {
  if (n <= 0 || N <= 0) return 0;
  if (K % 8) return -2;
  const int threads = N >= 16 ? 512 : N >= 8 ? 256 : 128;
  return launch_pdl(few_outputs_kernel, dim3(n), dim3(threads), 0, stream, (const __nv_bfloat16*)x, (const __nv_bfloat16*)w, K, N,
                    out) == cudaSuccess ? 0 : -5;
}
