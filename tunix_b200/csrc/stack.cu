// Kernels around the sublayers of layer-stack models (models/stack.py): parallel residual streams with their
// hyper-connection matrices, the norms at their ends, gated activations for any width. The streams and everything
// computed on them are fp32; T is the activation type of the model (bf16 or float).
//
//   stream_step : one launch between two sublayers. It closes the sublayer before it (streams <- mix^T streams +
//                 out * y) and opens the one after it (u = in . streams, h = RMS norm(u) * w), so that the streams are
//                 read and written once per sublayer. y is one tensor, or half the sum of two tensors that are
//                 RMS-normed first (two mixers side by side), or one tensor that is RMS-normed first (an update with a
//                 norm of its own). The first launch of a forward pass takes the embedding rows (normed, if the model
//                 norms them; scaled; with a learned row per position added) instead of streams, the last one has no
//                 successor but the final norm. A launch between two passes of a loop can add the embedding rows again,
//                 after the sum of the streams is reported. Norms may run over equal groups of a row. Without a norm
//                 the row itself is written in the activation type. In a decode step the launch can also mix the new
//                 row with the one before it (token shift). The embedding may add a row of a table of token pairs; its
//                 sum can be written out for a product that reads it again.
//   token_shift, keep_last : the same mixes for portions of prompts, and the rows that the next portions start from.
//   few_outputs, small_act : products with a handful of outputs, and what is applied to them (tanh; gelu times a row
//                 that belongs to the token).
//   xielu, glu  : the activations of feed-forwards without and with a gate.
//
// This file is compiled without fast-math: the same kernels serve the 32-bit mode.
#include "mma.cuh"
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
  const void* wy;             // T [D]; with y2 null: y alone is normed and weighted
  const void* wy2;            // T [D]
  const void* mix;            // T [S, S], row = from, column = to
  const void* out;            // T [S]
  // the start of a forward pass (instead of the above), or with y: rows that are added after it
  const long long* tokens;    // [n] or null
  const void* embed;          // T [V, D]
  int vocab;
  const void* embed_w;        // T [D] or null: weight of the norm of the embedding rows
  float embed_scale;          // factor of the (normed) embedding rows
  const void* pos;            // T [positions, D] or null: a row per position, added to the embedding rows
  int positions;
  const void* pairs;          // T [buckets + 1, D] or null: a row per pair of a token and the one before it, added as well;
  long long buckets, mul_prev, mul_cur;     //     row (before * mul_prev + token * mul_cur) mod buckets, the last row for a first token
  const long long* last;      // [slots] the token before an entry's first one
  void* start;                // T, rows ld_start apart, or null: the embedding rows as they are added
  long long ld_start;
  const int *cu, *ent;        // the batch's entries, with slot and pos0 below (read with pos, pairs, keep)
  int groups;                 // equal parts of a row that the norms of embedding and streams are taken over
  // the sublayer that follows
  const void* in;             // T [S]; null = all ones (the sum of the streams)
  const void* w;              // T [D] norm weight
  void* h;                    // T, rows ldh apart
  long long ldh;
  float* sum_out;             // fp32 [n, D] or null: the sum of the streams
  long long* keep;            // [slots] or null: receives the last token of every entry, from ids [n]
  const long long* ids;
  // token shift of a batch of single tokens (row = entry): mixes T [n_mix, n, D] instead of h
  const void* mu;             // T [n_mix, D] or null
  int n_mix;
  float* before;              // fp32 [slots, D]: the normed row of the token before, replaced by this one
  void* mixes;
  const int *slot, *pos0;
};

// 1 / rms of every group of the row u [D] in shared memory -> rs [groups]; part [groups + warps] is scratch. Starts and
// ends with a barrier.
__device__ __forceinline__ void group_rstd(const float* u, int D, int groups, float eps, float* part, float* rs) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  const int per = (nw + groups - 1) / groups, len = D / groups;
  __syncthreads();
  for (int i = warp; i < groups * per; i += nw) {
    const int g = i / per, p = i - g * per;
    const int a = g * len + (int)((long long)len * p / per), b = g * len + (int)((long long)len * (p + 1) / per);
    float s = 0.f;
    for (int d = a + lane; d < b; d += 32) s += u[d] * u[d];
    s = warp_sum(s);
    if (lane == 0) part[i] = s;
  }
  __syncthreads();
  for (int g = threadIdx.x; g < groups; g += blockDim.x) {
    float s = 0.f;
    for (int p = 0; p < per; ++p) s += part[g * per + p];
    rs[g] = 1.f / sqrtf(s / (float)len + eps);
  }
  __syncthreads();
}

// V elements of a row per thread and iteration (4, or 1 for widths that are no multiple of 4)
template <typename T, int S, int V>
__global__ void __launch_bounds__(512) stream_step_kernel(const StreamArgs a) {
  extern __shared__ float u_s[];          // [D], then scratch of the grouped norms
  __shared__ float red[33];
  float* part = u_s + ((a.D + 3) & ~3);   // [groups + warps]
  float* rs = part + a.groups + 32;       // [groups]
  const int glen = a.D / a.groups;
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
  if (a.wy && !y2) {
    float s1 = 0.f;
    for (int d = threadIdx.x * V; d < D; d += step) {
      float v1[V];
      load_v<V>(y + d, v1);
#pragma unroll
      for (int i = 0; i < V; ++i) s1 += v1[i] * v1[i];
    }
    r1 = 1.f / sqrtf(block_sum(s1, red) / (float)D + a.eps);
  }
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
  const T *emb = nullptr, *pos = nullptr, *pair = nullptr;
  if (a.keep && threadIdx.x == 0) {
    const int e = a.ent[row];
    if (row + 1 == a.cu[e + 1] && a.pos0[e] >= 0) a.keep[a.slot[e]] = a.ids[row];
  }
  if (a.tokens) {
    if (a.pos) {
      const int e = a.ent[row], p = a.pos0[e] + (int)row - a.cu[e];
      pos = static_cast<const T*>(a.pos) + (long long)min(max(p, 0), a.positions - 1) * D;
    }
    long long t = a.tokens[row];
    t = t < 0 ? 0 : (t >= a.vocab ? a.vocab - 1 : t);
    emb = static_cast<const T*>(a.embed) + t * D;
    if (a.pairs) {
      const int e = a.ent[row], p0 = a.pos0[e];
      const bool inside = row > a.cu[e];
      long long b = a.buckets;
      if (inside || p0 > 0) {
        long long before = inside ? a.tokens[row - 1] : a.last[a.slot[e]];
        before = before < 0 ? 0 : (before >= a.vocab ? a.vocab - 1 : before);
        b = (before * a.mul_prev + t * a.mul_cur) % a.buckets;
        if (b < 0) b += a.buckets;
      }
      pair = static_cast<const T*>(a.pairs) + b * D;
    }
    if (a.embed_w) {
      for (int d = threadIdx.x * V; d < D; d += step) {
        float ev[V];
        load_v<V>(emb + d, ev);
        store_v<V>(u_s + d, ev);
      }
      group_rstd(u_s, D, a.groups, a.eps, part, rs);
    }
  }
  float ss = 0.f;
  for (int d = threadIdx.x * V; d < D; d += step) {
    float v[S][V], ev[V];
    if (emb) {
      load_v<V>(emb + d, ev);
      if (a.embed_w) {
        float w[V];
        load_v<V>(static_cast<const T*>(a.embed_w) + d, w);
#pragma unroll
        for (int i = 0; i < V; ++i) ev[i] *= rs[(d + i) / glen] * w[i];
      }
#pragma unroll
      for (int i = 0; i < V; ++i) ev[i] *= a.embed_scale;
      if (pos) {
        float pv[V];
        load_v<V>(pos + d, pv);
#pragma unroll
        for (int i = 0; i < V; ++i) ev[i] += pv[i];
      }
      if (pair) {
        float pv[V];
        load_v<V>(pair + d, pv);
#pragma unroll
        for (int i = 0; i < V; ++i) ev[i] += pv[i];
      }
      if (a.start) store_v<V>(static_cast<T*>(a.start) + row * a.ld_start + d, ev);
    }
    if (emb && !y) {
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
        } else if (a.wy) {
          float w1[V];
          load_v<V>(static_cast<const T*>(a.wy) + d, w1);
#pragma unroll
          for (int i = 0; i < V; ++i) yv[i] *= r1 * w1[i];
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
    if (a.sum_out) {
      float tot[V];
#pragma unroll
      for (int i = 0; i < V; ++i) {
        tot[i] = 0.f;
#pragma unroll
        for (int s = 0; s < S; ++s) tot[i] += v[s][i];
      }
      store_v<V>(a.sum_out + row * D + d, tot);
    }
    if (emb && y) {
#pragma unroll
      for (int s = 0; s < S; ++s)
#pragma unroll
        for (int i = 0; i < V; ++i) v[s][i] += ev[i];
    }
#pragma unroll
    for (int s = 0; s < S; ++s) store_v<V>(x + (long long)s * D + d, v[s]);
    float u[V];
#pragma unroll
    for (int i = 0; i < V; ++i) {
      u[i] = 0.f;
#pragma unroll
      for (int s = 0; s < S; ++s) u[i] += inw[s] * v[s][i];
      ss += u[i] * u[i];
    }
    store_v<V>(u_s + d, u);
  }
  if (!a.h && !a.mu) return;
  if (!a.w) {                                            // the row itself
    T* h = static_cast<T*>(a.h) + row * a.ldh;
    for (int d = threadIdx.x * V; d < D; d += step) {
      float u[V];
      load_v<V>(u_s + d, u);
      store_v<V>(h + d, u);
    }
    return;
  }
  float r = 1.f;
  if (a.groups > 1) {
    group_rstd(u_s, D, a.groups, a.eps, part, rs);
  } else {
    r = 1.f / sqrtf(block_sum(ss, red) / (float)D + a.eps);
  }
  T* h = a.h ? static_cast<T*>(a.h) + row * a.ldh : nullptr;
  const int p0 = a.mu ? a.pos0[row] : 0;
  float* before = a.mu ? a.before + (long long)a.slot[row] * D : nullptr;
  for (int d = threadIdx.x * V; d < D; d += step) {      // each thread reads back what it wrote
    float u[V], w[V];
    load_v<V>(u_s + d, u);
    load_v<V>(static_cast<const T*>(a.w) + d, w);
    if (a.groups > 1) {
      const int g = d / glen;
      if (V == 1 || d + V - 1 < (g + 1) * glen) {
        const float rg = rs[g];
#pragma unroll
        for (int i = 0; i < V; ++i) u[i] *= rg * w[i];
      } else {
#pragma unroll
        for (int i = 0; i < V; ++i) u[i] *= rs[(d + i) / glen] * w[i];
      }
    } else {
#pragma unroll
      for (int i = 0; i < V; ++i) u[i] = u[i] * r * w[i];
    }
    if (h) store_v<V>(h + d, u);
    if (a.mu) {
      float b[V], m[V];
#pragma unroll
      for (int i = 0; i < V; ++i) { u[i] = to_f(from_f<T>(u[i])); b[i] = 0.f; }
      if (p0 > 0) load_v<V>(before + d, b);
      for (int k = 0; k < a.n_mix; ++k) {
        load_v<V>(static_cast<const T*>(a.mu) + (long long)k * D + d, m);
#pragma unroll
        for (int i = 0; i < V; ++i) m[i] = u[i] + (b[i] - u[i]) * m[i];
        store_v<V>(static_cast<T*>(a.mixes) + ((long long)k * gridDim.x + row) * D + d, m);
      }
      if (p0 >= 0) store_v<V>(before + d, u);
    }
  }
}

template <typename T, int S>
cudaError_t launch_stream_step(const StreamArgs& a, int n, cudaStream_t stream) {
  const bool vec = a.D % 4 == 0 && (!a.h || a.ldh % 4 == 0) && (!a.start || a.ld_start % 4 == 0);
  const int per = vec ? a.D / 4 : a.D;
  int threads = n <= 296 ? 512 : 256;              // few rows: the latency of one row counts
  while (threads > 128 && threads / 2 >= per) threads /= 2;
  const size_t smem = (size_t)(((a.D + 3) & ~3) + 2 * a.groups + 32) * 4;
  if (vec) return launch_pdl(stream_step_kernel<T, S, 4>, dim3(n), dim3(threads), smem, stream, a);
  return launch_pdl(stream_step_kernel<T, S, 1>, dim3(n), dim3(threads), smem, stream, a);
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

// h[r, f] = act(gu[r, f]) * gu[r, F + f] for any F; act: 0 silu, 1 gelu (tanh form)
template <typename T>
__global__ void glu_kernel(int kind, const T* __restrict__ gu, T* __restrict__ h, long long ldh, long long rows, int F) {
  pdl_trigger();
  pdl_wait();
  const long long total = rows * F;
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const long long r = i / F;
    const int f = (int)(i - r * F);
    const float g = to_f(gu[r * 2 * F + f]), u = to_f(gu[r * 2 * F + F + f]);
    h[r * ldh + f] = from_f<T>((kind == 0 ? g * sigmoid(g) : gelu_tanh(g)) * u);
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

// What is applied to a few outputs: 0 nothing, 1 tanh, 2 gelu (tanh form) times a row of the token's own,
// e[tokens[t], e_off + o].
template <typename T>
__device__ __forceinline__ float apply_small(int act, float z, const long long* tokens, int vocab, const T* e, long long lde,
                                             int e_off, long long t, int o) {
  if (act == 1) return tanhf(z);
  if (act == 2) {
    long long id = tokens[t];
    id = id < 0 ? 0 : (id >= vocab ? vocab - 1 : id);
    return gelu_tanh(z) * to_f(e[id * lde + e_off + o]);
  }
  return z;
}

// out[t, o] = act(sum_k x[t, k] w[o, k]) with an fp32 sum, for few outputs and few rows (gates and bottlenecks of a decode
// step): a CTA owns 16 rows x 8 outputs, its warps split the contraction and meet in shared memory. A lane loads 8 consecutive
// k of its two rows and its output at once; both operands see the same permutation of k, so no shuffle is needed.
constexpr int FW = 8;           // warps
template <typename TO>
__global__ void __launch_bounds__(32 * FW)
few_outputs_kernel(const __nv_bfloat16* __restrict__ x, const __nv_bfloat16* __restrict__ w, int n, int K, int N, int act,
                   const long long* __restrict__ tokens, int vocab, const __nv_bfloat16* __restrict__ e, long long lde, int e_off,
                   TO* __restrict__ out) {
  __shared__ float part[FW][16][9];
  pdl_trigger();
  pdl_wait();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, q8 = (lane & 3) * 8;
  const int r0 = blockIdx.y * 16 + g, r1 = r0 + 8, o = blockIdx.x * 8 + g;
  const __nv_bfloat16 *x0 = x + (long long)min(r0, n - 1) * K, *x1 = x + (long long)min(r1, n - 1) * K, *wo = w + (long long)min(o, N - 1) * K;
  float acc[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 8
  for (int kb = warp * 32; kb < K; kb += FW * 32) {             // whole warps stay together for the products
    const int k = kb + q8;                                      // K is a multiple of 8: a lane's 8 elements are in or out
    const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
    const uint4 a = k < K ? *reinterpret_cast<const uint4*>(x0 + k) : zero, b = k < K ? *reinterpret_cast<const uint4*>(x1 + k) : zero;
    const uint4 c = k < K ? *reinterpret_cast<const uint4*>(wo + k) : zero;
    const uint32_t s0[4] = {a.x, b.x, a.y, b.y}, s1[4] = {a.z, b.z, a.w, b.w};
    mma_16816(acc, s0, c.x, c.y);
    mma_16816(acc, s1, c.z, c.w);
  }
  const int c2 = 2 * (lane & 3);
  part[warp][g][c2] = acc[0];
  part[warp][g][c2 + 1] = acc[1];
  part[warp][g + 8][c2] = acc[2];
  part[warp][g + 8][c2 + 1] = acc[3];
  __syncthreads();
  if (threadIdx.x < 128) {
    const int r = threadIdx.x >> 3, c = threadIdx.x & 7, oo = blockIdx.x * 8 + c;
    const long long t = blockIdx.y * 16 + r;
    if (t < n && oo < N) {
      float v = 0.f;
#pragma unroll
      for (int i = 0; i < FW; ++i) v += part[i][r][c];
      out[t * N + oo] = from_f<TO>(apply_small(act, v, tokens, vocab, e, lde, e_off, t, oo));
    }
  }
}

// out[t, o] = act(z[t, o])
template <typename T>
__global__ void small_act_kernel(const float* __restrict__ z, int N, long long total, int act, const long long* __restrict__ tokens,
                                 int vocab, const T* __restrict__ e, long long lde, int e_off, T* __restrict__ out) {
  pdl_trigger();
  pdl_wait();
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const long long t = i / N;
    out[i] = from_f<T>(apply_small(act, z[i], tokens, vocab, e, lde, e_off, t, (int)(i - t * N)));
  }
}

// xIELU in place: z > 0: softplus(p) z^2 + z / 2; else (1/2 + softplus(q)) (e^z - 1 - z) + z / 2; (p, q) = act
template <typename T, int V>
__global__ void __launch_bounds__(256) xielu_kernel(T* __restrict__ x, const T* __restrict__ act, long long total) {
  pdl_trigger();
  pdl_wait();
  const float ap = softplus(to_f(act[0])), an = 0.5f + softplus(to_f(act[1]));
  for (long long i = ((long long)blockIdx.x * blockDim.x + threadIdx.x) * V; i < total; i += (long long)gridDim.x * blockDim.x * V) {
    float v[V];
    load_v<V>(x + i, v);
#pragma unroll
    for (int q = 0; q < V; ++q) {
      const float z = v[q], m = fminf(z, 0.f);
      const float em = sizeof(T) == 2 ? quick_expm1(m) : expm1f(m);
      v[q] = (z > 0.f ? ap * z * z : an * (em - z)) + 0.5f * z;
    }
    store_v<V>(x + i, v);
  }
}

// Token shift of a ragged batch: mixes[m, t] = h[t] + (before - h[t]) mu[m], where before is the row of the sequence's
// token before (its slot's `carry` at the start of a portion, zero at the start of the sequence). A thread keeps V
// channels of all mu and walks ST tokens. The carry is only read: whoever runs after this kernel replaces it.
constexpr int ST = 16;
template <typename T, int V, int NM>
__global__ void __launch_bounds__(128)
token_shift_kernel(const T* __restrict__ h, const T* __restrict__ mu, const float* __restrict__ carry, Ragged rb, int D,
                   int n_mix, T* __restrict__ mixes) {
  pdl_trigger();
  pdl_wait();
  const int d = (blockIdx.x * blockDim.x + threadIdx.x) * V;
  if (d >= D) return;
  const int t0 = blockIdx.y * ST, t1 = min(t0 + ST, rb.n);
  float m[NM][V], prev[V];
#pragma unroll
  for (int k = 0; k < NM; ++k)
    if (k < n_mix) load_v<V>(mu + (long long)k * D + d, m[k]);
  if (t0 > 0) load_v<V>(h + (long long)(t0 - 1) * D + d, prev);
  for (int t = t0; t < t1; ++t) {
    const int e = rb.ent[t];
    float u[V];
    load_v<V>(h + (long long)t * D + d, u);
    if (t == rb.cu[e]) {
      if (rb.pos0[e] > 0) {
        load_v<V>(carry + (long long)rb.slot[e] * D + d, prev);
      } else {
#pragma unroll
        for (int i = 0; i < V; ++i) prev[i] = 0.f;
      }
    }
#pragma unroll
    for (int k = 0; k < NM; ++k)
      if (k < n_mix) {
        float v[V];
#pragma unroll
        for (int i = 0; i < V; ++i) v[i] = u[i] + (prev[i] - u[i]) * m[k][i];
        store_v<V>(mixes + ((long long)k * rb.n + t) * D + d, v);
      }
#pragma unroll
    for (int i = 0; i < V; ++i) prev[i] = u[i];
  }
}

// carry[slot[e]] = the last row of entry e of h (fp32 copies)
template <typename T>
__global__ void __launch_bounds__(256) keep_last_kernel(const T* __restrict__ h, float* __restrict__ carry, Ragged rb, int D) {
  pdl_trigger();
  pdl_wait();
  const int e = blockIdx.y, d = blockIdx.x * blockDim.x + threadIdx.x;
  if (d < D && rb.pos0[e] >= 0) carry[(long long)rb.slot[e] * D + d] = to_f(h[(long long)(rb.cu[e + 1] - 1) * D + d]);
}

}  // namespace

// dtype: 0 = bf16, 1 = float (activations and weights). x fp32 [n, S, D]; see StreamArgs.
TB_API int tb_stream_step(int dtype, float* x, int n, int S, int D, float eps, const void* y, const void* y2, const void* wy,
                          const void* wy2, const void* mix, const void* out, const long long* tokens, const void* embed,
                          int vocab, const void* embed_w, float embed_scale, const void* pos, int positions, int groups,
                          const void* in, const void* w, void* h, long long ldh, float* sum_out, const void* mu, int n_mix, float* before,
                          void* mixes, const void* pairs, long long buckets, long long mul_prev, long long mul_cur,
                          const long long* last, void* start, long long ld_start, long long* keep, const long long* ids,
                          const int* cu, const int* slot, const int* pos0, const int* ent, cudaStream_t stream) {
  if (n <= 0) return 0;
  if (S < 1 || S > MAX_STREAMS || D <= 0 || D > 11000 || (y2 && !y)) return -2;
  if (pos && (!tokens || positions <= 0 || !cu || !pos0 || !ent)) return -2;
  if (groups < 1 || groups > 256 || D % groups || (mu && (!w || !before || !mixes))) return -2;
  if (pairs && (!tokens || buckets <= 0 || !last || !cu || !slot || !pos0 || !ent)) return -2;
  if (keep && (!ids || !cu || !slot || !pos0 || !ent)) return -2;
  StreamArgs a{x, D, eps, y, y2, wy, wy2, mix, out, tokens, embed, vocab, embed_w, embed_scale, pos, positions, pairs, buckets,
               mul_prev, mul_cur, last, start, ld_start, cu, ent, groups, in, w, h, ldh, sum_out, keep, ids, mu, n_mix, before,
               mixes, slot, pos0};
  return dtype == 0 ? dispatch_stream_step<__nv_bfloat16>(a, S, n, stream) : dispatch_stream_step<float>(a, S, n, stream);
}

// h T [n, D] contiguous, mu T [n_mix, D] with at most 8 mixes, carry fp32 [slots, D] -> mixes T [n_mix, n, D]
TB_API int tb_token_shift(int dtype, const void* h, const void* mu, int n_mix, const float* carry, const int* cu, const int* slot,
                          const int* pos0, const int* ent, int E, int n, int D, void* mixes, cudaStream_t stream) {
  if (n <= 0 || E <= 0) return 0;
  if (n_mix < 1 || n_mix > 8 || (n + ST - 1) / ST > 65535) return -2;
  Ragged rb{cu, slot, pos0, ent, E, n};
  typedef __nv_bfloat16 bf;
#define TS(T, V, NM)                                                                                                        \
  launch_pdl(token_shift_kernel<T, V, NM>, dim3((D / V + 127) / 128, (n + ST - 1) / ST), dim3(128), 0, stream, (const T*)h,  \
             (const T*)mu, carry, rb, D, n_mix, (T*)mixes)
  cudaError_t err = dtype != 0 ? TS(float, 1, 8)
                    : n_mix == 1 && D % 8 == 0 ? TS(bf, 8, 1)
                    : D % 4 ? TS(bf, 1, 8) : n_mix <= 5 ? TS(bf, 4, 5) : TS(bf, 4, 8);
#undef TS
  return err == cudaSuccess ? 0 : -5;
}

// h T [n, D] contiguous -> carry fp32 [slots, D]: the last row of every entry
TB_API int tb_keep_last(int dtype, const void* h, float* carry, const int* cu, const int* slot, const int* pos0, const int* ent, int E,
                        int n, int D, cudaStream_t stream) {
  if (n <= 0 || E <= 0) return 0;
  if (E > 65535) return -2;
  Ragged rb{cu, slot, pos0, ent, E, n};
  const dim3 grid((D + 255) / 256, E);
  const cudaError_t err = dtype == 0 ? launch_pdl(keep_last_kernel<__nv_bfloat16>, grid, dim3(256), 0, stream, (const __nv_bfloat16*)h, carry, rb, D)
                                     : launch_pdl(keep_last_kernel<float>, grid, dim3(256), 0, stream, (const float*)h, carry, rb, D);
  return err == cudaSuccess ? 0 : -5;
}

// act T [2]; x T [total] in place
TB_API int tb_xielu(int dtype, void* x, const void* act, long long total, cudaStream_t stream) {
  if (total <= 0) return 0;
  const int V = dtype == 0 && total % 8 == 0 ? 8 : 1;
  const long long want = (total / V + 255) / 256;
  const dim3 grid((unsigned)(want < 148 * 16 ? want : 148 * 16));
  typedef __nv_bfloat16 bf;
  cudaError_t err = dtype != 0 ? launch_pdl(xielu_kernel<float, 1>, grid, dim3(256), 0, stream, (float*)x, (const float*)act, total)
                    : V == 8   ? launch_pdl(xielu_kernel<bf, 8>, grid, dim3(256), 0, stream, (bf*)x, (const bf*)act, total)
                               : launch_pdl(xielu_kernel<bf, 1>, grid, dim3(256), 0, stream, (bf*)x, (const bf*)act, total);
  return err == cudaSuccess ? 0 : -5;
}

// z fp32 [n, N] -> out T [n, N]; act as in apply_small, e T [vocab, lde]
TB_API int tb_small_act(int dtype, const float* z, int n, int N, int act, const long long* tokens, int vocab, const void* e,
                        long long lde, int e_off, void* out, cudaStream_t stream) {
  const long long total = (long long)n * N, want = (total + 255) / 256;
  if (total <= 0) return 0;
  const dim3 grid((unsigned)(want < 148 * 16 ? want : 148 * 16));
  cudaError_t err = dtype == 0
      ? launch_pdl(small_act_kernel<__nv_bfloat16>, grid, dim3(256), 0, stream, z, N, total, act, tokens, vocab,
                   (const __nv_bfloat16*)e, lde, e_off, (__nv_bfloat16*)out)
      : launch_pdl(small_act_kernel<float>, grid, dim3(256), 0, stream, z, N, total, act, tokens, vocab, (const float*)e, lde,
                   e_off, (float*)out);
  return err == cudaSuccess ? 0 : -5;
}

// gu T [rows, 2 F] (gates, then ups) -> h T [rows, F], rows ldh apart; kind as in glu_kernel
TB_API int tb_glu(int dtype, int kind, const void* gu, void* h, long long ldh, long long rows, int F, cudaStream_t stream) {
  if (rows <= 0 || F <= 0) return 0;
  const long long want = (rows * F + 255) / 256;
  const dim3 grid((unsigned)(want < 148 * 16 ? want : 148 * 16));
  cudaError_t err = dtype == 0
      ? launch_pdl(glu_kernel<__nv_bfloat16>, grid, dim3(256), 0, stream, kind, (const __nv_bfloat16*)gu, (__nv_bfloat16*)h, ldh, rows, F)
      : launch_pdl(glu_kernel<float>, grid, dim3(256), 0, stream, kind, (const float*)gu, (float*)h, ldh, rows, F);
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

// x bf16 [n, K], w bf16 [N, K] (contiguous, K a multiple of 8) -> out [n, N], fp32 or (out_bf16) bf16; act, e as in apply_small
TB_API int tb_few_outputs(const void* x, const void* w, int n, int K, int N, int act, const long long* tokens, int vocab,
                          const void* e, long long lde, int e_off, void* out, int out_bf16, cudaStream_t stream) {
  if (n <= 0 || N <= 0) return 0;
  if (K % 8) return -2;
  typedef __nv_bfloat16 bf;
  const dim3 grid((N + 7) / 8, (n + 15) / 16);
  if (grid.y > 65535) return -2;
#define FO(TO)                                                                                                              \
  launch_pdl(few_outputs_kernel<TO>, grid, dim3(32 * FW), 0, stream, (const bf*)x, (const bf*)w, n, K, N, act, tokens, vocab, \
             (const bf*)e, lde, e_off, (TO*)out)
  return (out_bf16 ? FO(bf) : FO(float)) == cudaSuccess ? 0 : -5;
#undef FO
}
