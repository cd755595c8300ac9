// Attention over a paged cache for the ragged batches of layer-stack models: sliding windows with kept first tokens or
// chunks, learned distance bias, score cap, rotary positions.
//
//   qk_norm_write : after the fused projection of a step: RMS norm of q and of k over the WHOLE projection (all heads at
//                   once), q to a compact buffer, k and v rows to their pages (value rows may be wider or narrower than
//                   key rows).
//   rope_norm_write : the same place for rotary attention: every query and key head is divided by its root mean square
//                   (and weighted, if the model has weights), then its first `rd` dimensions turn by the angles of the
//                   token's position, element i together with i + rd / 2, or (interleaved) 2 i together with 2 i + 1. Heads
//                   can be stored wider than they are, with zeros behind them, so that the tensor-core kernels fit them. A
//                   layer that reads another layer's cache has queries only. Which heads are normed (queries and keys,
//                   values) is the caller's choice; without query heads only keys and values are written.
//   window_attn   : any head sizes, bf16 or float: one warp per (token, query head), lanes over keys for the scores and
//                   over value columns for the output, online softmax in fp32. Position i sees j <= i with
//                   (i - j < window and j in i's chunk) or j < keep. A sink is one more score, without a value, in the sum
//                   of the weights (-inf: none), the same or a learned one per head. A head's output may have a gate of
//                   its own. Models whose heads fit the tensor-core kernels (attention_fwd.cu, decode.cu) use those instead.
//
// This file is compiled without fast-math: the same kernels serve the 32-bit mode.
#include "precise.cuh"

using namespace tb;

namespace {

struct Paged {
  const int* table;
  int max_pages, page_size;
};

__device__ __forceinline__ long long page_row(const Paged& pg, const int* pt, int p) {
  return (long long)pt[p / pg.page_size] * pg.page_size + p % pg.page_size;
}

template <typename T, int V>
__global__ void __launch_bounds__(256)
qk_norm_write_kernel(const T* __restrict__ proj, long long ldp, int q_off, int k_off, int v_off, const T* __restrict__ qw,
                     const T* __restrict__ kw, float eps, Ragged rb, Paged pg, int NQ, int NK, int NVv, T* __restrict__ q,
                     T* __restrict__ kp, T* __restrict__ vp) {
  __shared__ float red[33];
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x, tid = threadIdx.x;
  const int e = rb.ent[t], p0 = rb.pos0[e];
  const T* row = proj + (long long)t * ldp;
  if (p0 < 0) {
    for (int c = tid; c < NQ; c += blockDim.x) q[(long long)t * NQ + c] = from_f<T>(0.f);
    return;
  }
  float sq = 0.f, sk = 0.f;
  const int step = blockDim.x * V;
  auto sumsq = [&](int off, int N) {
    float s = 0.f;
    for (int c = tid * V; c < N; c += step) {
      float v[V];
      load_v<V>(row + off + c, v);
#pragma unroll
      for (int i = 0; i < V; ++i) s += v[i] * v[i];
    }
    return s;
  };
  sq = block_sum(sumsq(q_off, NQ), red);
  sk = block_sum(sumsq(k_off, NK), red);
  const float rq = 1.f / sqrtf(sq / (float)NQ + eps), rk = 1.f / sqrtf(sk / (float)NK + eps);
  const int p = p0 + t - rb.cu[e];
  const long long pr = page_row(pg, pg.table + (long long)rb.slot[e] * pg.max_pages, p);
  auto norm = [&](int off, int N, float r, const T* w, T* dst) {
    for (int c = tid * V; c < N; c += step) {
      float v[V], ww[V];
      load_v<V>(row + off + c, v);
      load_v<V>(w + c, ww);
#pragma unroll
      for (int i = 0; i < V; ++i) v[i] = v[i] * r * ww[i];
      store_v<V>(dst + c, v);
    }
  };
  norm(q_off, NQ, rq, qw, q + (long long)t * NQ);
  norm(k_off, NK, rk, kw, kp + pr * NK);
  for (int c = tid * V; c < NVv; c += step) {
    float v[V];
    load_v<V>(row + v_off + c, v);
    store_v<V>(vp + pr * NVv + c, v);
  }
}

constexpr int NORM_QK = 1, NORM_V = 2;     // which heads are divided by their root mean square

// Heads of a multiple of 8 dimensions that turn by a multiple of 16 (8 if interleaved): LPH lanes per head, 8 elements per lane;
// the partner of a rotation sits rd / 16 lanes away, or in the same lane. Otherwise like rope_norm_write_kernel.
template <int LPH, bool INTER>
__global__ void __launch_bounds__(256)
rope_norm_write_vec_kernel(const __nv_bfloat16* __restrict__ proj, long long ldp, int q_off, int k_off, int v_off,
                           const __nv_bfloat16* __restrict__ qw, const __nv_bfloat16* __restrict__ kw, const float* __restrict__ cos_t,
                           const float* __restrict__ sin_t, int rd, float eps, int norms, Ragged rb, Paged pg, int H, int G, int dq,
                           int dv, int wq, int wv, __nv_bfloat16* __restrict__ q, __nv_bfloat16* __restrict__ kp,
                           __nv_bfloat16* __restrict__ vp) {
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x, lane = threadIdx.x & 31, sub = threadIdx.x % LPH, e = rb.ent[t], p0 = rb.pos0[e];
  const int heads = H + 2 * G, base = lane - sub, half8 = rd >> 4;
  const __nv_bfloat16* row = proj + (long long)t * ldp;
  const int p = p0 + t - rb.cu[e];
  long long pr = 0;
  if (p0 >= 0 && G > 0) pr = page_row(pg, pg.table + (long long)rb.slot[e] * pg.max_pages, p);
  const bool turns = sub * 8 < rd && p0 >= 0;
  const int partner = turns ? (sub < half8 ? sub + half8 : sub - half8) : sub;
  float c[8], s[8];
#pragma unroll
  for (int i = 0; i < 8; ++i) { c[i] = 1.f; s[i] = 0.f; }
  if (INTER && turns) {
    float c4[4], s4[4];
    load_v<4>(cos_t + (long long)p * (rd >> 1) + sub * 4, c4);
    load_v<4>(sin_t + (long long)p * (rd >> 1) + sub * 4, s4);
#pragma unroll
    for (int i = 0; i < 8; ++i) { c[i] = c4[i >> 1]; s[i] = (i & 1) ? s4[i >> 1] : -s4[i >> 1]; }
  } else if (turns) {
    const long long at = (long long)p * (rd >> 1) + (sub < half8 ? sub : sub - half8) * 8;
    load_v<8>(cos_t + at, c);
    load_v<8>(sin_t + at, s);
    if (sub < half8) {
#pragma unroll
      for (int i = 0; i < 8; ++i) s[i] = -s[i];
    }
  }
  float wa[8], wb[8];                                   // norm weights of this lane's elements of a query / key head
#pragma unroll
  for (int i = 0; i < 8; ++i) wa[i] = wb[i] = 1.f;
  if (qw && sub * 8 < dq) load_v<8>(qw + sub * 8, wa);
  if (kw && sub * 8 < dq) load_v<8>(kw + sub * 8, wb);
  for (int h0 = 0; h0 < heads; h0 += 256 / LPH) {       // whole warps stay together for the shuffles
    const int hh = h0 + threadIdx.x / LPH;
    const bool is_v = hh >= H + G, ok = hh < heads && sub * 8 < (is_v ? dv : dq) && p0 >= 0;
    float v[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) v[i] = 0.f;
    if (ok) load_v<8>(row + (hh < H ? q_off + hh * dq : is_v ? v_off + (hh - H - G) * dv : k_off + (hh - H) * dq) + sub * 8, v);
    float o[8], ss = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) ss += v[i] * v[i];
#pragma unroll
    for (int w = LPH / 2; w >= 1; w >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, w);
    if (norms & (is_v ? NORM_V : NORM_QK)) {
      const float r = 1.f / sqrtf(ss / (float)(is_v ? dv : dq) + eps);
#pragma unroll
      for (int i = 0; i < 8; ++i) v[i] *= is_v ? r : r * (hh < H ? wa[i] : wb[i]);
    }
#pragma unroll
    for (int i = 0; i < 8; ++i)
      o[i] = v[i] * c[i] + (INTER ? v[i ^ 1] : __shfl_sync(0xffffffffu, v[i], base + partner)) * s[i];
    if (hh < H) {
      if (sub * 8 < wq) store_v<8>(q + ((long long)t * H + hh) * wq + sub * 8, o);
    } else if (hh < heads && p0 >= 0) {
      if (!is_v && sub * 8 < wq) store_v<8>(kp + (pr * G + hh - H) * wq + sub * 8, o);
      if (is_v && sub * 8 < wv) store_v<8>(vp + (pr * G + hh - H - G) * wv + sub * 8, v);
    }
  }
}

// One warp per (token, head) over the query heads, then key heads, then value heads of a row. cos / sin [positions, rd / 2].
template <typename T>
__global__ void __launch_bounds__(256)
rope_norm_write_kernel(const T* __restrict__ proj, long long ldp, int q_off, int k_off, int v_off, const T* __restrict__ qw,
                       const T* __restrict__ kw, const float* __restrict__ cos_t, const float* __restrict__ sin_t, int rd, int inter,
                       float eps, int norms, Ragged rb, Paged pg, int H, int G, int dq, int dv, int wq, int wv, T* __restrict__ q,
                       T* __restrict__ kp, T* __restrict__ vp) {
  pdl_trigger();
  pdl_wait();
  const int heads = H + 2 * G;
  const long long wid = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (wid >= (long long)rb.n * heads) return;
  const int lane = threadIdx.x & 31;
  const int t = (int)(wid / heads), hh = (int)(wid - (long long)t * heads);
  const int e = rb.ent[t], p0 = rb.pos0[e];
  const T* row = proj + (long long)t * ldp;
  if (p0 < 0) {
    if (hh < H)
      for (int c = lane; c < wq; c += 32) q[((long long)t * H + hh) * wq + c] = from_f<T>(0.f);
    return;
  }
  const int p = p0 + t - rb.cu[e];
  long long pr = 0;
  if (hh >= H) pr = page_row(pg, pg.table + (long long)rb.slot[e] * pg.max_pages, p);
  if (hh >= H + G) {
    const int g = hh - H - G;
    const T* src = row + v_off + g * dv;
    float ss = 0.f, r = 1.f;
    if (norms & NORM_V) {
      for (int c = lane; c < dv; c += 32) { const float x = to_f(src[c]); ss += x * x; }
      r = 1.f / sqrtf(warp_sum(ss) / (float)dv + eps);
    }
    for (int c = lane; c < wv; c += 32) vp[(pr * G + g) * wv + c] = from_f<T>(c < dv ? to_f(src[c]) * r : 0.f);
    return;
  }
  const T* src = row + (hh < H ? q_off + hh * dq : k_off + (hh - H) * dq);
  const T* w = hh < H ? qw : kw;
  T* dst = hh < H ? q + ((long long)t * H + hh) * wq : kp + (pr * G + hh - H) * wq;
  const int half = rd >> 1;
  const float *ct = cos_t + (long long)p * half, *st = sin_t + (long long)p * half;
  float ss = 0.f;
  for (int c = lane; c < dq; c += 32) { const float x = to_f(src[c]); ss += x * x; }
  const float r = norms & NORM_QK ? 1.f / sqrtf(warp_sum(ss) / (float)dq + eps) : 1.f;
  auto normed = [&](int c) { return to_f(src[c]) * r * (w ? to_f(w[c]) : 1.f); };
  for (int c = lane; c < wq; c += 32) {
    float x = 0.f;
    if (c >= rd) {
      if (c < dq) x = normed(c);
    } else if (inter) {
      const float a = normed(c), b = normed(c ^ 1);
      x = (c & 1) ? a * ct[c >> 1] + b * st[c >> 1] : a * ct[c >> 1] - b * st[c >> 1];
    } else {
      x = c < half ? normed(c) * ct[c] - normed(c + half) * st[c] : normed(c) * ct[c - half] + normed(c - half) * st[c - half];
    }
    dst[c] = from_f<T>(x);
  }
}

constexpr int VREG = 16;        // value columns per lane: wider value heads are cut over blockIdx.y

template <typename T>
__global__ void __launch_bounds__(128)
window_attn_kernel(const T* __restrict__ q, long long ldq, int qs_heads, const T* __restrict__ kp, const T* __restrict__ vp, Ragged rb,
                   Paged pg, int H, int G, int dq, int dv, int wq, int wv, float scale, float cap, const float* __restrict__ bias, int far,
                   int window, int chunk, int keep, float sink, const float* __restrict__ sinks, const T* __restrict__ gate,
                   long long ldg, float out_scale, T* __restrict__ out, long long ldo) {
  extern __shared__ float qs_all[];               // [4][dq]
  pdl_trigger();
  pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long wid = (long long)blockIdx.x * 4 + warp;
  if (wid >= (long long)rb.n * H) return;
  const int t = (int)(wid / H), h = (int)(wid - (long long)t * H), g = h / (H / G);
  const int e = rb.ent[t], p0 = rb.pos0[e];
  T* o = out + (long long)t * ldo + (long long)h * dv;
  const int c0 = blockIdx.y * VREG * 32;          // first value column of this block
  if (p0 < 0) {
    for (int c = c0 + lane; c < min(dv, c0 + VREG * 32); c += 32) o[c] = from_f<T>(0.f);
    return;
  }
  float* qs = qs_all + warp * dq;
  for (int d = lane; d < dq; d += 32) qs[d] = to_f(q[(long long)t * ldq + (long long)h * qs_heads + d]) * scale;
  __syncwarp();
  const int i = p0 + t - rb.cu[e];
  const int lo = first_visible(i, window, chunk);
  const int kept = min(keep, lo);                 // keys 0 .. kept-1 lie before the window
  const int cnt = kept + i - lo + 1;
  const int* pt = pg.table + (long long)rb.slot[e] * pg.max_pages;
  float m = -INFINITY, l = 0.f;
  float acc[VREG];
#pragma unroll
  for (int r = 0; r < VREG; ++r) acc[r] = 0.f;
  for (int b = 0; b < cnt; b += 32) {
    const int x = b + lane;
    float s = -INFINITY;
    long long row = 0;
    if (x < cnt) {
      const int j = x < kept ? x : lo + x - kept;
      row = page_row(pg, pt, j);
      const T* k = kp + (row * G + g) * wq;
      float dot = 0.f;
      for (int d = 0; d < dq; ++d) dot += qs[d] * to_f(k[d]);
      s = cap > 0.f ? cap * tanhf(dot / cap) : dot;
      if (bias) s += bias[(long long)h * (far + 1) + min(i - j, far)];
    }
    const float mn = fmaxf(m, warp_max(s));
    const float p = expf(s - mn), c = expf(m - mn);
    l = l * c + warp_sum(p);
    m = mn;
#pragma unroll
    for (int r = 0; r < VREG; ++r) acc[r] *= c;
    const int lim = min(32, cnt - b);
    for (int y = 0; y < lim; ++y) {
      const float py = __shfl_sync(0xffffffffu, p, y);
      const long long ry = __shfl_sync(0xffffffffu, row, y);
      const T* v = vp + (ry * G + g) * wv;
#pragma unroll
      for (int r = 0; r < VREG; ++r) {
        const int cc = c0 + r * 32 + lane;
        if (cc < dv) acc[r] += py * to_f(v[cc]);
      }
    }
  }
  const float inv = out_scale * (gate ? sigmoid(to_f(gate[(long long)t * ldg + h])) : 1.f) / (l + expf((sinks ? sinks[h] : sink) - m));
#pragma unroll
  for (int r = 0; r < VREG; ++r) {
    const int cc = c0 + r * 32 + lane;
    if (cc < dv) o[cc] = from_f<T>(acc[r] * inv);
  }
}

}  // namespace

#define RAGGED Ragged rb{cu, slot, pos0, ent, E, n}
#define PAGED Paged pg{table, max_pages, page_size}

// NQ = H * dq, NK = G * dq, NV = G * dv columns of proj [n, ldp]; pools [pages, page_size, NK] and [.., NV]; q [n, NQ].
TB_API int tb_qk_norm_write(int dtype, const void* proj, long long ldp, int q_off, int k_off, int v_off, const void* qw,
                            const void* kw, float eps, const int* cu, const int* slot, const int* pos0, const int* ent, int E,
                            int n, const int* table, int max_pages, int page_size, int NQ, int NK, int NV, void* q, void* kp,
                            void* vp, cudaStream_t stream) {
  if (n <= 0) return 0;
  RAGGED;
  PAGED;
  const bool vec = NQ % 8 == 0 && NK % 8 == 0 && NV % 8 == 0 && q_off % 8 == 0 && k_off % 8 == 0 && v_off % 8 == 0 && ldp % 8 == 0;
#define RUN(T, V)                                                                                                            \
  launch_pdl(qk_norm_write_kernel<T, V>, dim3(n), dim3(256), 0, stream, (const T*)proj, ldp, q_off, k_off, v_off,            \
             (const T*)qw, (const T*)kw, eps, rb, pg, NQ, NK, NV, (T*)q, (T*)kp, (T*)vp)
  const cudaError_t err = dtype == 0 ? (vec ? RUN(__nv_bfloat16, 8) : RUN(__nv_bfloat16, 1)) : RUN(float, 1);
#undef RUN
  return err == cudaSuccess ? 0 : -5;
}

// q | k | v: columns of proj [n, ldp]; H query heads of dq, G key / value heads (0: queries only) of dq / dv; qw, kw T [dq] or
// null: weights of the heads' norms; norms: bit 0 query and key heads, bit 1 value heads; rd rotated dimensions (inter: neighbours turn together) with tables cos / sin fp32
// [positions, rd / 2]. Heads are stored wq / wv wide: q [n, H * wq] (H 0: keys and values only); pools [pages, page_size, G * wq]
// and [.., G * wv].
TB_API int tb_rope_norm_write(int dtype, const void* proj, long long ldp, int q_off, int k_off, int v_off, const void* qw,
                              const void* kw, const float* cos_t, const float* sin_t, int rd, int inter, float eps, int norms, const int* cu,
                              const int* slot, const int* pos0, const int* ent, int E, int n, const int* table, int max_pages,
                              int page_size, int H, int G, int dq, int dv, int wq, int wv, void* q, void* kp, void* vp,
                              cudaStream_t stream) {
  if (n <= 0) return 0;
  if (rd < 0 || rd % 2 || rd > dq || wq < dq || wv < dv || (rd > 0 && (!cos_t || !sin_t))) return -2;
  RAGGED;
  PAGED;
  const int wide = wq > wv ? wq : wv;
  if (dtype == 0 && dq % 8 == 0 && dv % 8 == 0 && wq % 8 == 0 && wv % 8 == 0 && rd % (inter ? 8 : 16) == 0 && wide <= 256 &&
      ldp % 8 == 0 && q_off % 8 == 0 && k_off % 8 == 0 && v_off % 8 == 0) {
    typedef __nv_bfloat16 bf;
#define VEC(L, I)                                                                                                           \
  launch_pdl(rope_norm_write_vec_kernel<L, I>, dim3(n), dim3(256), 0, stream, (const bf*)proj, ldp, q_off, k_off, v_off,     \
             (const bf*)qw, (const bf*)kw, cos_t, sin_t, rd, eps, norms, rb, pg, H, G, dq, dv, wq, wv, (bf*)q, (bf*)kp, (bf*)vp)
    const cudaError_t err = inter ? (wide <= 64 ? VEC(8, true) : wide <= 128 ? VEC(16, true) : VEC(32, true))
                                  : (wide <= 64 ? VEC(8, false) : wide <= 128 ? VEC(16, false) : VEC(32, false));
    return err == cudaSuccess ? 0 : -5;
#undef VEC
  }
  const long long warps = (long long)n * (H + 2 * G);
  const dim3 grid((unsigned)((warps + 7) / 8));
#define RUN(T)                                                                                                              \
  launch_pdl(rope_norm_write_kernel<T>, grid, dim3(256), 0, stream, (const T*)proj, ldp, q_off, k_off, v_off, (const T*)qw,  \
             (const T*)kw, cos_t, sin_t, rd, inter, eps, norms, rb, pg, H, G, dq, dv, wq, wv, (T*)q, (T*)kp, (T*)vp)
  return (dtype == 0 ? RUN(__nv_bfloat16) : RUN(float)) == cudaSuccess ? 0 : -5;
#undef RUN
}

// bias fp32 [H, far + 1] or null: what is added to the score of a key at distance min(i - j, far). window, chunk <= 0: none;
// cap > 0: scores become cap * tanh(score / cap). sink: one more score without a value in the sum of the weights (-inf: none), or
// sinks fp32 [H], one per head. gate T, rows ldg apart, or null: head h's output is multiplied by sigmoid(gate[row, h]).
// q T, rows ldq and heads q_heads apart. Cached heads are stored wq / wv wide; out T [n, ldo], head h at columns h * dv, times
// out_scale.
TB_API int tb_window_attn(int dtype, const void* q, long long ldq, int q_heads, const void* kp, const void* vp, const int* cu, const int* slot,
                          const int* pos0, const int* ent, int E, int n, const int* table, int max_pages, int page_size, int H,
                          int G, int dq, int dv, int wq, int wv, float scale, float cap, const float* bias, int far, int window,
                          int chunk, int keep, float sink, const float* sinks, const void* gate, long long ldg, float out_scale, void* out,
                          long long ldo, cudaStream_t stream) {
  if (n <= 0) return 0;
  if (G <= 0 || H % G || dv <= 0 || dq > 3000) return -2;
  RAGGED;
  PAGED;
  const long long warps = (long long)n * H;
  const dim3 grid((unsigned)((warps + 3) / 4), (dv + VREG * 32 - 1) / (VREG * 32));
#define RUN(T)                                                                                                              \
  return launch_pdl(window_attn_kernel<T>, grid, dim3(128), (size_t)4 * dq * 4, stream, (const T*)q, ldq, q_heads, (const T*)kp, \
                    (const T*)vp, rb, pg, H, G, dq, dv, wq, wv, scale, cap, bias, far, window, chunk, keep, sink, sinks,     \
                    (const T*)gate, ldg, out_scale, (T*)out, ldo) == cudaSuccess ? 0 : -5
  if (dtype == 0) RUN(__nv_bfloat16);
  RUN(float);
#undef RUN
}
