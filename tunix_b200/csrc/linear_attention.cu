// Gated linear attention over ragged batches: a matrix state S [dk, dv] per head whose rows decay by a factor of their own at
// every token, S <- diag(f) S + k v^T. The state lives in fp32 per slot; a sequence's first token starts from zero.
//
// What makes f, k and the read-out differs per mechanism (MODE):
//   BONUS (RWKV time mixing)  f = exp(-exp(z + c0)); o = (S_before + diag(c1) k v^T)^T q
//   LOWER (HGRN2)             f = c1 + (1 - c1) sigmoid(z + c0), k = 1 - f, q = silu(q); o = S^T q
//   ROOT (gated linear attention)  f = sigmoid(z + c0)^(1 / tau), q times a constant; o = S^T q
// with z fp32 from a projection and c0, c1 parameters per head and channel. Then every head's o is divided by its root mean
// square over dv, weighted (one weight for all heads or one per head), gated by silu if there is a gate, and scaled.
//
//   gla_step  : one token per entry. The state streams through registers once; norm and gate in the same launch. z may be given
//               as the product of a short row per token (a bottleneck) with a weight row per channel, which is formed here.
//   gla_chunk : portions of prompts, bf16, on tensor cores (below).
//   gla_seq   : token by token, any sizes, also 32-bit; head_norm after it.
//
// This file is compiled without fast-math: the same kernels serve the 32-bit mode.
#include "mma.cuh"
#include "precise.cuh"

using namespace tb;

namespace {

typedef __nv_bfloat16 bf;
enum Mode { BONUS = 0, LOWER = 1, ROOT = 2 };
__host__ __device__ constexpr bool has_keys(int mode) { return mode != LOWER; }      // else made from the gates
__host__ __device__ constexpr bool reads_after(int mode) { return mode != BONUS; }   // the read-out sees the token's own update

struct GlaArgs {
  const void *q, *k, *v, *gate;       // T [n, ld*], head h at columns h * dk or h * dv; k null with LOWER, gate may be null
  long long ldq, ldk, ldv, ldg;
  const float* z;                     // fp32 [n, ldz], or null (gla_step): z = w2 x
  long long ldz;
  const void* x;                      // T [n, ldx], the first `rank` columns
  const void* w2;                     // T [heads * dk, rank]
  long long ldx;
  int rank;
  const void *c0, *c1;                // T [heads * dk]; c1 not with ROOT
  float qscale, inv_tau;              // ROOT
  int heads, dk, dv;
  Ragged rb;
  float* S;                           // fp32 [slots, heads, dk, dv]
  // token shift: the last row of every portion is carried to the next one (gla_chunk, gla_seq; null: nothing to carry)
  const void* h;                      // T [n, D]
  float* carry;                       // fp32 [slots, D]
  int D;
  // output norm
  const void* nw;                     // T [dv] or [heads * dv]
  int per_head;
  float eps, out_scale;
  long long ldo;                      // row stride of the output
};

template <int MODE>
__device__ __forceinline__ void gates_exact(const GlaArgs& a, float z, float c0, float c1, float& f, float& k) {
  if (MODE == BONUS) {
    f = decay_exp(-expf(z + c0));
  } else if (MODE == ROOT) {
    f = decay_exp(log_sigmoid(z + c0) * a.inv_tau);
  } else {
    // near 1 the decay is rounded once: 1 - k
    k = (1.f - c1) * sigmoid(-(z + c0));
    f = k < 0.5f ? 1.f - k : c1 + (1.f - c1) * sigmoid(z + c0);
  }
}
// log2 f for bf16 models; bounded where f is zero in any sum of them. b0 = gates_offset(c0)
template <int MODE>
__device__ __forceinline__ float gates_offset(float c0) { return c0 * LOG2_E + (MODE == BONUS ? 0.5287663729448977f : 0.f); }   // + log2(log2 e)
template <int MODE>
__device__ __forceinline__ float gates_log2(const GlaArgs& a, float z, float b0, float c1, float& k) {
  const float y = fmaf(z, LOG2_E, b0), e = quick_exp2(fminf(y, 100.f));
  if (MODE == BONUS) return -fminf(e, 150.f);
  const float s = quick_rcp(1.f + e), r = 1.f - c1;    // sigmoid of the negative; e s: of the positive
  if (MODE == ROOT) return fmaxf((y > 0.f ? quick_log2_decay(s, 1.f) : y - quick_log2(1.f + e)) * a.inv_tau, -150.f);
  k = r * s;
  return quick_log2_decay(k, fmaf(r, e * s, c1));
}

template <typename T>
__device__ __forceinline__ float silu(float z) {
  return z * (sizeof(T) == 2 ? quick_sigmoid(z) : sigmoid(z));
}

// z of channel c for token t from its bottleneck row
template <typename T>
__device__ __forceinline__ float low_rank(const GlaArgs& a, int t, int c) {
  const T *x = static_cast<const T*>(a.x) + t * a.ldx, *w = static_cast<const T*>(a.w2) + (long long)c * a.rank;
  float z = 0.f;
  int r = 0;
  if (sizeof(T) == 2 && a.rank % 8 == 0 && ((uintptr_t)x & 15) == 0) {
    for (; r < a.rank; r += 8) {
      float xv[8], wv[8];
      load_v<8>(x + r, xv);
      load_v<8>(w + r, wv);
#pragma unroll
      for (int i = 0; i < 8; ++i) z += xv[i] * wv[i];
    }
  }
  for (; r < a.rank; ++r) z += to_f(x[r]) * to_f(w[r]);
  return z;
}

template <typename T>
__device__ __forceinline__ void carry_rows(const GlaArgs& a, int last, long long slot, int part, int parts) {
  if (!a.h) return;
  const T* h = static_cast<const T*>(a.h) + (long long)last * a.D;
  for (int c = part * blockDim.x + threadIdx.x; c < a.D; c += parts * blockDim.x) a.carry[slot * a.D + c] = to_f(h[c]);
}

// ------------------------------------------------------------------------------------------------ one token
constexpr int GT = 256;

template <typename T, int MODE, int V>
__global__ void __launch_bounds__(GT)
gla_step_kernel(const GlaArgs a, T* __restrict__ out) {
  extern __shared__ float sm[];
  const int dk = a.dk, dv = a.dv, hd = blockIdx.x, e = blockIdx.y, tid = threadIdx.x;
  float* qs = sm;                      // [dk]
  float* ks = qs + dk;                 // [dk]
  float* fs = ks + dk;                 // [dk]
  float* us = fs + dk;                 // [dk]
  float* part = us + dk;               // [R][dv]
  __shared__ float red[33];
  pdl_trigger();
  pdl_wait();
  const int p0 = a.rb.pos0[e];
  T* o = out + e * a.ldo + hd * dv;
  if (p0 < 0) {
    for (int c = tid; c < dv; c += GT) o[c] = from_f<T>(0.f);
    return;
  }
  const bool old = p0 > 0;
  float* S = a.S + ((long long)a.rb.slot[e] * a.heads + hd) * dk * dv;
  for (int d = tid; d < dk; d += GT) {
    const int c = hd * dk + d;
    const float c1 = MODE == ROOT ? 0.f : to_f(static_cast<const T*>(a.c1)[c]);
    float q = to_f(static_cast<const T*>(a.q)[e * a.ldq + c]), k = 0.f, f;
    if (has_keys(MODE)) k = to_f(static_cast<const T*>(a.k)[e * a.ldk + c]);
    if (MODE == LOWER) q = silu<T>(q);
    if (MODE == ROOT) q *= a.qscale;
    gates_exact<MODE>(a, a.z ? a.z[e * a.ldz + c] : low_rank<T>(a, e, c), to_f(static_cast<const T*>(a.c0)[c]), c1, f, k);
    qs[d] = q;
    ks[d] = k;
    fs[d] = f;
    us[d] = MODE == BONUS ? c1 : 0.f;
  }
  __syncthreads();
  const int C = dv / V, R = GT / C, r = tid / C, col = (tid - r * C) * V;
  if (r < R) {
    float v[V], acc[V];
    load_v<V>(static_cast<const T*>(a.v) + e * a.ldv + hd * dv + col, v);
#pragma unroll
    for (int i = 0; i < V; ++i) acc[i] = 0.f;
    constexpr int U = 4;
    for (int d0 = r; d0 < dk; d0 += U * R) {
      float s[U][V];
#pragma unroll
      for (int j = 0; j < U; ++j) {
        const int d = d0 + j * R;
        if (old && d < dk) {
          load_v<V>(S + (long long)d * dv + col, s[j]);
        } else {
#pragma unroll
          for (int i = 0; i < V; ++i) s[j][i] = 0.f;
        }
      }
#pragma unroll
      for (int j = 0; j < U; ++j) {
        const int d = d0 + j * R;
        if (d < dk) {
          const float k = ks[d], f = fs[d], q = qs[d], uk = us[d] * k;
#pragma unroll
          for (int i = 0; i < V; ++i) {
            if (!reads_after(MODE)) acc[i] += q * (s[j][i] + uk * v[i]);
            s[j][i] = f * s[j][i] + k * v[i];
            if (reads_after(MODE)) acc[i] += q * s[j][i];
          }
          store_v<V>(S + (long long)d * dv + col, s[j]);
        }
      }
    }
    store_v<V>(part + r * dv + col, acc);
  }
  __syncthreads();
  float ss = 0.f;
  for (int c = tid; c < dv; c += GT) {
    float x = 0.f;
    for (int j = 0; j < R; ++j) x += part[j * dv + c];
    part[c] = x;                       // row 0, read by this thread only
    ss += x * x;
  }
  ss = block_sum(ss, red);
  const float rstd = a.out_scale / sqrtf(ss / (float)dv + a.eps);
  for (int c = tid; c < dv; c += GT) {
    float x = part[c] * rstd * to_f(static_cast<const T*>(a.nw)[a.per_head ? hd * dv + c : c]);
    if (a.gate) x *= silu<T>(to_f(static_cast<const T*>(a.gate)[e * a.ldg + hd * dv + c]));
    o[c] = from_f<T>(x);
  }
}

// ------------------------------------------------------------------------------------------------ token by token
constexpr int SV = 32;          // value columns per CTA

template <typename T, int MODE>
__global__ void __launch_bounds__(GT)
gla_seq_kernel(const GlaArgs a, float* __restrict__ out) {
  extern __shared__ float sm[];
  const int dk = a.dk, dv = a.dv, e = blockIdx.z, hd = blockIdx.y, sl = blockIdx.x;
  float* S = sm;                       // [dk][SV]
  float* qs = S + dk * SV;             // [dk]
  float* ks = qs + dk;
  float* fs = ks + dk;
  float* us = fs + dk;
  float* vs = us + dk;                 // [SV]
  float* part = vs + SV;               // [8][SV]
  pdl_trigger();
  pdl_wait();
  const int t0 = a.rb.cu[e], t1 = a.rb.cu[e + 1], p0 = a.rb.pos0[e];
  const int c0 = sl * SV, nc = min(SV, dv - c0), tid = threadIdx.x, col = tid & 31, rg = tid >> 5;
  if (t0 >= t1) return;
  if (p0 < 0) {
    for (int t = t0; t < t1; ++t)
      if (tid < nc) out[((long long)t * a.heads + hd) * dv + c0 + tid] = 0.f;
    return;
  }
  const long long slot = a.rb.slot[e];
  float* Sg = a.S + (slot * a.heads + hd) * dk * dv + c0;
  for (int i = tid; i < dk * SV; i += GT) {
    const int d = i / SV, c = i - d * SV;
    S[i] = (p0 > 0 && c < nc) ? Sg[(long long)d * dv + c] : 0.f;
  }
  for (int t = t0; t < t1; ++t) {
    for (int d = tid; d < dk; d += GT) {
      const int c = hd * dk + d;
      const float c1 = MODE == ROOT ? 0.f : to_f(static_cast<const T*>(a.c1)[c]);
      float q = to_f(static_cast<const T*>(a.q)[t * a.ldq + c]), k = 0.f, f;
      if (has_keys(MODE)) k = to_f(static_cast<const T*>(a.k)[t * a.ldk + c]);
      if (MODE == LOWER) q = silu<T>(q);
      if (MODE == ROOT) q *= a.qscale;
      gates_exact<MODE>(a, a.z[t * a.ldz + c], to_f(static_cast<const T*>(a.c0)[c]), c1, f, k);
      qs[d] = q;
      ks[d] = k;
      fs[d] = f;
      us[d] = MODE == BONUS ? c1 * k : 0.f;
    }
    if (tid < SV) vs[tid] = tid < nc ? to_f(static_cast<const T*>(a.v)[t * a.ldv + hd * dv + c0 + tid]) : 0.f;
    __syncthreads();
    float acc = 0.f;
    const float v = vs[col];
    for (int d = rg; d < dk; d += GT / 32) {
      const float s = S[d * SV + col], n = fs[d] * s + ks[d] * v;
      acc += qs[d] * (MODE == BONUS ? s + us[d] * v : n);
      S[d * SV + col] = n;
    }
    part[rg * SV + col] = acc;
    __syncthreads();
    if (tid < nc) {
      float o = 0.f;
#pragma unroll
      for (int j = 0; j < GT / 32; ++j) o += part[j * SV + tid];
      out[((long long)t * a.heads + hd) * dv + c0 + tid] = o;
    }
  }
  __syncthreads();
  for (int i = tid; i < dk * SV; i += GT) {
    const int d = i / SV, c = i - d * SV;
    if (c < nc) Sg[(long long)d * dv + c] = S[i];
  }
  carry_rows<T>(a, t1 - 1, slot, hd * gridDim.x + sl, gridDim.x * gridDim.y);
}

// o fp32 [n, heads, dv] -> out T [n, heads * dv]: norm per head, weight, gate. One CTA per token, a warp per head.
template <typename T, int V>
__global__ void __launch_bounds__(256)
head_norm_kernel(const GlaArgs a, const float* __restrict__ o, T* __restrict__ out) {
  pdl_trigger();
  pdl_wait();
  const long long t = blockIdx.x;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5, dv = a.dv;
  const T* w = static_cast<const T*>(a.nw);
  const T* gate = a.gate ? static_cast<const T*>(a.gate) + t * a.ldg : nullptr;
  for (int hd = warp; hd < a.heads; hd += nw) {
    const float* x = o + (t * a.heads + hd) * dv;
    float ss = 0.f;
    for (int c = lane * V; c < dv; c += 32 * V) {
      float v[V];
      load_v<V>(x + c, v);
#pragma unroll
      for (int i = 0; i < V; ++i) ss += v[i] * v[i];
    }
    const float r = a.out_scale / sqrtf(warp_sum(ss) / (float)dv + a.eps);
    for (int c = lane * V; c < dv; c += 32 * V) {
      float v[V], ww[V], g[V];
      load_v<V>(x + c, v);
      load_v<V>(w + (a.per_head ? hd * dv + c : c), ww);
      if (gate) load_v<V>(gate + hd * dv + c, g);
#pragma unroll
      for (int i = 0; i < V; ++i) v[i] *= r * ww[i] * (gate ? silu<T>(g[i]) : 1.f);
      store_v<V>(out + t * a.ldo + hd * dv + c, v);
    }
  }
}

// ------------------------------------------------------------------------------------------------ portions, tensor cores
// A CTA owns 64 or 128 value columns of one head, 16 per warp, and walks its entry in blocks of 16 tokens. With L_t the sum of log f (in the code: of log2 f)
// from the block's start through token t, m its value at the block's middle and L at its end,
//   o_t = (q_t e^(L_t - m)) (diag(e^m) S) + sum_{s <= t} (q_t e^(L_t - m) . k_s e^(m - L_s)) v_s,
//   S' = diag(e^(L - m)) diag(e^m) S + sum_s (k_s e^(L - L_s)) v_s^T
// (BONUS reads S before the token: L_(t-1), s < t, and the current token weighs q . (c1 k)).
// S^T stays in fp32 accumulators [16 values, dk]: their layout is that of the B operand of q S, so the state is packed to bf16
// for the read-out without leaving registers. The updates k e^(L - L_s) go to the tensor cores as bf16 pairs hi + lo, v is
// bf16 and exact. Several blocks are prepared at once (TT tokens); every warp prepares one block (half of its channels at
// dk > 64), so a tile of tokens costs two barriers.
// The factors around m must stay finite: where some channel decays by more than e^-SAFE within half a block, the tile takes
// m = 0 and sums its weights directly, with e^(L_t - L_s) per pair and channel.
constexpr float SAFE = 70.f * LOG2_E;
constexpr int PPITCH = 48;

struct ChunkSmem {
  int tt, pitch, vpitch, q, k, z, v, Q, Ki, Kh, Kl, P, D, E, dg, ssq, total;
};
__host__ __device__ constexpr ChunkSmem chunk_smem(int KP, int warps) {
  ChunkSmem L{};
  L.tt = 16 * warps * 64 / KP;
  L.pitch = KP * 2 + 16;
  L.vpitch = 16 * warps * 2 + 16;
  L.q = 0;
  L.k = L.q + L.tt * L.pitch;
  L.z = L.k + L.tt * L.pitch;
  L.v = L.z + L.tt * KP * 4;
  L.Q = L.v + 2 * L.tt * L.vpitch;
  L.Ki = L.Q + L.tt * L.pitch;
  L.Kh = L.Ki + L.tt * L.pitch;
  L.Kl = L.Kh + L.tt * L.pitch;
  L.P = L.Kl + L.tt * L.pitch;
  L.D = L.P + (L.tt / 16) * 16 * PPITCH;
  L.E = L.D + (L.tt / 16) * KP * 4;
  L.dg = L.E + (L.tt / 16) * KP * 4;
  L.ssq = L.dg + (KP / 64) * L.tt * 4;
  L.total = L.ssq + warps * L.tt * 4;
  return L;
}

template <int KP, int MODE, int WARPS>
__global__ void __launch_bounds__(32 * WARPS)
gla_chunk_kernel(const GlaArgs a, float* __restrict__ raw, bf* __restrict__ out) {
  extern __shared__ __align__(16) uint8_t smem[];
  constexpr ChunkSmem M = chunk_smem(KP, WARPS);
  constexpr int TT = M.tt, SUBS = TT / 16, HALVES = KP / 64, KT = KP / 8, DV = 16 * WARPS, NT = 32 * WARPS, VPITCH = M.vpitch;
  const uint32_t sb = smem_u32(smem);
  float* Dd = reinterpret_cast<float*>(smem + M.D);     // [SUBS][KP] e^(L - m)
  float* De = reinterpret_cast<float*>(smem + M.E);     // [SUBS][KP] e^m
  float* Dg = reinterpret_cast<float*>(smem + M.dg);    // [HALVES][TT] q . (c1 k)
  float* Ssq = reinterpret_cast<float*>(smem + M.ssq);  // [WARPS][TT]
  const float* Z = reinterpret_cast<const float*>(smem + M.z);
  pdl_trigger();
  pdl_wait();
  const int dk = a.dk, dv = a.dv, e = blockIdx.z, hd = blockIdx.y, sl = blockIdx.x;
  const int p0 = a.rb.pos0[e], t0 = a.rb.cu[e], len = a.rb.cu[e + 1] - t0;
  if (p0 < 0 || len <= 0) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, li = lane >> 3, lr = lane & 7;
  const int g = lane >> 2, qd = 2 * (lane & 3);         // row and first column of this lane in an accumulator tile
  const int c0 = sl * DV, nc = min(DV, dv - c0), v0 = warp * 16;
  const bool active = v0 < nc;
  const long long slot = a.rb.slot[e];
  float* Sg = a.S + (slot * a.heads + hd) * dk * dv + c0;

  const bf* qg = static_cast<const bf*>(a.q) + (long long)t0 * a.ldq + hd * dk;
  const bf* kg = has_keys(MODE) ? static_cast<const bf*>(a.k) + (long long)t0 * a.ldk + hd * dk : nullptr;
  const bf* vg = static_cast<const bf*>(a.v) + (long long)t0 * a.ldv + hd * dv + c0;
  const float* zg = a.z + (long long)t0 * a.ldz + hd * dk;
  const bf* gg = a.gate ? static_cast<const bf*>(a.gate) + (long long)t0 * a.ldg + hd * dv + c0 : nullptr;
  uint32_t nw[2];                       // norm weights of this lane's columns
#pragma unroll
  for (int j = 0; j < 2; ++j) {
    const int c = c0 + v0 + j * 8 + 2 * (lane & 3);
    nw[j] = c < dv ? *reinterpret_cast<const uint32_t*>(static_cast<const bf*>(a.nw) + (a.per_head ? hd * dv + c : c)) : 0u;
  }
  auto load = [&](int tile) {
    const int at = tile * TT, rows = min(TT, len - at);
    for (int i = tid; i < TT * (KP / 8); i += NT) {
      const int r = i / (KP / 8), c = i % (KP / 8);
      const bool ok = r < rows && c * 8 < dk;
      cp_async16(sb + M.q + r * M.pitch + c * 16, qg + (ok ? (at + r) * a.ldq + c * 8 : 0), ok ? 16 : 0);
      if (has_keys(MODE)) cp_async16(sb + M.k + r * M.pitch + c * 16, kg + (ok ? (at + r) * a.ldk + c * 8 : 0), ok ? 16 : 0);
    }
    for (int i = tid; i < TT * (KP / 4); i += NT) {
      const int r = i / (KP / 4), c = i % (KP / 4);
      const bool ok = r < rows && c * 4 < dk;
      cp_async16(sb + M.z + r * (KP * 4) + c * 16, zg + (ok ? (at + r) * a.ldz + c * 4 : 0), ok ? 16 : 0);
    }
    const uint32_t vb = sb + M.v + (tile & 1) * TT * VPITCH;
    for (int i = tid; i < TT * (DV / 8); i += NT) {
      const int r = i / (DV / 8), c = i % (DV / 8);
      const bool ok = r < rows && c * 8 < nc;
      cp_async16(vb + r * VPITCH + c * 16, vg + (ok ? (at + r) * a.ldv + c * 8 : 0), ok ? 16 : 0);
    }
    cp_async_commit();
  };
  load(0);

  // S^T: tile j holds channels 8 j + qd, + 1 of values v0 + g (elements 0, 1) and v0 + g + 8 (2, 3)
  float S[KT][4];
#pragma unroll
  for (int j = 0; j < KT; ++j)
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int d = j * 8 + qd + (i & 1), v = v0 + g + (i >> 1) * 8;
      S[j][i] = (p0 > 0 && d < dk && v < nc) ? Sg[(long long)d * dv + v] : 0.f;
    }

  // the block and the two channels this lane prepares
  const int psub = warp / HALVES, pd = (warp % HALVES) * 64 + 2 * lane;
  float b0[2], b1[2];
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const bool ok = pd + i < dk;
    b0[i] = gates_offset<MODE>(ok ? to_f(static_cast<const bf*>(a.c0)[hd * dk + pd + i]) : 0.f);
    b1[i] = MODE == ROOT ? 0.f : ok ? to_f(static_cast<const bf*>(a.c1)[hd * dk + pd + i]) : (MODE == LOWER ? 1.f : 0.f);
  }

  const int tiles = (len + TT - 1) / TT;
  for (int tile = 0; tile < tiles; ++tile) {
    const int rows = min(TT, len - tile * TT);
    cp_async_wait<0>();
    __syncthreads();                    // the tile is in; nobody reads the last tile's operands any more
    // log2 f and k of this lane's two channels. Every factor below is the power of a sum of its own, never of a difference
    // of sums: where one token decays much, the others keep their accuracy.
    float l[16][2], h0[2] = {0.f, 0.f}, h1[2] = {0.f, 0.f};      // h0, h1: sums over the halves of the block
#pragma unroll
    for (int t = 0; t < 16; ++t) {
      const int row = psub * 16 + t;
      const float2 z = *reinterpret_cast<const float2*>(Z + row * KP + pd);
      float2 k;
      l[t][0] = gates_log2<MODE>(a, z.x, b0[0], b1[0], k.x);
      l[t][1] = gates_log2<MODE>(a, z.y, b0[1], b1[1], k.y);
      if (row >= rows) l[t][0] = l[t][1] = k.x = k.y = 0.f;
      // keys made from the gates take the place of z: only the sums stay in registers
      if (MODE == LOWER) *reinterpret_cast<float2*>(smem + M.z + (row * KP + pd) * 4) = k;
#pragma unroll
      for (int i = 0; i < 2; ++i) (t < 8 ? h0[i] : h1[i]) += l[t][i];
    }
    const bool direct = __syncthreads_or(fminf(fminf(h0[0], h1[0]), fminf(h0[1], h1[1])) < -SAFE);
    auto queries = [&](int row, float& q0, float& q1) {
      const uint32_t q2 = *reinterpret_cast<const uint32_t*>(smem + M.q + row * M.pitch + pd * 2);
      q0 = bf16_lo(q2);
      q1 = bf16_hi(q2);
      if (MODE == LOWER) { q0 = silu<bf>(q0); q1 = silu<bf>(q1); }
      if (MODE == ROOT) { q0 *= a.qscale; q1 *= a.qscale; }
    };
    auto keys = [&](int row) {                          // rows past the end hold zeros
      if (MODE == LOWER) return *reinterpret_cast<const float2*>(smem + M.z + (row * KP + pd) * 4);
      const uint32_t k2 = *reinterpret_cast<const uint32_t*>(smem + M.k + row * M.pitch + pd * 2);
      return make_float2(bf16_lo(k2), bf16_hi(k2));
    };
    // token t: read-out scaled by e^(log2 r), key by e^(log2 w)
    auto scaled = [&](int t, float r0, float r1, float w0, float w1) {
      const int row = psub * 16 + t;
      const uint32_t at = row * M.pitch + pd * 2;
      float q0, q1;
      queries(row, q0, q1);
      const float2 k = keys(row);
      *reinterpret_cast<uint32_t*>(smem + M.Q + at) = pack_bf16(q0 * quick_exp2(r0), q1 * quick_exp2(r1));
      *reinterpret_cast<uint32_t*>(smem + M.Ki + at) = pack_bf16(k.x * quick_exp2(w0), k.y * quick_exp2(w1));
    };
    float end0 = 0.f, end1 = 0.f;                       // sums from the token after t to the block's end
#pragma unroll
    for (int t = 15; t >= 0; --t) {
      const uint32_t at = (psub * 16 + t) * M.pitch + pd * 2;
      const float2 k = keys(psub * 16 + t);
      bf hi0, hi1, lo0, lo1;
      split_bf16(k.x * quick_exp2(end0), hi0, lo0);
      split_bf16(k.y * quick_exp2(end1), hi1, lo1);
      *reinterpret_cast<__nv_bfloat162*>(smem + M.Kh + at) = __halves2bfloat162(hi0, hi1);
      *reinterpret_cast<__nv_bfloat162*>(smem + M.Kl + at) = __halves2bfloat162(lo0, lo1);
      end0 += l[t][0];
      end1 += l[t][1];
    }
    if (MODE == BONUS) {
      float dg[16];
#pragma unroll
      for (int t = 0; t < 16; ++t) {
        float q0, q1;
        queries(psub * 16 + t, q0, q1);
        const float2 k = keys(psub * 16 + t);
        dg[t] = q0 * b1[0] * k.x + q1 * b1[1] * k.y;
      }
      // 16 sums over the warp: halve the values a lane holds at every step
#pragma unroll
      for (int w = 8; w >= 1; w >>= 1) {
#pragma unroll
        for (int t = 0; t < w; ++t) {
          const float mine = (lane & w) ? dg[t + w] : dg[t], other = (lane & w) ? dg[t] : dg[t + w];
          dg[t] = mine + __shfl_xor_sync(0xffffffffu, other, w);
        }
      }
      dg[0] += __shfl_xor_sync(0xffffffffu, dg[0], 16);
      if (lane < 16) Dg[(warp % HALVES) * TT + psub * 16 + lane] = dg[0];
    }
    if (!direct) {
      float c0s = 0.f, c1s = 0.f;                       // from the token after t to the middle
#pragma unroll
      for (int t = 7; t >= 0; --t) {
        const float n0 = c0s + l[t][0], n1 = c1s + l[t][1];
        scaled(t, reads_after(MODE) ? -c0s : -n0, reads_after(MODE) ? -c1s : -n1, c0s, c1s);
        c0s = n0;
        c1s = n1;
      }
      c0s = c1s = 0.f;                                  // from the middle to the token
#pragma unroll
      for (int t = 8; t < 16; ++t) {
        const float n0 = c0s + l[t][0], n1 = c1s + l[t][1];
        scaled(t, reads_after(MODE) ? n0 : c0s, reads_after(MODE) ? n1 : c1s, -n0, -n1);
        c0s = n0;
        c1s = n1;
      }
    } else {
      // read-outs from the block's start; sums, queries and keys of the whole tile for the weights below
      float c0s = 0.f, c1s = 0.f;
#pragma unroll
      for (int t = 0; t < 16; ++t) {
        const int row = psub * 16 + t;
        const uint32_t at = row * M.pitch + pd * 2;
        const float n0 = c0s + l[t][0], n1 = c1s + l[t][1];
        float q0, q1;
        queries(row, q0, q1);
        const float2 k = keys(row);
        *reinterpret_cast<uint32_t*>(smem + M.Q + at) = pack_bf16(q0 * quick_exp2(reads_after(MODE) ? n0 : c0s), q1 * quick_exp2(reads_after(MODE) ? n1 : c1s));
        *reinterpret_cast<float2*>(smem + M.z + (row * KP + pd) * 4) = make_float2(n0, n1);
        *reinterpret_cast<uint32_t*>(smem + M.k + at) = pack_bf16(k.x, k.y);
        *reinterpret_cast<uint32_t*>(smem + M.q + at) = pack_bf16(q0, q1);
        c0s = n0;
        c1s = n1;
      }
    }
    *reinterpret_cast<float2*>(De + psub * KP + pd) = direct ? make_float2(1.f, 1.f) : make_float2(quick_exp2(h0[0]), quick_exp2(h0[1]));
    *reinterpret_cast<float2*>(Dd + psub * KP + pd) = direct ? make_float2(quick_exp2(end0), quick_exp2(end1)) : make_float2(quick_exp2(h1[0]), quick_exp2(h1[1]));
    __syncthreads();
    if (direct) {                       // one thread per weight
      for (int i = tid; i < SUBS * 256; i += NT) {
        const int sub = i >> 8, t = (i >> 4) & 15, s = i & 15, rt = sub * 16 + t, rs = sub * 16 + s;
        float p = 0.f;
        if (MODE == BONUS && s == t) {
#pragma unroll
          for (int h = 0; h < HALVES; ++h) p += Dg[h * TT + rt];
        } else if (s <= t) {
          const bf* q = reinterpret_cast<const bf*>(smem + M.q + rt * M.pitch);
          const bf* k = reinterpret_cast<const bf*>(smem + M.k + rs * M.pitch);
          const float *Lt = Z + (MODE == BONUS ? rt - 1 : rt) * KP, *Ls = Z + rs * KP;
          for (int d = 0; d < dk; ++d) p += to_f(q[d]) * to_f(k[d]) * quick_exp2(Lt[d] - Ls[d]);
        }
        *reinterpret_cast<bf*>(smem + M.P + (sub * 16 + t) * PPITCH + s * 2) = __float2bfloat16(p);
      }
      __syncthreads();
    }
    if (tile + 1 < tiles) load(tile + 1);

    // the gates of this lane's outputs, on their way while the products run
    uint32_t gate[SUBS][2][2];
    if (active && out != nullptr && a.gate) {
#pragma unroll
      for (int sub = 0; sub < SUBS; ++sub)
#pragma unroll
        for (int h = 0; h < 2; ++h)
#pragma unroll
          for (int j = 0; j < 2; ++j) {
            const int r = sub * 16 + g + h * 8, c = v0 + j * 8 + qd;
            gate[sub][h][j] = r < rows && c < nc ? __ldg(reinterpret_cast<const uint32_t*>(gg + (tile * TT + r) * a.ldg + c)) : 0u;
          }
    }
    float O[SUBS][2][4];
    const uint32_t vb = sb + M.v + (tile & 1) * TT * VPITCH;
    if (active) {
#pragma unroll
      for (int sub = 0; sub < SUBS; ++sub) {
        float P[2][4];
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
          for (int i = 0; i < 4; ++i) O[sub][j][i] = P[j][i] = 0.f;
        const uint32_t r_nt = sub * 16 + (li & 1) * 8 + lr, r_b = sub * 16 + (li >> 1) * 8 + lr;
#pragma unroll
        for (int ks = 0; ks < KP / 16; ++ks) {
          uint32_t q[4], k[4];
          ldsm_x4(q, sb + M.Q + r_nt * M.pitch + (ks * 2 + (li >> 1)) * 16);
          if (!direct) {
            ldsm_x4(k, sb + M.Ki + r_b * M.pitch + (ks * 2 + (li & 1)) * 16);
            mma_16816(P[0], q, k[0], k[1]);
            mma_16816(P[1], q, k[2], k[3]);
          }
          const float2 f0 = *reinterpret_cast<const float2*>(De + sub * KP + ks * 16 + qd);
          const float2 f1 = *reinterpret_cast<const float2*>(De + sub * KP + ks * 16 + 8 + qd);
          float (&s0)[4] = S[2 * ks], (&s1)[4] = S[2 * ks + 1];
          s0[0] *= f0.x; s0[1] *= f0.y; s0[2] *= f0.x; s0[3] *= f0.y;
          s1[0] *= f1.x; s1[1] *= f1.y; s1[2] *= f1.x; s1[3] *= f1.y;
          mma_16816(O[sub][0], q, pack_bf16(s0[0], s0[1]), pack_bf16(s1[0], s1[1]));
          mma_16816(O[sub][1], q, pack_bf16(s0[2], s0[3]), pack_bf16(s1[2], s1[3]));
        }
        uint32_t ap[4], bv[4], av[4];
        if (direct) {
          ldsm_x4(ap, sb + M.P + r_nt * PPITCH + (li >> 1) * 16);
        } else {
#pragma unroll
          for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int i = 0; i < 4; ++i) {
              const int t = g + (i >> 1) * 8, s = j * 8 + qd + (i & 1);
              if (s > t) P[j][i] = 0.f;
              if (MODE == BONUS && s == t) {
                P[j][i] = Dg[sub * 16 + t];
                if (HALVES == 2) P[j][i] += Dg[TT + sub * 16 + t];
              }
            }
          ap[0] = pack_bf16(P[0][0], P[0][1]);
          ap[1] = pack_bf16(P[0][2], P[0][3]);
          ap[2] = pack_bf16(P[1][0], P[1][1]);
          ap[3] = pack_bf16(P[1][2], P[1][3]);
        }
        ldsm_x4_t(bv, vb + r_nt * VPITCH + (v0 / 8 + (li >> 1)) * 16);
        mma_16816(O[sub][0], ap, bv[0], bv[1]);
        mma_16816(O[sub][1], ap, bv[2], bv[3]);
        ldsm_x4_t(av, vb + r_b * VPITCH + (v0 / 8 + (li & 1)) * 16);
#pragma unroll
        for (int j = 0; j < KT; j += 2) {
          const float2 d0 = *reinterpret_cast<const float2*>(Dd + sub * KP + j * 8 + qd);
          const float2 d1 = *reinterpret_cast<const float2*>(Dd + sub * KP + j * 8 + 8 + qd);
          S[j][0] *= d0.x; S[j][1] *= d0.y; S[j][2] *= d0.x; S[j][3] *= d0.y;
          S[j + 1][0] *= d1.x; S[j + 1][1] *= d1.y; S[j + 1][2] *= d1.x; S[j + 1][3] *= d1.y;
          uint32_t k[4];
          ldsm_x4_t(k, sb + M.Kh + r_nt * M.pitch + (j + (li >> 1)) * 16);
          mma_16816(S[j], av, k[0], k[1]);
          mma_16816(S[j + 1], av, k[2], k[3]);
          ldsm_x4_t(k, sb + M.Kl + r_nt * M.pitch + (j + (li >> 1)) * 16);
          mma_16816(S[j], av, k[0], k[1]);
          mma_16816(S[j + 1], av, k[2], k[3]);
        }
      }
    }
    // outputs: of a whole head normed and gated here, of a slice in fp32 for head_norm
    if (out != nullptr) {
#pragma unroll
      for (int sub = 0; sub < SUBS; ++sub)
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          float s = 0.f;
          if (active) {
#pragma unroll
            for (int j = 0; j < 2; ++j) s += O[sub][j][2 * h] * O[sub][j][2 * h] + O[sub][j][2 * h + 1] * O[sub][j][2 * h + 1];
          }
          s += __shfl_xor_sync(0xffffffffu, s, 1);
          s += __shfl_xor_sync(0xffffffffu, s, 2);
          if ((lane & 3) == 0) Ssq[warp * TT + sub * 16 + g + h * 8] = s;
        }
      __syncthreads();
    }
    if (active) {
#pragma unroll
      for (int sub = 0; sub < SUBS; ++sub)
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          const int r = sub * 16 + g + h * 8;
          if (r >= rows) continue;
          const long long t = t0 + tile * TT + r;
          float rstd = 1.f;
          if (out != nullptr) {
            float s = 0.f;
#pragma unroll
            for (int w = 0; w < WARPS; ++w) s += Ssq[w * TT + r];
            rstd = a.out_scale * rsqrtf(s / (float)dv + a.eps);
          }
#pragma unroll
          for (int j = 0; j < 2; ++j) {
            const int c = c0 + v0 + j * 8 + qd;
            if (c >= dv) continue;                      // dv is a multiple of 8
            const float x0 = O[sub][j][2 * h], x1 = O[sub][j][2 * h + 1];
            if (out == nullptr) {
              *reinterpret_cast<float2*>(raw + (t * a.heads + hd) * dv + c) = make_float2(x0, x1);
            } else {
              float y0 = x0 * rstd * bf16_lo(nw[j]), y1 = x1 * rstd * bf16_hi(nw[j]);
              if (a.gate) {
                y0 *= silu<bf>(bf16_lo(gate[sub][h][j]));
                y1 *= silu<bf>(bf16_hi(gate[sub][h][j]));
              }
              *reinterpret_cast<uint32_t*>(out + t * a.ldo + hd * dv + c) = pack_bf16(y0, y1);
            }
          }
        }
    }
  }
#pragma unroll
  for (int j = 0; j < KT; ++j)
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int d = j * 8 + qd + (i & 1), v = v0 + g + (i >> 1) * 8;
      if (d < dk && v < nc) Sg[(long long)d * dv + v] = S[j][i];
    }
  carry_rows<bf>(a, t0 + len - 1, slot, hd * gridDim.x + sl, gridDim.x * gridDim.y);
}

template <int KP, int MODE, int WARPS>
int launch_chunk(const GlaArgs& a, float* raw, bf* out, cudaStream_t stream) {
  constexpr int smem = chunk_smem(KP, WARPS).total, DV = 16 * WARPS;
  bf* o = a.dv <= DV ? out : nullptr;
  static DeviceOnce once;
  if (once.first() &&
      (cudaFuncSetAttribute(gla_chunk_kernel<KP, MODE, WARPS>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess ||
       // two of the smaller CTAs fit an SM only if the launches around them leave it this carveout
       cudaFuncSetAttribute(gla_chunk_kernel<KP, MODE, WARPS>, cudaFuncAttributePreferredSharedMemoryCarveout,
                            cudaSharedmemCarveoutMaxShared) != cudaSuccess)) return -5;
  const dim3 grid((a.dv + DV - 1) / DV, a.heads, a.rb.E);
  return launch_pdl(gla_chunk_kernel<KP, MODE, WARPS>, grid, dim3(32 * WARPS), smem, stream, a, raw, o) == cudaSuccess ? 0 : -5;
}

template <typename T, int MODE, int V>
int launch_step(const GlaArgs& a, T* out, cudaStream_t stream) {
  const int R = GT / (a.dv / V);
  const size_t smem = ((size_t)4 * a.dk + (size_t)R * a.dv) * 4;
  static DeviceOnce once;
  if (smem > 200 * 1024) return -2;
  if (once.first() &&
      cudaFuncSetAttribute(gla_step_kernel<T, MODE, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024) != cudaSuccess) return -5;
  return launch_pdl(gla_step_kernel<T, MODE, V>, dim3(a.heads, a.rb.E), dim3(GT), smem, stream, a, out) == cudaSuccess ? 0 : -5;
}

bool aligned(const void* p, int bytes) { return ((uintptr_t)p & (bytes - 1)) == 0; }

template <typename T, int MODE>
int run(const GlaArgs& a, float* raw, T* out, int one, int chunked, cudaStream_t stream) {
  if (one) {
    const bool vec = a.dv % 4 == 0 && a.ldv % 4 == 0 && a.dk % 4 == 0 && aligned(a.v, 4 * sizeof(T));
    if (vec && a.dv <= 4 * GT) return launch_step<T, MODE, 4>(a, out, stream);
    if (a.dv <= GT) return launch_step<T, MODE, 1>(a, out, stream);
  }
  if (!a.z || !raw) return -2;
  bool sliced = false;
  if constexpr (sizeof(T) == 2) {
    if (chunked && !one && a.dk <= 128 && a.dk % 8 == 0 && a.dv % 8 == 0 && a.ldq % 8 == 0 && a.ldv % 8 == 0 && a.ldz % 4 == 0 &&
        (!has_keys(MODE) || (a.ldk % 8 == 0 && aligned(a.k, 16))) && a.ldg % 2 == 0 && a.ldo % 2 == 0 && aligned(a.q, 16) &&
        aligned(a.v, 16) && aligned(a.z, 16) && aligned(a.gate, 4) && aligned(out, 4)) {
      const bool wide = a.dv > 64;
      const int rc = a.dk <= 64 ? (wide ? launch_chunk<64, MODE, 8>(a, raw, out, stream) : launch_chunk<64, MODE, 4>(a, raw, out, stream))
                                : (wide ? launch_chunk<128, MODE, 8>(a, raw, out, stream) : launch_chunk<128, MODE, 4>(a, raw, out, stream));
      if (rc || a.dv <= 128) return rc;
      sliced = true;
    }
  }
  if (!sliced) {
    const size_t smem = ((size_t)a.dk * (SV + 4) + SV + (GT / 32) * SV) * 4;
    static DeviceOnce once;
    if (smem > 220 * 1024) return -2;
    if (once.first() &&
        cudaFuncSetAttribute(gla_seq_kernel<T, MODE>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024) != cudaSuccess) return -5;
    const dim3 grid((a.dv + SV - 1) / SV, a.heads, a.rb.E);
    if (launch_pdl(gla_seq_kernel<T, MODE>, grid, dim3(GT), smem, stream, a, raw) != cudaSuccess) return -5;
  }
  const bool vec = a.dv % 4 == 0 && a.ldg % 4 == 0 && a.ldo % 4 == 0 && aligned(a.gate, 4 * sizeof(T)) && aligned(out, 4 * sizeof(T));
  const dim3 grid(a.rb.n);
  const cudaError_t err = vec ? launch_pdl(head_norm_kernel<T, 4>, grid, dim3(256), 0, stream, a, (const float*)raw, out)
                              : launch_pdl(head_norm_kernel<T, 1>, grid, dim3(256), 0, stream, a, (const float*)raw, out);
  return err == cudaSuccess ? 0 : -5;
}

}  // namespace

// mode: 0 BONUS, 1 LOWER, 2 ROOT. q, k [n, heads * dk], v, gate [n, heads * dv] (row strides ld*; k null with LOWER, gate may be
// null), z fp32 [n, heads * dk] with row stride ldz, or (with `one`) null: x T [n, rank] with row stride ldx times w2 T
// [heads * dk, rank]; c0, c1 T [heads * dk] (c1 null with ROOT); qscale, inv_tau: ROOT's constants; S fp32 [slots, heads, dk, dv].
// h T [n, D] / carry fp32 [slots, D] (or null): last rows of portions kept for the token shift (not with `one`).
// nw T [dv], or [heads * dv] with per_head; raw fp32 [n, heads * dv] workspace; out T [n, heads * dv] with row stride ldo, times
// out_scale.
// one: every entry is one token. chunked: bf16 portions take the tensor-core form where the sizes allow.
TB_API int tb_gated_linear(int dtype, int mode, const void* q, long long ldq, const void* k, long long ldk, const void* v,
                           long long ldv, const void* gate, long long ldg, const float* z, long long ldz, const void* x,
                           long long ldx, const void* w2, int rank, const void* c0, const void* c1, float qscale, float inv_tau,
                           const int* cu, const int* slot, const int* pos0, const int* ent, int E, int n,
                           int heads, int dk, int dv, float* S, const void* h, float* carry, int D, const void* nw, int per_head,
                           float eps, float out_scale, float* raw, void* out, long long ldo, int one, int chunked,
                           cudaStream_t stream) {
  if (n <= 0 || E <= 0) return 0;
  if (heads <= 0 || dk <= 0 || dv <= 0 || E > 65535 || heads > 65535 || mode < BONUS || mode > ROOT || (has_keys(mode) && !k) ||
      (mode != ROOT && !c1) || (!z && (!one || !x || !w2 || rank <= 0))) return -2;
  GlaArgs a{q, k, v, gate, ldq, ldk, ldv, ldg, z, ldz, x, w2, ldx, rank, c0, c1, qscale, inv_tau, heads, dk, dv,
            Ragged{cu, slot, pos0, ent, E, n}, S, h, carry, D, nw, per_head, eps, out_scale, ldo};
#define GL(T) (mode == BONUS ? run<T, BONUS>(a, raw, (T*)out, one, chunked, stream) : mode == LOWER \
                   ? run<T, LOWER>(a, raw, (T*)out, one, chunked, stream) : run<T, ROOT>(a, raw, (T*)out, one, chunked, stream))
  return dtype == 0 ? GL(bf) : GL(float);
#undef GL
}
