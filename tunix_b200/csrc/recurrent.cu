// Recurrent mixers over ragged batches: state lives in fp32 per slot, a sequence's first token starts from zero.
//
//   rglru_*  : real-gated linear recurrent unit behind a short causal convolution (Griffin's recurrent block):
//              u = conv(x), r = sigmoid(Ra u + ba), i = sigmoid(Ri u + bi) with block-diagonal Ra, Ri,
//              log a = -8 r softplus(lam), S <- a S + sqrt(1 - a^2) i u, output S * gelu(y).
//              The convolution's past inputs are a ring of `taps` rows per slot, indexed by position modulo taps: a
//              step never reads the row it writes.
//   mlstm_*  : matrix memory with exponential input gate and running maximum m (from 0):
//              m' = max(f + m, i); S <- e^(f+m-m') S + e^(i-m') k v^T; n likewise with k;
//              o = S^T q / (max(|n . q|, e^-m') + 1e-6).
//              The value columns are cut into slices of MV; every slice keeps its own copy of n and m, so that the CTAs
//              of a head need not meet.
//
// This file is compiled without fast-math: the same kernels serve the 32-bit mode.
#include "mma.cuh"
#include "precise.cuh"

using namespace tb;

namespace {

// ------------------------------------------------------------------------------------------------ RG-LRU
// u[t, c] = bias[c] + sum_j w[c, K-1-j] * x[position - j]; x is the columns x_off.. of the projection rows.
template <typename T>
__global__ void rglru_conv_kernel(const T* __restrict__ proj, long long ldp, int x_off, const T* __restrict__ w,
                                  const T* __restrict__ bias, const float* __restrict__ ring, Ragged rb, int W, int K,
                                  T* __restrict__ u) {
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.y;
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c >= W) return;
  const int e = rb.ent[t], p0 = rb.pos0[e];
  if (p0 < 0) { u[(long long)t * W + c] = from_f<T>(0.f); return; }
  const int first = rb.cu[e], p = p0 + t - first;
  float acc = to_f(bias[c]);
  for (int j = 0; j < K && j <= p; ++j) {
    const int s = t - j;
    const float v = s >= first ? to_f(proj[(long long)s * ldp + x_off + c])
                               : ring[((long long)rb.slot[e] * K + (p - j) % K) * W + c];
    acc += to_f(w[(long long)c * K + K - 1 - j]) * v;
  }
  u[(long long)t * W + c] = from_f<T>(acc);
}

// a = exp(-8 r softplus(lam)) and b = sqrt(1 - a^2) i u per channel, from the block-diagonal gates. CTA: one block,
// GT tokens, GC output channels.
constexpr int GT = 16, GC = 32;
template <typename T>
__global__ void __launch_bounds__(128)
rglru_gates_kernel(const T* __restrict__ u, const T* __restrict__ ra, const T* __restrict__ ba, const T* __restrict__ ri,
                   const T* __restrict__ bi, const T* __restrict__ lam, int n, int W, int bs, float* __restrict__ A,
                   float* __restrict__ B) {
  extern __shared__ float us[];           // [GT][bs]
  pdl_trigger();
  pdl_wait();
  const int blk = blockIdx.y, t0 = blockIdx.z * GT, c0 = blockIdx.x * GC;
  const int nt = min(GT, n - t0);
  for (int i = threadIdx.x; i < GT * bs; i += blockDim.x) {
    const int t = i / bs, k = i - t * bs;
    us[i] = t < nt ? to_f(u[(long long)(t0 + t) * W + (long long)blk * bs + k]) : 0.f;
  }
  __syncthreads();
  const int col = c0 + (threadIdx.x & 31);           // channel inside the block
  const int tg = threadIdx.x >> 5;                   // 4 groups of GT / 4 tokens
  if (col >= bs) return;
  const int ch = blk * bs + col;
  const T* war = ra + ((long long)blk * bs + col) * bs;
  const T* wir = ri + ((long long)blk * bs + col) * bs;
  float sr[GT / 4], si[GT / 4];
#pragma unroll
  for (int j = 0; j < GT / 4; ++j) { sr[j] = to_f(ba[ch]); si[j] = to_f(bi[ch]); }
  for (int k = 0; k < bs; ++k) {
    const float wr = to_f(war[k]), wi = to_f(wir[k]);
#pragma unroll
    for (int j = 0; j < GT / 4; ++j) {
      const float v = us[(tg * (GT / 4) + j) * bs + k];
      sr[j] += wr * v;
      si[j] += wi * v;
    }
  }
  const float sp = softplus(to_f(lam[ch]));
#pragma unroll
  for (int j = 0; j < GT / 4; ++j) {
    const int t = tg * (GT / 4) + j;
    if (t >= nt) continue;
    const float la = -8.f * sigmoid(sr[j]) * sp;
    const long long o = (long long)(t0 + t) * W + ch;
    A[o] = decay_exp(la);
    B[o] = sqrtf(-expm1f(2.f * la)) * sigmoid(si[j]) * us[t * bs + col];
  }
}

// One thread per (entry, channel): the recurrence over the entry's tokens, the output gate, the new state and ring rows.
template <typename T>
__global__ void rglru_scan_kernel(const float* __restrict__ A, const float* __restrict__ B, const T* __restrict__ proj,
                                  long long ldp, int x_off, int y_off, Ragged rb, int W, int K, float* __restrict__ state,
                                  float* __restrict__ ring, T* __restrict__ out) {
  pdl_trigger();
  pdl_wait();
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  const int e = blockIdx.y;
  if (c >= W) return;
  const int t0 = rb.cu[e], t1 = rb.cu[e + 1], p0 = rb.pos0[e];
  if (p0 < 0) {
    for (int t = t0; t < t1; ++t) out[(long long)t * W + c] = from_f<T>(0.f);
    return;
  }
  const long long sl = rb.slot[e];
  float s = p0 > 0 ? state[sl * W + c] : 0.f;
  for (int t = t0; t < t1; ++t) {
    const long long o = (long long)t * W + c;
    s = A[o] * s + B[o];
    out[o] = from_f<T>(s * gelu_tanh(to_f(proj[(long long)t * ldp + y_off + c])));
  }
  if (t1 > t0) state[sl * W + c] = s;
  for (int t = max(t0, t1 - K); t < t1; ++t)
    ring[(sl * K + (p0 + t - t0) % K) * W + c] = to_f(proj[(long long)t * ldp + x_off + c]);
}

// ---- bf16, prompt portions: the gates on tensor cores, the recurrence cut into tiles of LT tokens
// A tile is LT consecutive tokens of one entry (tile_t0 / tile_ent from the host). The gate kernel leaves, per token and
// channel, the tile-local recurrence h (from zero) and the running product p of the decays; a small kernel chains the
// tiles' last rows; the last kernel adds p * carry and applies the output gate. Nothing waits on another block.
constexpr int LT = 64;          // tokens per tile
constexpr int LC = 32;          // channels per CTA of the gate kernel
constexpr int LTPC = 8;         // consecutive tiles per CTA: the weights stay in shared memory

struct Tiles {
  const int* t0;      // [tiles] first token of the tile
  const int* ent;     // [tiles] its entry
  int count;
};

// u [n, W] -> H, P fp32 [n, W], and the tiles' last rows in LH, LP fp32 [tiles, W]
template <int KP>       // block size rounded up to 16, or 0 for a run-time value
__global__ void __launch_bounds__(256, 2)
rglru_tile_kernel(const __nv_bfloat16* __restrict__ u, const __nv_bfloat16* __restrict__ ra,
                  const __nv_bfloat16* __restrict__ ba, const __nv_bfloat16* __restrict__ ri,
                  const __nv_bfloat16* __restrict__ bi, const __nv_bfloat16* __restrict__ lam, Ragged rb, Tiles tl, int W,
                  int bs, float* __restrict__ H, float* __restrict__ P, float* __restrict__ LH, float* __restrict__ LP) {
  extern __shared__ __align__(16) uint8_t smem[];
  const int kp = KP > 0 ? KP : (bs + 15) & ~15;         // contraction length, zero-padded
  const int pitch = kp * 2 + 16;                        // bytes per row
  const int ubytes = max(LT * pitch, 2 * LT * (LC + 1) * 4);   // one buffer: a u tile, later the scan's a and b
  uint8_t* Ws = smem + 2 * ubytes;                      // [2 * LC] rows: LC of ra, LC of ri
  constexpr int SEGS = 256 / LC, SEG = LT / SEGS;              // segments of a tile in the scan, tokens per segment
  __shared__ float segA[SEGS][LC], segB[SEGS][LC];
  __shared__ float s_sp[LC], s_ba[LC], s_bi[LC];
  pdl_trigger();
  pdl_wait();
  const int per_blk = (bs + LC - 1) / LC;
  const int blk = blockIdx.x / per_blk, o0 = (blockIdx.x - blk * per_blk) * LC;    // channels o0.. of block blk
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, li = lane >> 3, lr = lane & 7;
  const int chunks = kp / 8;
  const uint32_t ws = smem_u32(Ws);
  const int tile_end = min(tl.count, ((int)blockIdx.y + 1) * LTPC);
  const GridWalk walk(tid, 256, chunks);
  auto load_u = [&](int tile) {
    const int t0 = tl.t0[tile], nt = min(LT, rb.cu[tl.ent[tile] + 1] - t0);
    const uint32_t dst = smem_u32(smem) + (tile & 1) * ubytes;
    const __nv_bfloat16* src = u + (long long)t0 * W + blk * bs;
    for (GridWalk g = walk; g.r < LT; g.next()) {
      const bool ok = g.r < nt && g.c * 8 < bs;
      cp_async16(dst + g.r * pitch + g.c * 16, ok ? src + (long long)g.r * W + g.c * 8 : u, ok ? 16 : 0);
    }
    cp_async_commit();
  };
  for (int i = tid; i < 2 * LC * chunks; i += 256) {
    const int r = i / chunks, c = i - r * chunks;
    const int o = o0 + (r & (LC - 1));
    const bool ok = o < bs && c * 8 < bs;
    const __nv_bfloat16* src = (r < LC ? ra : ri) + ((long long)blk * bs + (ok ? o : 0)) * bs + (ok ? c * 8 : 0);
    cp_async16(ws + r * pitch + c * 16, src, ok ? 16 : 0);
  }
  load_u(blockIdx.y * LTPC);                            // one group: the weights and the first tile
  if (tid < LC && o0 + tid < bs) {
    const int ch = blk * bs + o0 + tid;
    s_sp[tid] = -8.f * softplus(to_f(lam[ch]));
    s_ba[tid] = to_f(ba[ch]);
    s_bi[tid] = to_f(bi[ch]);
  }
  for (int tile = blockIdx.y * LTPC; tile < tile_end; ++tile) {
    const int e = tl.ent[tile], t0 = tl.t0[tile];
    const int nt = min(LT, rb.cu[e + 1] - t0);
    uint8_t* Us = smem + (tile & 1) * ubytes;
    const uint32_t us = smem_u32(Us);
    float* As = reinterpret_cast<float*>(Us);           // [LT][LC + 1], once the tile has been consumed
    float* Bs = As + LT * (LC + 1);
    cp_async_wait<0>();
    __syncthreads();                                    // the tile is in; the other buffer is done with
    if (tile + 1 < tile_end) load_u(tile + 1);
    // warps: 4 rows of 16 tokens x 2 halves of 16 channels; both gates of a channel in the same thread
    const int m0 = (warp & 3) * 16, n0 = (warp >> 2) * 16;
    float r[2][4], g[2][4];
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int q = 0; q < 4; ++q) r[j][q] = g[j][q] = 0.f;
    const uint32_t ua = us + (m0 + (li & 1) * 8 + lr) * pitch + (li >> 1) * 16;
    const uint32_t wa = ws + (n0 + (li >> 1) * 8 + lr) * pitch + (li & 1) * 16;
#pragma unroll 4
    for (int ks = 0; ks < kp / 16; ++ks) {
      uint32_t a[4], w0[4], w1[4];
      ldsm_x4(a, ua + ks * 32);
      ldsm_x4(w0, wa + ks * 32);
      ldsm_x4(w1, wa + LC * pitch + ks * 32);
      mma_16816(r[0], a, w0[0], w0[1]);
      mma_16816(r[1], a, w0[2], w0[3]);
      mma_16816(g[0], a, w1[0], w1[1]);
      mma_16816(g[1], a, w1[2], w1[3]);
    }
    float bvs[2][4];
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        const int c = n0 + j * 8 + 2 * (lane & 3) + (q & 1), t = m0 + (lane >> 2) + (q >> 1) * 8;
        float av = 1.f, bv = 0.f;
        if (t < nt && o0 + c < bs) {
          const float em = quick_expm1(quick_sigmoid(r[j][q] + s_ba[c]) * s_sp[c]);      // a - 1
          const float uv = to_f(*reinterpret_cast<const __nv_bfloat16*>(Us + t * pitch + (o0 + c) * 2));
          av = 1.f + em;
          bv = quick_sqrt(-em * (2.f + em)) * quick_sigmoid(g[j][q] + s_bi[c]) * uv;
        }
        r[j][q] = av;
        bvs[j][q] = bv;
      }
    __syncthreads();                                    // every warp is done with u
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        const int c = n0 + j * 8 + 2 * (lane & 3) + (q & 1), t = m0 + (lane >> 2) + (q >> 1) * 8;
        As[t * (LC + 1) + c] = r[j][q];
        Bs[t * (LC + 1) + c] = bvs[j][q];
      }
    __syncthreads();
    // recurrence inside the tile: SEGS segments per channel, then the segments in order
    const int c = tid & (LC - 1), sg = tid / LC;
    float pa[SEG], hb[SEG];
#pragma unroll
    for (int t = 0; t < SEG; ++t) {
      const int x = (sg * SEG + t) * (LC + 1) + c;
      const float av = As[x];
      hb[t] = t ? av * hb[t - 1] + Bs[x] : Bs[x];
      pa[t] = t ? pa[t - 1] * av : av;
    }
    segA[sg][c] = pa[SEG - 1];
    segB[sg][c] = hb[SEG - 1];
    __syncthreads();
    float cp = 1.f, chn = 0.f;
    for (int j = 0; j < sg; ++j) { chn = segA[j][c] * chn + segB[j][c]; cp *= segA[j][c]; }
    if (o0 + c < bs) {
      const int col = blk * bs + o0 + c;
      const long long first = (long long)(t0 + sg * SEG) * W + col;
      float *hp = H + first, *pp = P + first;
#pragma unroll
      for (int t = 0; t < SEG; ++t, hp += W, pp += W) {
        const int tt = sg * SEG + t;
        if (tt < nt) {
          const float h = hb[t] + pa[t] * chn, p = pa[t] * cp;
          *hp = h;
          *pp = p;
          if (tt == nt - 1) {
            LH[(long long)tile * W + col] = h;
            LP[(long long)tile * W + col] = p;
          }
        }
      }
    }
  }
}

// One thread per (entry, channel): LH becomes the state before each tile; the entry's new state and ring rows.
// first_tile[e]: the entry's first tile.
__global__ void rglru_chain_kernel(float* __restrict__ LH, const float* __restrict__ LP, const __nv_bfloat16* __restrict__ proj,
                                   long long ldp, int x_off, Ragged rb, const int* __restrict__ first_tile, int W, int K,
                                   float* __restrict__ state, float* __restrict__ ring) {
  pdl_trigger();
  pdl_wait();
  const int c = blockIdx.x * blockDim.x + threadIdx.x, e = blockIdx.y;
  if (c >= W) return;
  const int p0 = rb.pos0[e], t0 = rb.cu[e], t1 = rb.cu[e + 1];
  if (p0 < 0 || t1 <= t0) return;
  const long long sl = rb.slot[e];
  float s = p0 > 0 ? state[sl * W + c] : 0.f;
  const int a = first_tile[e], b = a + (t1 - t0 + LT - 1) / LT;
  for (int x = a; x < b; x += 8) {
    float h[8], p[8];
#pragma unroll
    for (int j = 0; j < 8; ++j)
      if (x + j < b) { h[j] = LH[(long long)(x + j) * W + c]; p[j] = LP[(long long)(x + j) * W + c]; }
#pragma unroll
    for (int j = 0; j < 8; ++j)
      if (x + j < b) {
        LH[(long long)(x + j) * W + c] = s;
        s = p[j] * s + h[j];
      }
  }
  state[sl * W + c] = s;
  for (int t = max(t0, t1 - K); t < t1; ++t)
    ring[(sl * K + (p0 + t - t0) % K) * W + c] = to_f(proj[(long long)t * ldp + x_off + c]);
}

// out = (H + P * state before the tile) * gelu(y); 4 channels per thread
__global__ void __launch_bounds__(256)
rglru_out_kernel(const float* __restrict__ H, const float* __restrict__ P, const float* __restrict__ carry,
                 const __nv_bfloat16* __restrict__ proj, long long ldp, int y_off, Ragged rb, const int* __restrict__ first_tile,
                 int W, __nv_bfloat16* __restrict__ out) {
  pdl_trigger();
  pdl_wait();
  const int per = W / 4;
  const long long total = (long long)rb.n * per;
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const int t = (int)(i / per), c = (int)(i - (long long)t * per) * 4;
    const int e = rb.ent[t];
    const int tile = first_tile[e] + (t - rb.cu[e]) / LT;
    const float4 h = *reinterpret_cast<const float4*>(H + (long long)t * W + c);
    const float4 p = *reinterpret_cast<const float4*>(P + (long long)t * W + c);
    const float4 s = *reinterpret_cast<const float4*>(carry + (long long)tile * W + c);
    const uint2 y = *reinterpret_cast<const uint2*>(proj + (long long)t * ldp + y_off + c);
    uint2 o;
    o.x = pack_bf16((h.x + p.x * s.x) * quick_gelu_tanh(bf16_lo(y.x)), (h.y + p.y * s.y) * quick_gelu_tanh(bf16_hi(y.x)));
    o.y = pack_bf16((h.z + p.z * s.z) * quick_gelu_tanh(bf16_lo(y.y)), (h.w + p.w * s.w) * quick_gelu_tanh(bf16_hi(y.y)));
    *reinterpret_cast<uint2*>(out + (long long)t * W + c) = o;
  }
}

// rglru_conv_kernel for whole tiles: a thread takes 4 channels of CT consecutive tokens and keeps the KT taps and the
// past inputs in registers.
constexpr int CT = 16;
template <int KT>
__global__ void __launch_bounds__(128)
rglru_conv_tile_kernel(const __nv_bfloat16* __restrict__ proj, long long ldp, int x_off, const __nv_bfloat16* __restrict__ w,
                       const __nv_bfloat16* __restrict__ bias, const float* __restrict__ ring, Ragged rb, Tiles tl, int W,
                       __nv_bfloat16* __restrict__ u) {
  pdl_trigger();
  pdl_wait();
  const int c = (blockIdx.x * 128 + threadIdx.x) * 4;
  const int tile = blockIdx.y, e = tl.ent[tile];
  const int first = rb.cu[e], p0 = rb.pos0[e];
  const int t0 = tl.t0[tile] + blockIdx.z * CT, t1 = min(min(t0 + CT, tl.t0[tile] + LT), rb.cu[e + 1]);
  if (c >= W || t0 >= t1) return;
  float taps[KT][4], past[KT][4], b4[4];                // past[j]: the input j tokens back
#pragma unroll
  for (int q = 0; q < 4; ++q) {
    b4[q] = to_f(bias[c + q]);
#pragma unroll
    for (int j = 0; j < KT; ++j) taps[j][q] = to_f(w[(long long)(c + q) * KT + KT - 1 - j]);
  }
#pragma unroll
  for (int j = 1; j < KT; ++j) {
    const int t = t0 - j, p = p0 + t - first;
#pragma unroll
    for (int q = 0; q < 4; ++q) past[j][q] = 0.f;
    if (t >= first) load_v<4>(proj + (long long)t * ldp + x_off + c, past[j]);
    else if (p >= 0) load_v<4>(ring + ((long long)rb.slot[e] * KT + p % KT) * W + c, past[j]);
  }
  for (int t = t0; t < t1; ++t) {
    load_v<4>(proj + (long long)t * ldp + x_off + c, past[0]);
    float o[4];
#pragma unroll
    for (int q = 0; q < 4; ++q) {
      o[q] = b4[q];
#pragma unroll
      for (int j = 0; j < KT; ++j) o[q] += taps[j][q] * past[j][q];
    }
    store_v<4>(u + (long long)t * W + c, o);
#pragma unroll
    for (int j = KT - 1; j > 0; --j)
#pragma unroll
      for (int q = 0; q < 4; ++q) past[j][q] = past[j - 1][q];
  }
}

// ---- bf16, one token per entry: convolution, gates, recurrence and output gate in one launch. CTA: 16 entries x DC output
// channels of one block; every CTA computes the convolution of its whole block (the ring row written is never read).
constexpr int DC = 32;
template <int KT>               // taps, or 0 for any number
__global__ void __launch_bounds__(256)
rglru_step_kernel(const __nv_bfloat16* __restrict__ proj, long long ldp, int x_off, int y_off,
                  const __nv_bfloat16* __restrict__ cw, const __nv_bfloat16* __restrict__ cb,
                  const __nv_bfloat16* __restrict__ ra, const __nv_bfloat16* __restrict__ ba,
                  const __nv_bfloat16* __restrict__ ri, const __nv_bfloat16* __restrict__ bi,
                  const __nv_bfloat16* __restrict__ lam, Ragged rb, int W, int bs, int K, float* __restrict__ state,
                  float* __restrict__ ring, __nv_bfloat16* __restrict__ out) {
  extern __shared__ __align__(16) uint8_t smem[];
  const int kp = (bs + 15) & ~15, pitch = kp * 2 + 16, chunks = kp / 8;
  uint8_t* Us = smem;                                   // [16] rows of u
  uint8_t* Ws = smem + 16 * pitch;                      // [2 * DC] rows
  const uint32_t us = smem_u32(Us), ws = smem_u32(Ws);
  const int per_blk = (bs + DC - 1) / DC;
  const int blk = blockIdx.x / per_blk, o0 = (blockIdx.x - blk * per_blk) * DC, e0 = blockIdx.y * 16;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, li = lane >> 3, lr = lane & 7;
  // weights do not depend on the kernels before
  for (int i = tid; i < 2 * DC * chunks; i += 256) {
    const int r = i / chunks, c = i - r * chunks, o = o0 + (r & (DC - 1));
    const bool ok = o < bs && c * 8 < bs;
    cp_async16(ws + r * pitch + c * 16, (r < DC ? ra : ri) + ((long long)blk * bs + (ok ? o : 0)) * bs + (ok ? c * 8 : 0), ok ? 16 : 0);
  }
  cp_async_commit();
  pdl_trigger();
  pdl_wait();
  // a thread keeps its 4 channels (one pass per 1024) and walks the entries
  const int quads = kp / 4, span = min(quads, 256), rstep = 256 / span;
  for (int cq = tid % span; cq < quads && tid < rstep * span; cq += span) {
    const int c = cq * 4, ch = blk * bs + c;
    const bool in = c < bs;
    float taps[KT > 0 ? KT : 1][4], b4[4];
    if (in) {
      load_v<4>(cb + ch, b4);
#pragma unroll
      for (int j = 0; j < KT; ++j)
#pragma unroll
        for (int q = 0; q < 4; ++q) taps[j][q] = to_f(cw[(long long)(ch + q) * KT + KT - 1 - j]);
    }
#pragma unroll 4
    for (int r = tid / span; r < 16; r += rstep) {
      const int e = e0 + r;
      float acc[4] = {0.f, 0.f, 0.f, 0.f};
      const int p = in && e < rb.E ? rb.pos0[e] : -1;
      if (p >= 0) {
        const long long rows = (long long)rb.slot[e] * K;
        float x[4];
        load_v<4>(proj + (long long)e * ldp + x_off + ch, x);
        if constexpr (KT > 0) {
          float v[KT][4];
#pragma unroll
          for (int j = 1; j < KT; ++j) {
            v[j][0] = v[j][1] = v[j][2] = v[j][3] = 0.f;
            if (j <= p) load_v<4>(ring + (rows + (p - j) % KT) * W + ch, v[j]);
          }
#pragma unroll
          for (int q = 0; q < 4; ++q) {
            acc[q] = b4[q] + taps[0][q] * x[q];
#pragma unroll
            for (int j = 1; j < KT; ++j) acc[q] += taps[j][q] * v[j][q];
          }
        } else {
#pragma unroll
          for (int q = 0; q < 4; ++q) acc[q] = b4[q] + to_f(cw[(long long)(ch + q) * K + K - 1]) * x[q];
          for (int j = 1; j < K && j <= p; ++j) {
            float v[4];
            load_v<4>(ring + (rows + (p - j) % K) * W + ch, v);
#pragma unroll
            for (int q = 0; q < 4; ++q) acc[q] += to_f(cw[(long long)(ch + q) * K + K - 1 - j]) * v[q];
          }
        }
        if (c >= o0 && c < o0 + DC) store_v<4>(ring + (rows + p % K) * W + ch, x);
      }
      store_v<4>(reinterpret_cast<__nv_bfloat16*>(Us + r * pitch) + c, acc);
    }
  }
  cp_async_wait<0>();
  __syncthreads();
  // 8 warps: 4 groups of 8 channels x 2 halves of the contraction, summed through shared memory
  float r[4] = {0.f, 0.f, 0.f, 0.f}, g[4] = {0.f, 0.f, 0.f, 0.f};
  __shared__ float half_sum[4][32][8];
  const int cg = warp & 3, kh = warp >> 2, nks = kp / 16, kmid = (nks + 1) / 2;
#pragma unroll 4
  for (int ks = kh ? kmid : 0; ks < (kh ? nks : kmid); ++ks) {
    uint32_t a[4], w[4];
    ldsm_x4(a, us + ((li & 1) * 8 + lr) * pitch + (ks * 2 + (li >> 1)) * 16);
    // matrices 0, 1: this warp's 8 channels of ra; 2, 3: of ri
    ldsm_x4(w, ws + ((li >> 1) * DC + cg * 8 + lr) * pitch + (ks * 2 + (li & 1)) * 16);
    mma_16816(r, a, w[0], w[1]);
    mma_16816(g, a, w[2], w[3]);
  }
  if (kh) {
#pragma unroll
    for (int q = 0; q < 4; ++q) { half_sum[cg][lane][q] = r[q]; half_sum[cg][lane][4 + q] = g[q]; }
  }
  __syncthreads();
  if (kh) return;
#pragma unroll
  for (int q = 0; q < 4; ++q) { r[q] += half_sum[cg][lane][q]; g[q] += half_sum[cg][lane][4 + q]; }
#pragma unroll
  for (int q = 0; q < 4; ++q) {
    const int o = o0 + cg * 8 + 2 * (lane & 3) + (q & 1), row = (lane >> 2) + (q >> 1) * 8, e = e0 + row;
    if (o >= bs || e >= rb.E) continue;
    const int ch = blk * bs + o, p = rb.pos0[e];
    float res = 0.f;
    if (p >= 0) {
      const float em = quick_expm1(-8.f * quick_sigmoid(r[q] + to_f(ba[ch])) * softplus(to_f(lam[ch])));   // a - 1
      const float uv = to_f(*reinterpret_cast<const __nv_bfloat16*>(Us + row * pitch + o * 2));
      float* st = state + (long long)rb.slot[e] * W + ch;
      const float s = (p > 0 ? (1.f + em) * *st : 0.f) + sqrtf(-em * (2.f + em)) * quick_sigmoid(g[q] + to_f(bi[ch])) * uv;
      *st = s;
      res = s * quick_gelu_tanh(to_f(proj[(long long)e * ldp + y_off + ch]));
    }
    out[(long long)e * W + ch] = __float2bfloat16(res);
  }
}

// ------------------------------------------------------------------------------------------------ mLSTM
constexpr int MV = 32;          // value columns per CTA (a slice)
constexpr int MTHREADS = 256;

// One CTA per (entry, head, slice): token by token, S in shared memory.
template <typename T>
__global__ void __launch_bounds__(MTHREADS)
mlstm_seq_kernel(const T* __restrict__ proj, long long ldp, int q_off, int k_off, int v_off, const float* __restrict__ gates,
                 const T* __restrict__ ib, const T* __restrict__ fb, float cap, Ragged rb, int heads, int dk, int dv,
                 float* __restrict__ Sg, float* __restrict__ Ng, float* __restrict__ Mg, float* __restrict__ out) {
  extern __shared__ float sm[];
  float* S = sm;                       // [dk][MV]
  float* nv = S + dk * MV;             // [dk]
  float* qs = nv + dk;                 // [dk]
  float* ks = qs + dk;                 // [dk]
  float* vs = ks + dk;                 // [MV]
  float* part = vs + MV;               // [8][MV]
  __shared__ float red[33];
  pdl_trigger();
  pdl_wait();
  const int e = blockIdx.z, hd = blockIdx.y, sl = blockIdx.x, slices = gridDim.x;
  const int t0 = rb.cu[e], t1 = rb.cu[e + 1], p0 = rb.pos0[e];
  const int c0 = sl * MV, nc = min(MV, dv - c0);
  const int tid = threadIdx.x, col = tid & 31, rg = tid >> 5;
  if (p0 < 0) {
    for (int t = t0; t < t1; ++t)
      if (tid < nc) out[((long long)t * heads + hd) * dv + c0 + tid] = 0.f;
    return;
  }
  if (t0 >= t1) return;
  const long long slot = rb.slot[e];
  float* Sh = Sg + (slot * heads + hd) * (long long)dk * dv;
  float* Nh = Ng + ((slot * heads + hd) * slices + sl) * (long long)dk;
  float* Mh = Mg + (slot * heads + hd) * slices + sl;
  float m = p0 > 0 ? *Mh : 0.f;
  for (int i = tid; i < dk * MV; i += MTHREADS) {
    const int d = i / MV, c = i - d * MV;
    S[i] = (p0 > 0 && c < nc) ? Sh[(long long)d * dv + c0 + c] : 0.f;
  }
  for (int d = tid; d < dk; d += MTHREADS) nv[d] = p0 > 0 ? Nh[d] : 0.f;
  const float bi = to_f(ib[hd]), bf = to_f(fb[hd]);
  const float qscale = 1.f / sqrtf((float)dk);
  for (int t = t0; t < t1; ++t) {
    const T* row = proj + (long long)t * ldp;
    __syncthreads();
    for (int d = tid; d < dk; d += MTHREADS) {
      qs[d] = to_f(row[q_off + hd * dk + d]) * qscale;
      ks[d] = to_f(row[k_off + hd * dk + d]);
    }
    if (tid < MV) vs[tid] = tid < nc ? to_f(row[v_off + hd * dv + c0 + tid]) : 0.f;
    const float ig = cap * tanhf((gates[(long long)t * 2 * heads + hd] + bi) / cap);
    const float fg = log_sigmoid(cap * tanhf((gates[(long long)t * 2 * heads + heads + hd] + bf) / cap));
    const float mn = fmaxf(fg + m, ig);
    const float da = decay_exp(fg + m - mn), db = expf(ig - mn);
    m = mn;
    __syncthreads();
    float nq = 0.f;
    for (int d = tid; d < dk; d += MTHREADS) {
      const float nn = da * nv[d] + db * ks[d];
      nv[d] = nn;
      nq += nn * qs[d];
    }
    float acc = 0.f;
    const float bv = db * vs[col];
    for (int d = rg; d < dk; d += MTHREADS / 32) {
      const float s = da * S[d * MV + col] + bv * ks[d];
      S[d * MV + col] = s;
      acc += s * qs[d];
    }
    part[rg * MV + col] = acc;
    nq = block_sum(nq, red);           // ends with a barrier: `part` is complete too
    if (tid < nc) {
      float o = 0.f;
#pragma unroll
      for (int j = 0; j < MTHREADS / 32; ++j) o += part[j * MV + tid];
      out[((long long)t * heads + hd) * dv + c0 + tid] = o / (fmaxf(fabsf(nq), expf(-m)) + 1e-6f);
    }
  }
  __syncthreads();
  for (int i = tid; i < dk * MV; i += MTHREADS) {
    const int d = i / MV, c = i - d * MV;
    if (c < nc) Sh[(long long)d * dv + c0 + c] = S[i];
  }
  for (int d = tid; d < dk; d += MTHREADS) Nh[d] = nv[d];
  if (tid == 0) *Mh = m;
}

// ---- one token per entry: the state slice streams through registers, nothing is staged
template <typename T>
__global__ void __launch_bounds__(MTHREADS)
mlstm_step_kernel(const T* __restrict__ proj, long long ldp, int q_off, int k_off, int v_off, const float* __restrict__ gates,
                  const T* __restrict__ ib, const T* __restrict__ fb, float cap, Ragged rb, int heads, int dk, int dv,
                  float* __restrict__ Sg, float* __restrict__ Ng, float* __restrict__ Mg, float* __restrict__ out) {
  extern __shared__ float sm[];
  float* qs = sm;                      // [dk]
  float* ks = qs + dk;                 // [dk]
  __shared__ float part[MTHREADS / 32][MV];
  __shared__ float red[33];
  pdl_trigger();
  pdl_wait();
  const int e = blockIdx.z, hd = blockIdx.y, sl = blockIdx.x, slices = gridDim.x;
  const int p0 = rb.pos0[e];
  const int c0 = sl * MV, nc = min(MV, dv - c0);
  const int tid = threadIdx.x, col = tid & 31, rg = tid >> 5;
  float* o = out + ((long long)e * heads + hd) * dv + c0;
  if (p0 < 0) {
    if (tid < nc) o[tid] = 0.f;
    return;
  }
  const bool old = p0 > 0;
  const long long slot = rb.slot[e];
  float* Sh = Sg + (slot * heads + hd) * (long long)dk * dv + c0;
  float* Nh = Ng + ((slot * heads + hd) * slices + sl) * (long long)dk;
  float* Mh = Mg + (slot * heads + hd) * slices + sl;
  const T* row = proj + (long long)e * ldp;
  const float m = old ? *Mh : 0.f;
  const float ig = cap * tanhf((gates[(long long)e * 2 * heads + hd] + to_f(ib[hd])) / cap);
  const float fg = log_sigmoid(cap * tanhf((gates[(long long)e * 2 * heads + heads + hd] + to_f(fb[hd])) / cap));
  const float mn = fmaxf(fg + m, ig);
  const float da = decay_exp(fg + m - mn), db = expf(ig - mn);
  const float qscale = 1.f / sqrtf((float)dk);
  float nq = 0.f;
  for (int d = tid; d < dk; d += MTHREADS) {
    const float q = to_f(row[q_off + hd * dk + d]) * qscale, k = to_f(row[k_off + hd * dk + d]);
    qs[d] = q;
    ks[d] = k;
    const float nn = da * (old ? Nh[d] : 0.f) + db * k;
    Nh[d] = nn;
    nq += nn * q;
  }
  nq = block_sum(nq, red);             // also: every thread has read m, and qs / ks are complete
  if (tid == 0) *Mh = mn;
  float acc = 0.f;
  if (col < nc) {
    const float bv = db * to_f(row[v_off + hd * dv + c0 + col]);
    constexpr int U = 8;
    for (int d0 = rg; d0 < dk; d0 += U * (MTHREADS / 32)) {
      float s[U];
#pragma unroll
      for (int j = 0; j < U; ++j) {
        const int d = d0 + j * (MTHREADS / 32);
        s[j] = (old && d < dk) ? Sh[(long long)d * dv + col] : 0.f;
      }
#pragma unroll
      for (int j = 0; j < U; ++j) {
        const int d = d0 + j * (MTHREADS / 32);
        if (d < dk) {
          const float v = da * s[j] + bv * ks[d];
          Sh[(long long)d * dv + col] = v;
          acc += v * qs[d];
        }
      }
    }
  }
  part[rg][col] = acc;
  __syncthreads();
  if (tid < nc) {
    float v = 0.f;
#pragma unroll
    for (int j = 0; j < MTHREADS / 32; ++j) v += part[j][tid];
    o[tid] = v / (fmaxf(fabsf(nq), expf(-mn)) + 1e-6f);
  }
}

// gates [n, 2 * heads], in place: pre-activations -> log input gate i and log forget gate f
template <typename T>
__global__ void mlstm_gates_kernel(float* __restrict__ gates, const T* __restrict__ ib, const T* __restrict__ fb, float cap,
                                   int n, int heads) {
  pdl_trigger();
  pdl_wait();
  for (int i = blockIdx.x * blockDim.x + threadIdx.x; i < n * 2 * heads; i += gridDim.x * blockDim.x) {
    const int h = i % (2 * heads);
    const float z = cap * tanhf((gates[i] + to_f(h < heads ? ib[h] : fb[h - heads])) / cap);
    gates[i] = h < heads ? z : log_sigmoid(z);
  }
}

// ---- bf16, prompt portions: chunks of ML tokens on tensor cores
// With F the running sum of f inside a chunk, g_s = i_s - F_s and M_t = max(m_prev, max_{s <= t} g_s), the recurrence above
// unrolls to  m_t = F_t + M_t,
//   o_t ~ e^(m_prev - M_t) q_t S + sum_{s <= t} e^(g_s - M_t) (q_t . k_s) v_s,   S' = e^(m_prev - M_L) S + sum_s e^(g_s - M_L) k_s v_s^T.
// n rides along as one more column of S, fed by a value column of ones. What enters the recurrence keeps 32-bit accuracy: S
// and n stay in fp32 accumulators, the scaled values go to the tensor cores as bf16 pairs hi + lo, k is bf16 and exact. The
// read-out q S takes S rounded to bf16 (n as a pair, since the denominator may cancel); row sums of the weights are fp32.
constexpr int ML = 64;
constexpr int MN = MV + 8;              // value columns with the ones column (index MV), padded to 8
constexpr int MVP = MN * 2;             // row pitch in bytes of [.., MN] bf16 tiles: 80, an odd multiple of 16
constexpr int MPP = ML * 2 + 16;        // row pitch of the [ML, ML] weight tiles

struct MlstmSmem {
  int pitch, q, k, v, wv, p, s, gate, total;            // byte offsets
};
__host__ __device__ constexpr MlstmSmem mlstm_smem(int kp) {
  MlstmSmem L{};
  L.pitch = kp * 2 + 16;
  L.q = 0;
  L.k = L.q + ML * L.pitch;
  L.v = L.k + ML * L.pitch;
  L.wv = L.v + ML * MVP;
  L.p = L.wv + 2 * ML * MVP;
  L.s = L.p + ML * MPP;
  L.gate = L.s + kp * MVP;
  L.total = L.gate + 8 * ML * 4;
  return L;
}

template <int KP>       // key size, zero-padded
__global__ void __launch_bounds__(256, 2)
mlstm_chunk_kernel(const __nv_bfloat16* __restrict__ proj, long long ldp, int q_off, int k_off, int v_off,
                   const float* __restrict__ gates, Ragged rb, int heads, int dk, int dv, float* __restrict__ Sg, float* __restrict__ Ng,
                   float* __restrict__ Mg, float* __restrict__ out) {
  extern __shared__ __align__(16) uint8_t smem[];
  constexpr MlstmSmem L = mlstm_smem(KP);
  constexpr int mtiles = KP / 16, MT = (mtiles + 7) / 8;        // 16-row tiles of S, and per warp
  const uint32_t sb = smem_u32(smem);
  float* G = reinterpret_cast<float*>(smem + L.gate);   // g_s
  float* Mx = G + ML;                                   // M_t
  float* Ct = Mx + ML;                                  // e^(m_prev - M_t)
  float* Wt = Ct + ML;                                  // e^(g_s - M_L)
  float* Em = Wt + ML;                                  // e^(-m_t)
  float* Den = Em + ML;
  float* Sum = Den + ML;                                // [2][ML] row sums of the weights, per half of the keys
  __shared__ float s_m, s_decay;
  pdl_trigger();
  pdl_wait();
  const int e = blockIdx.z, hd = blockIdx.y, sl = blockIdx.x, slices = gridDim.x;
  const int p0 = rb.pos0[e], t0 = rb.cu[e], len = rb.cu[e + 1] - t0;
  if (p0 < 0 || len <= 0) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, li = lane >> 3, lr = lane & 7;
  const int c0 = sl * MV, nc = min(MV, dv - c0);
  const long long slot = rb.slot[e];
  float* Sh = Sg + (slot * heads + hd) * (long long)dk * dv + c0;
  float* Nh = Ng + ((slot * heads + hd) * slices + sl) * (long long)dk;
  float* Mh = Mg + (slot * heads + hd) * slices + sl;
  const float qscale = 1.f / sqrtf((float)dk);

  const GridWalk walk(tid, 256, KP / 8);
  auto load = [&](int ch) {
    const int rows = min(ML, len - ch * ML);
    const __nv_bfloat16* base = proj + (long long)(t0 + ch * ML) * ldp;
    const __nv_bfloat16 *qs = base + q_off + hd * dk, *ks = base + k_off + hd * dk;
    for (GridWalk g = walk; g.r < ML; g.next()) {
      const bool ok = g.r < rows && g.c * 8 < dk;
      const long long src = ok ? g.r * ldp + g.c * 8 : 0;
      const uint32_t d = g.r * L.pitch + g.c * 16;
      cp_async16(sb + L.q + d, qs + src, ok ? 16 : 0);
      cp_async16(sb + L.k + d, ks + src, ok ? 16 : 0);
    }
    for (int i = tid; i < ML * (MV / 8); i += 256) {
      const int r = i / (MV / 8), c = i - r * (MV / 8);
      const bool ok = r < rows && c * 8 < nc;
      cp_async16(sb + L.v + r * MVP + c * 16, base + v_off + (ok ? (long long)r * ldp + hd * dv + c0 + c * 8 : 0), ok ? 16 : 0);
    }
    cp_async_commit();
  };

  // the ones column (and its padding)
  for (int i = tid; i < ML; i += 256)
    *reinterpret_cast<uint4*>(smem + L.v + i * MVP + MV * 2) = make_uint4(0x3f80u, 0u, 0u, 0u);   // 1.0 in the first of 8 columns
  load(0);

  // state -> accumulators: warp w owns the 16-row tiles w, w + 8, ...
  float S[MT][5][4];
#pragma unroll
  for (int a = 0; a < MT; ++a)
#pragma unroll
    for (int j = 0; j < 5; ++j)
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        const int d = (warp + a * 8) * 16 + (lane >> 2) + (q >> 1) * 8, c = j * 8 + 2 * (lane & 3) + (q & 1);
        float v = 0.f;
        if (p0 > 0 && d < dk) {
          if (c < nc) v = Sh[(long long)d * dv + c];
          else if (c == MV) v = Nh[d];
        }
        S[a][j][q] = v;
      }
  // S as the B operand of Q S: bf16, and in the last column tile n as hi (column MV) and lo (column MV + 1)
  auto store_s = [&]() {
#pragma unroll
    for (int a = 0; a < MT; ++a) {
      if (warp + a * 8 >= mtiles) continue;
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int d = (warp + a * 8) * 16 + (lane >> 2) + h * 8;
#pragma unroll
        for (int j = 0; j < 4; ++j)
          *reinterpret_cast<uint32_t*>(smem + L.s + d * MVP + (j * 8 + 2 * (lane & 3)) * 2) = pack_bf16(S[a][j][2 * h], S[a][j][2 * h + 1]);
        __nv_bfloat16 hi, lo;
        split_bf16((lane & 3) == 0 ? S[a][4][2 * h] : 0.f, hi, lo);
        *reinterpret_cast<__nv_bfloat162*>(smem + L.s + d * MVP + (MV + 2 * (lane & 3)) * 2) = __halves2bfloat162(hi, lo);
      }
    }
  };
  store_s();
  float m_prev = p0 > 0 ? *Mh : 0.f;
  const int n_ch = (len + ML - 1) / ML;
  const int wm = (warp & 3) * 16, wn = warp >> 2;       // 16 tokens; half of the keys (P) or of the value columns (O)
  for (int ch = 0; ch < n_ch; ++ch) {
    const int rows = min(ML, len - ch * ML);
    cp_async_wait<0>();
    __syncthreads();                    // the tiles are in, S of the last chunk is stored
    const uint32_t qb = sb + L.q, kb = sb + L.k, vb = sb + L.v;
    if (warp == 0) {
      // gates of the chunk, two tokens per lane
      float f[2], ii[2];
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        const int t = 2 * lane + j;
        f[j] = 0.f;
        ii[j] = -INFINITY;
        if (t < rows) {
          const float* gr = gates + (long long)(t0 + ch * ML + t) * 2 * heads + hd;
          ii[j] = gr[0];
          f[j] = gr[heads];
        }
      }
      float run = f[0] + f[1];
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float x = __shfl_up_sync(0xffffffffu, run, o);
        if (lane >= o) run += x;
      }
      const float F1 = run, F0 = run - f[1];
      const float g0 = ii[0] - F0, g1 = ii[1] - F1;
      float mx = fmaxf(g0, g1);
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float x = __shfl_up_sync(0xffffffffu, mx, o);
        if (lane >= o) mx = fmaxf(mx, x);
      }
      float before = __shfl_up_sync(0xffffffffu, mx, 1);
      if (lane == 0) before = -INFINITY;
      const float M0 = fmaxf(m_prev, fmaxf(before, g0)), M1 = fmaxf(m_prev, mx);
      const float ML_ = __shfl_sync(0xffffffffu, M1, 31), FL = __shfl_sync(0xffffffffu, F1, 31);
      const int t = 2 * lane;
      G[t] = g0; G[t + 1] = g1;
      Mx[t] = M0; Mx[t + 1] = M1;
      Ct[t] = quick_exp(m_prev - M0); Ct[t + 1] = quick_exp(m_prev - M1);
      Wt[t] = expf(g0 - ML_); Wt[t + 1] = expf(g1 - ML_);
      Em[t] = quick_exp(-(F0 + M0)); Em[t + 1] = quick_exp(-(F1 + M1));
      if (lane == 0) { s_m = FL + ML_; s_decay = expf(m_prev - ML_); }
    }
    // P = Q K^T (this warp: 16 tokens x 32 keys; key tiles past the diagonal are skipped)
    float P[4][4];
#pragma unroll
    for (int j = 0; j < 4; ++j) P[j][0] = P[j][1] = P[j][2] = P[j][3] = 0.f;
    const int kn = wn * 32;
    if (kn <= wm + 15) {
#pragma unroll 4
      for (int ks = 0; ks < mtiles; ++ks) {
        uint32_t a[4], b[4];
        ldsm_x4(a, qb + (wm + (li & 1) * 8 + lr) * L.pitch + (ks * 2 + (li >> 1)) * 16);
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          ldsm_x4(b, kb + (kn + h * 16 + (li >> 1) * 8 + lr) * L.pitch + (ks * 2 + (li & 1)) * 16);
          mma_16816(P[2 * h], a, b[0], b[1]);
          mma_16816(P[2 * h + 1], a, b[2], b[3]);
        }
      }
    }
    __syncthreads();                    // gates are in shared memory
    m_prev = s_m;
    const float decay = s_decay;
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int t = wm + (lane >> 2) + h * 8;
      const float M = Mx[t];
      float sum = 0.f;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int s = kn + j * 8 + 2 * (lane & 3);
        const float w0 = s <= t ? P[j][2 * h] * qscale * quick_exp(G[s] - M) : 0.f;
        const float w1 = s + 1 <= t ? P[j][2 * h + 1] * qscale * quick_exp(G[s + 1] - M) : 0.f;
        sum += w0 + w1;
        *reinterpret_cast<uint32_t*>(smem + L.p + t * MPP + s * 2) = pack_bf16(w0, w1);
      }
      sum += __shfl_xor_sync(0xffffffffu, sum, 1);
      sum += __shfl_xor_sync(0xffffffffu, sum, 2);
      if ((lane & 3) == 0) Sum[wn * ML + t] = sum;
    }
    for (int i = tid; i < ML * (MN / 2); i += 256) {    // w_s v_s, hi and lo
      const int r = i / (MN / 2), c = (i - r * (MN / 2)) * 2;
      const uint32_t v2 = *reinterpret_cast<const uint32_t*>(smem + L.v + r * MVP + c * 2);
      const float w = Wt[r];
      __nv_bfloat16 h0, l0, h1, l1;
      split_bf16(w * bf16_lo(v2), h0, l0);
      split_bf16(w * bf16_hi(v2), h1, l1);
      *reinterpret_cast<__nv_bfloat162*>(smem + L.wv + r * MVP + c * 2) = __halves2bfloat162(h0, h1);
      *reinterpret_cast<__nv_bfloat162*>(smem + L.wv + ML * MVP + r * MVP + c * 2) = __halves2bfloat162(l0, l1);
    }
    __syncthreads();
    // O = diag(c) Q S + P V; column tiles 0, 1 and the pair of n (first half of the warps) or 2, 3 (second half)
    float O[3][4];
#pragma unroll
    for (int j = 0; j < 3; ++j) O[j][0] = O[j][1] = O[j][2] = O[j][3] = 0.f;
    const uint32_t row16 = (li & 1) * 8 + lr;           // row inside a 16-row B tile
#pragma unroll 4
    for (int ks = 0; ks < mtiles; ++ks) {
      uint32_t a[4], b[4], b2[2];
      ldsm_x4(a, qb + (wm + (li & 1) * 8 + lr) * L.pitch + (ks * 2 + (li >> 1)) * 16);
      const uint32_t base = sb + L.s + (ks * 16 + row16) * MVP;
      ldsm_x4_t(b, base + (wn * 2 + (li >> 1)) * 16);
      mma_16816(O[0], a, b[0], b[1]);
      mma_16816(O[1], a, b[2], b[3]);
      if (wn == 0) {
        ldsm_x2_t(b2, base + 4 * 16);
        mma_16816(O[2], a, b2[0], b2[1]);
      }
    }
    {
      const float ca = Ct[wm + (lane >> 2)] * qscale, cb = Ct[wm + (lane >> 2) + 8] * qscale;
#pragma unroll
      for (int j = 0; j < 3; ++j) { O[j][0] *= ca; O[j][1] *= ca; O[j][2] *= cb; O[j][3] *= cb; }
    }
#pragma unroll
    for (int ks = 0; ks < ML / 16; ++ks) {
      if (ks * 16 > wm + 15) continue;                  // weights past the diagonal are zero
      uint32_t a[4], b[4];
      ldsm_x4_t(b, vb + (ks * 16 + row16) * MVP + (wn * 2 + (li >> 1)) * 16);
      ldsm_x4(a, sb + L.p + (wm + (li & 1) * 8 + lr) * MPP + (ks * 2 + (li >> 1)) * 16);
      mma_16816(O[0], a, b[0], b[1]);
      mma_16816(O[1], a, b[2], b[3]);
    }
    if (wn == 0 && (lane & 3) == 0) {                   // n . q
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int t = wm + (lane >> 2) + h * 8;
        const float nq = O[2][2 * h] + O[2][2 * h + 1] + Sum[t] + Sum[ML + t];
        Den[t] = 1.f / (fmaxf(fabsf(nq), Em[t]) + 1e-6f);
      }
    }
    // S = decay S + K^T (w V)
#pragma unroll
    for (int a = 0; a < MT; ++a) {
      const int mt = warp + a * 8;
      if (mt >= mtiles) continue;
#pragma unroll
      for (int j = 0; j < 5; ++j)
#pragma unroll
        for (int q = 0; q < 4; ++q) S[a][j][q] *= decay;
#pragma unroll
      for (int ks = 0; ks < ML / 16; ++ks) {
        uint32_t ak[4];
        ldsm_x4_t(ak, kb + (ks * 16 + (li >> 1) * 8 + lr) * L.pitch + (mt * 2 + (li & 1)) * 16);
#pragma unroll
        for (int part = 0; part < 2; ++part) {
          uint32_t b[4], b2[2];
          const uint32_t base = sb + L.wv + part * ML * MVP + (ks * 16 + row16) * MVP;
          ldsm_x4_t(b, base + (li >> 1) * 16);
          mma_16816(S[a][0], ak, b[0], b[1]);
          mma_16816(S[a][1], ak, b[2], b[3]);
          ldsm_x4_t(b, base + (2 + (li >> 1)) * 16);
          mma_16816(S[a][2], ak, b[0], b[1]);
          mma_16816(S[a][3], ak, b[2], b[3]);
          ldsm_x2_t(b2, base + 4 * 16);
          mma_16816(S[a][4], ak, b2[0], b2[1]);
        }
      }
    }
    __syncthreads();                    // Den is complete; nobody reads the tiles or the old S any more
    if (ch + 1 < n_ch) load(ch + 1);
    store_s();
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int tile = wn * 2 + j;
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int t = wm + (lane >> 2) + h * 8, c = tile * 8 + 2 * (lane & 3);
        if (t < rows && c < nc) {
          const float dn = Den[t];
          *reinterpret_cast<float2*>(out + ((long long)(t0 + ch * ML + t) * heads + hd) * dv + c0 + c) =
              make_float2(O[j][2 * h] * dn, O[j][2 * h + 1] * dn);      // dv and c are even
        }
      }
    }
  }
#pragma unroll
  for (int a = 0; a < MT; ++a)
#pragma unroll
    for (int j = 0; j < 5; ++j)
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        const int d = (warp + a * 8) * 16 + (lane >> 2) + (q >> 1) * 8, c = j * 8 + 2 * (lane & 3) + (q & 1);
        if (d < dk) {
          if (c < nc) Sh[(long long)d * dv + c] = S[a][j][q];
          else if (c == MV) Nh[d] = S[a][j][q];
        }
      }
  if (tid == 0) *Mh = m_prev;
}

}  // namespace

#define RAGGED Ragged rb{cu, slot, pos0, ent, E, n}

// x and y are columns x_off.. and y_off.. of proj [n, ldp]. u / A / B: workspaces [n, W] (T, fp32, fp32).
// state fp32 [slots, W], ring fp32 [slots, K, W]; out T [n, W]. `one`: every entry is one token.
// bf16 portions also take tile lists (LT tokens a tile): tile_t0 / tile_ent [tiles], first_tile [E], and workspaces
// LH / LP fp32 [tiles, W]; with tiles == 0 the plain kernels run.
TB_API int tb_rglru(int dtype, const void* proj, long long ldp, int x_off, int y_off, const void* conv_w, const void* conv_b,
                    const void* ra, const void* rab, const void* ri, const void* rib, const void* lam, const int* cu,
                    const int* slot, const int* pos0, const int* ent, int E, int n, int W, int K, int blocks, float* state,
                    float* ring, void* u, float* A, float* B, void* out, int one, const int* tile_t0, const int* tile_ent,
                    const int* first_tile, int tiles, float* LH, float* LP, cudaStream_t stream) {
  if (n <= 0 || E <= 0) return 0;
  if (blocks <= 0 || W % blocks || K < 1 || E > 65535) return -2;
  const int bs = W / blocks, kp = (bs + 15) & ~15, pitch = kp * 2 + 16;
  RAGGED;
  typedef __nv_bfloat16 bf;
  if (dtype == 0 && bs % 8 == 0 && x_off % 4 == 0 && y_off % 4 == 0 && ldp % 4 == 0) {
    if (one) {
      const size_t smem = (size_t)(16 + 2 * DC) * pitch;
      if (smem <= 200 * 1024) {
        const dim3 grid(blocks * ((bs + DC - 1) / DC), (E + 15) / 16);
#define STEP(KT)                                                                                                              \
  {                                                                                                                           \
    static DeviceOnce once;                                                                                                   \
    if (once.first() && cudaFuncSetAttribute(rglru_step_kernel<KT>, cudaFuncAttributeMaxDynamicSharedMemorySize,              \
                                             200 * 1024) != cudaSuccess) return -5;                                           \
    return launch_pdl(rglru_step_kernel<KT>, grid, dim3(256), smem, stream, (const bf*)proj, ldp, x_off, y_off,               \
                      (const bf*)conv_w, (const bf*)conv_b, (const bf*)ra, (const bf*)rab, (const bf*)ri, (const bf*)rib,     \
                      (const bf*)lam, rb, W, bs, K, state, ring, (bf*)out) == cudaSuccess ? 0 : -5;                           \
  }
        switch (K) {
          case 2: STEP(2)
          case 3: STEP(3)
          case 4: STEP(4)
          default: STEP(0)
        }
#undef STEP
      }
    } else if (tiles > 0) {
      const size_t ub = (size_t)(LT * pitch > 2 * LT * (LC + 1) * 4 ? LT * pitch : 2 * LT * (LC + 1) * 4);
      const size_t smem = 2 * ub + (size_t)2 * LC * pitch;
      if (smem <= 220 * 1024) {
        Tiles tl{tile_t0, tile_ent, tiles};
        const long long want = ((long long)n * (W / 4) + 255) / 256;
        const dim3 flat((unsigned)(want < 148 * 16 ? want : 148 * 16));
        const dim3 gtile(blocks * ((bs + LC - 1) / LC), (tiles + LTPC - 1) / LTPC);
        if (gtile.y > 65535) return -2;
        if (tiles > 65535) return -2;
        cudaError_t err;
#define CONV(KT)                                                                                                              \
  case KT:                                                                                                                    \
    err = launch_pdl(rglru_conv_tile_kernel<KT>, dim3((W / 4 + 127) / 128, tiles, LT / CT), dim3(128), 0, stream,              \
                     (const bf*)proj, ldp, x_off, (const bf*)conv_w, (const bf*)conv_b, (const float*)ring, rb, tl, W, (bf*)u); \
    break;
        switch (K) {
          CONV(1) CONV(2) CONV(3) CONV(4) CONV(5) CONV(6) CONV(7) CONV(8)
          default:
            if (n > 65535) return -2;
            err = launch_pdl(rglru_conv_kernel<bf>, dim3((W + 127) / 128, n), dim3(128), 0, stream, (const bf*)proj, ldp, x_off,
                             (const bf*)conv_w, (const bf*)conv_b, (const float*)ring, rb, W, K, (bf*)u);
        }
#undef CONV
#define TILE(KP)                                                                                                              \
  {                                                                                                                           \
    static DeviceOnce once;                                                                                                   \
    if (once.first() && cudaFuncSetAttribute(rglru_tile_kernel<KP>, cudaFuncAttributeMaxDynamicSharedMemorySize,              \
                                             220 * 1024) != cudaSuccess) return -5;                                           \
    err = launch_pdl(rglru_tile_kernel<KP>, gtile, dim3(256), smem, stream, (const bf*)u, (const bf*)ra, (const bf*)rab,       \
                     (const bf*)ri, (const bf*)rib, (const bf*)lam, rb, tl, W, bs, A, B, LH, LP);                              \
  }
        if (err != cudaSuccess) return -5;
        if (kp == 64) TILE(64) else if (kp == 128) TILE(128) else if (kp == 256) TILE(256) else TILE(0)
#undef TILE
        if (err == cudaSuccess)
          err = launch_pdl(rglru_chain_kernel, dim3((W + 63) / 64, E), dim3(64), 0, stream, LH, (const float*)LP, (const bf*)proj,
                           ldp, x_off, rb, first_tile, W, K, state, ring);
        if (err == cudaSuccess)
          err = launch_pdl(rglru_out_kernel, flat, dim3(256), 0, stream, (const float*)A, (const float*)B, (const float*)LH,
                           (const bf*)proj, ldp, y_off, rb, first_tile, W, (bf*)out);
        return err == cudaSuccess ? 0 : -5;
      }
    }
  }
  const dim3 gconv((W + 127) / 128, n), ggate((bs + GC - 1) / GC, blocks, (n + GT - 1) / GT), gscan((W + 63) / 64, E);
  if (n > 65535 || blocks > 65535) return -2;
  const size_t smem = (size_t)GT * bs * 4;
  if (smem > 200 * 1024) return -2;
#define RUN(T)                                                                                                              \
  {                                                                                                                         \
    static DeviceOnce once;                                                                                                 \
    if (once.first() && cudaFuncSetAttribute(rglru_gates_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize,            \
                                             200 * 1024) != cudaSuccess) return -5;                                         \
    cudaError_t err = launch_pdl(rglru_conv_kernel<T>, gconv, dim3(128), 0, stream, (const T*)proj, ldp, x_off,             \
                                 (const T*)conv_w, (const T*)conv_b, (const float*)ring, rb, W, K, (T*)u);                  \
    if (err != cudaSuccess) return -5;                                                                                      \
    err = launch_pdl(rglru_gates_kernel<T>, ggate, dim3(128), smem, stream, (const T*)u, (const T*)ra, (const T*)rab,       \
                     (const T*)ri, (const T*)rib, (const T*)lam, n, W, bs, A, B);                                           \
    if (err != cudaSuccess) return -5;                                                                                      \
    err = launch_pdl(rglru_scan_kernel<T>, gscan, dim3(64), 0, stream, (const float*)A, (const float*)B, (const T*)proj,    \
                     ldp, x_off, y_off, rb, W, K, state, ring, (T*)out);                                                    \
    return err == cudaSuccess ? 0 : -5;                                                                                     \
  }
  if (dtype == 0) RUN(__nv_bfloat16) else RUN(float)
#undef RUN
}

TB_API int tb_mlstm_slices(int dv) { return (dv + MV - 1) / MV; }

// q, k, v: columns of proj [n, ldp]; gates fp32 [n, 2 * heads] = (W_i h, W_f h) without bias.
// S fp32 [slots, heads, dk, dv], N fp32 [slots, heads, slices, dk], M fp32 [slots, heads, slices]; out fp32 [n, heads, dv].
// `one`: every entry is one token. `chunked` (overwrites gates): bf16 portions take the tensor-core form where the sizes allow.
TB_API int tb_mlstm(int dtype, const void* proj, long long ldp, int q_off, int k_off, int v_off, float* gates,
                    const void* ib, const void* fb, float cap, const int* cu, const int* slot, const int* pos0,
                    const int* ent, int E, int n, int heads, int dk, int dv, float* S, float* N, float* M, float* out, int one,
                    int chunked, cudaStream_t stream) {
  if (n <= 0 || E <= 0) return 0;
  if (E > 65535 || heads > 65535) return -2;
  RAGGED;
  const dim3 grid(tb_mlstm_slices(dv), heads, E);
#define ARGS(T) (const T*)proj, ldp, q_off, k_off, v_off, gates, (const T*)ib, (const T*)fb, cap, rb, heads, dk, dv, S, N, M, out
  if (one) {
    const size_t smem = (size_t)2 * dk * 4;
    if (smem > 48 * 1024) return -2;
    cudaError_t err = dtype == 0 ? launch_pdl(mlstm_step_kernel<__nv_bfloat16>, grid, dim3(MTHREADS), smem, stream, ARGS(__nv_bfloat16))
                                 : launch_pdl(mlstm_step_kernel<float>, grid, dim3(MTHREADS), smem, stream, ARGS(float));
    return err == cudaSuccess ? 0 : -5;
  }
  if (dtype == 0 && chunked && dk <= 256 && dk % 8 == 0 && dv % 8 == 0 && q_off % 8 == 0 && k_off % 8 == 0 && v_off % 8 == 0 &&
      ldp % 8 == 0 && (reinterpret_cast<uintptr_t>(proj) & 15) == 0) {
    if ((long long)n * 2 * heads > (1 << 30)) return -2;
    const int want = (n * 2 * heads + 255) / 256;
    cudaError_t err = launch_pdl(mlstm_gates_kernel<__nv_bfloat16>, dim3(want < 148 * 8 ? want : 148 * 8), dim3(256), 0, stream, gates,
                                 (const __nv_bfloat16*)ib, (const __nv_bfloat16*)fb, cap, n, heads);
    if (err != cudaSuccess) return -5;
#define CHUNK(KP)                                                                                                             \
  {                                                                                                                           \
    static DeviceOnce once;                                                                                                   \
    if (once.first() && cudaFuncSetAttribute(mlstm_chunk_kernel<KP>, cudaFuncAttributeMaxDynamicSharedMemorySize,             \
                                             mlstm_smem(KP).total) != cudaSuccess) return -5;                                 \
    return launch_pdl(mlstm_chunk_kernel<KP>, grid, dim3(256), mlstm_smem(KP).total, stream, (const __nv_bfloat16*)proj, ldp, \
                      q_off, k_off, v_off, (const float*)gates, rb, heads, dk, dv, S, N, M, out) == cudaSuccess ? 0 : -5;     \
  }
    if (dk <= 32) CHUNK(32)
    if (dk <= 64) CHUNK(64)
    if (dk <= 128) CHUNK(128)
    if (dk <= 192) CHUNK(192)
    CHUNK(256)
#undef CHUNK
  }
  const size_t smem = ((size_t)dk * (MV + 3) + MV * 9) * 4;
  if (smem > 200 * 1024) return -2;
#define RUN(T)                                                                                                              \
  {                                                                                                                         \
    static DeviceOnce once;                                                                                                 \
    if (once.first() && cudaFuncSetAttribute(mlstm_seq_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize,              \
                                             200 * 1024) != cudaSuccess) return -5;                                         \
    return launch_pdl(mlstm_seq_kernel<T>, grid, dim3(MTHREADS), smem, stream, ARGS(T)) == cudaSuccess ? 0 : -5;            \
  }
  if (dtype == 0) RUN(__nv_bfloat16) else RUN(float)
#undef RUN
#undef ARGS
}
