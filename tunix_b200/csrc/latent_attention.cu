// Latent attention over a paged cache: a token keeps one row, its normed latent c (R columns) followed by one rotated key part
// (rot columns) that all heads share. Head h's key is [U_h c, rotated part] and its value is V_h c.
//
//   latent_write  : after the joint projection of a step: the rotated parts of all query heads turn in place, the latent is
//                   RMS-normed with weights, the shared key part turns, and both go to the token's page.
//   latent_gather : copies blocks of 64 cached rows into one array, so that a product can expand them to the heads' keys and
//                   values for the flash attention of a portion (attention_fwd.cu).
//   head_product  : a product with a matrix per head and few rows. Single tokens use the absorbed form: the score is
//                   (U_h^T q) . c + rotated parts, and the weighted sum of latents goes through V_h once, so a query reads R + rot
//                   columns per key whatever the number of heads.
//   latent_decode : that attention on tcgen05. One CTA per (query token, up to 32 heads, split of the context): tiles of 64 rows come
//                   by TMA and serve as keys and, in their first R columns, as values. With a handful of heads the products are
//                   taken the other way round: keys, then value columns, are the 128 rows of a product and heads its columns.
//
// Other sizes and 32-bit use window_attn (window_attention.cu) on the absorbed form: one key head, values = the key's columns.
// This file is compiled without fast-math: latent_write serves the 32-bit mode as well.
#include "decode_splits.cuh"
#include "mma.cuh"
#include "precise.cuh"

using namespace tb;

namespace {

// proj [n, ldp]: H query heads of dim + rot columns, then (c_off) the latent and the key part. V elements per access.
template <typename T, int V>
__global__ void __launch_bounds__(192)
latent_write_kernel(T* __restrict__ proj, long long ldp, int H, int dim, int rot, int c_off, int R, const T* __restrict__ w, float eps,
                    const float* __restrict__ cos_t, const float* __restrict__ sin_t, int rd, Ragged rb, const int* __restrict__ table,
                    int max_pages, int page_size, int W, T* __restrict__ pool) {
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x, e = rb.ent[t], p0 = rb.pos0[e];
  if (p0 < 0) return;
  const int p = p0 + t - rb.cu[e];
  T* row = proj + (long long)t * ldp;
  const int page = table[(long long)rb.slot[e] * max_pages + p / page_size];
  T* dst = pool + ((long long)page * page_size + p % page_size) * W;
  if (threadIdx.x < 32) {
    const int lane = threadIdx.x;
    const T* c = row + c_off;
    float ss = 0.f;
    for (int i = lane * V; i < R; i += 32 * V) {
      float v[V];
      load_v<V>(c + i, v);
#pragma unroll
      for (int k = 0; k < V; ++k) ss += v[k] * v[k];
    }
    const float r = 1.f / sqrtf(warp_sum(ss) / (float)R + eps);
    for (int i = lane * V; i < R; i += 32 * V) {
      float v[V], ww[V];
      load_v<V>(c + i, v);
      load_v<V>(w + i, ww);
#pragma unroll
      for (int k = 0; k < V; ++k) v[k] = v[k] * r * ww[k];
      store_v<V>(dst + i, v);
    }
    return;
  }
  const int half = rd >> 1, per = half / V, tid = threadIdx.x - 32;
  const float *ct = cos_t + (long long)p * half, *st = sin_t + (long long)p * half;
  for (int i = tid; i < (H + 1) * per; i += blockDim.x - 32) {
    const int hh = i / per, d = (i - hh * per) * V;
    T* src = hh < H ? row + (long long)hh * (dim + rot) + dim : row + c_off + R;
    T* to = hh < H ? src : dst + R;
    float u[V], v[V], c[V], s[V];
    load_v<V>(src + d, u);
    load_v<V>(src + half + d, v);
    load_v<V>(ct + d, c);
    load_v<V>(st + d, s);
#pragma unroll
    for (int k = 0; k < V; ++k) {
      const float a = u[k], b = v[k];
      u[k] = a * c[k] - b * s[k];
      v[k] = b * c[k] + a * s[k];
    }
    store_v<V>(to + d, u);
    store_v<V>(to + half + d, v);
  }
  for (int d = rd + tid; d < rot; d += blockDim.x - 32) dst[R + d] = row[c_off + R + d];
}

// dst rows i * 64 .. i * 64 + 63 = the rows of positions pos[i] .. in the sequence of slot[i]; page_size is a multiple of 64
__global__ void __launch_bounds__(256)
latent_gather_kernel(const uint4* __restrict__ pool, const int* __restrict__ slot, const int* __restrict__ pos,
                     const int* __restrict__ table, int max_pages, int page_size, int vec, uint4* __restrict__ dst) {
  pdl_trigger();
  pdl_wait();
  const int i = blockIdx.x, p = pos[i];
  const int page = table[(long long)slot[i] * max_pages + p / page_size];
  const uint4* src = pool + ((long long)page * page_size + p % page_size) * vec;
  uint4* to = dst + (long long)i * 64 * vec;
  for (int c = blockIdx.y * 256 + threadIdx.x; c < 64 * vec; c += gridDim.y * 256) to[c] = src[c];
}

// out[t, h, n] = sum_k x[t, h, k] w[h, k, n] (WN) or w[h, n, k]: a CTA owns 64 rows x 32 columns of one head and the whole
// contraction. WN also copies the `tail` columns behind x's K behind out's N, zeros up to `pad` columns. All sizes and strides are
// multiples of 8.
constexpr int HP_ROWS = 64, HP_COLS = 32;
template <bool WN>
__global__ void __launch_bounds__(128)
head_product_kernel(const __nv_bfloat16* __restrict__ x, long long ldx, int x_heads, const int* __restrict__ xrows,
                    const __nv_bfloat16* __restrict__ w, int K, int N, __nv_bfloat16* __restrict__ out, long long ldo, int o_heads,
                    const int* __restrict__ orows, int T, int tail, int pad) {
  extern __shared__ __align__(128) uint8_t smem[];
  pdl_trigger();
  pdl_wait();
  const int Kp = (K + 63) & ~63, h = blockIdx.y, n0 = blockIdx.x * HP_COLS, t0 = blockIdx.z * HP_ROWS;
  const uint32_t sx = smem_u32(smem), sw = sx + HP_ROWS * Kp * 2;
  const int cpr = Kp >> 3;
  for (int i = threadIdx.x; i < HP_ROWS * cpr; i += 128) {
    const int r = i / cpr, c = i - r * cpr, t = t0 + r;
    const bool ok = t < T && c * 8 < K;
    const long long row = ok ? (xrows ? xrows[t] : t) : 0;
    cp_async16(sx + r * Kp * 2 + (((c & ~7) | ((c ^ r) & 7)) << 4), x + (ok ? row * ldx + (long long)h * x_heads + c * 8 : 0), ok ? 16 : 0);
  }
  const __nv_bfloat16* wh = w + (long long)h * K * N;
  if (WN) {
    for (int i = threadIdx.x; i < Kp * 4; i += 128) {
      const int r = i >> 2, c = i & 3;
      const bool ok = r < K && n0 + c * 8 < N;
      cp_async16(sw + r * 64 + ((c ^ ((r >> 1) & 3)) << 4), wh + (ok ? (long long)r * N + n0 + c * 8 : 0), ok ? 16 : 0);
    }
  } else {
    for (int i = threadIdx.x; i < HP_COLS * cpr; i += 128) {
      const int r = i / cpr, c = i - r * cpr;
      const bool ok = n0 + r < N && c * 8 < K;
      cp_async16(sw + r * Kp * 2 + (((c & ~7) | ((c ^ r) & 7)) << 4), wh + (ok ? (long long)(n0 + r) * K + c * 8 : 0), ok ? 16 : 0);
    }
  }
  cp_async_commit();
  if (WN && blockIdx.x == 0) {
    for (int i = threadIdx.x; i < HP_ROWS * (pad >> 3); i += 128) {
      const int r = i / (pad >> 3), c = i - r * (pad >> 3), t = t0 + r;
      if (t >= T) continue;
      uint4 v = make_uint4(0u, 0u, 0u, 0u);
      if (c * 8 < tail) v = *reinterpret_cast<const uint4*>(x + (long long)(xrows ? xrows[t] : t) * ldx + (long long)h * x_heads + K + c * 8);
      *reinterpret_cast<uint4*>(out + (long long)(orows ? orows[t] : t) * ldo + (long long)h * o_heads + N + c * 8) = v;
    }
  }
  cp_async_wait<0>();
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, li = lane >> 3, lr = lane & 7;
  float acc[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
#pragma unroll 4
  for (int ks = 0; ks < Kp / 16; ++ks) {
    uint32_t a[4];
    {
      const int r = warp * 16 + (li & 1) * 8 + lr, c = ks * 2 + (li >> 1);
      ldsm_x4(a, sx + r * Kp * 2 + (((c & ~7) | ((c ^ r) & 7)) << 4));
    }
#pragma unroll
    for (int g = 0; g < 2; ++g) {
      uint32_t b[4];
      if (WN) {
        const int r = ks * 16 + (li & 1) * 8 + lr, c = g * 2 + (li >> 1);
        ldsm_x4_t(b, sw + r * 64 + ((c ^ ((r >> 1) & 3)) << 4));
      } else {
        const int r = g * 16 + (li >> 1) * 8 + lr, c = ks * 2 + (li & 1);
        ldsm_x4(b, sw + r * Kp * 2 + (((c & ~7) | ((c ^ r) & 7)) << 4));
      }
      mma_16816(acc[2 * g], a, b[0], b[1]);
      mma_16816(acc[2 * g + 1], a, b[2], b[3]);
    }
  }
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    const int t = t0 + warp * 16 + (lane >> 2) + 8 * half;
    if (t >= T) continue;
    __nv_bfloat16* o = out + (long long)(orows ? orows[t] : t) * ldo + (long long)h * o_heads;
#pragma unroll
    for (int g = 0; g < 4; ++g) {
      const int n = n0 + g * 8 + 2 * (lane & 3);
      if (n < N) *reinterpret_cast<uint32_t*>(o + n) = pack_bf16(acc[g][2 * half], acc[g][2 * half + 1]);
    }
  }
}

// The layout of a CTA's shared memory: two stages of 64 cached rows, the queries of NH heads, the weights of a tile as product
// operand, what the softmax warps tell each other per head, barriers. An output product may read 64 columns past a stage (rows that
// nobody uses), so at least that much follows the second one.
constexpr int LD_THREADS = 192;
struct LatentSmem {
  int stage, q, p, row, bars, total;
  __host__ __device__ LatentSmem(int W, int NH) : stage(64 * W * 2), q(2 * stage), p(q + NH * W * 2), row(p + NH * 128), bars(row + 6 * NH * 4) {
    total = (bars + 128 - q < 8192 ? q + 8192 : bars + 128);
  }
};

__device__ __forceinline__ void bar_sync(int id, int threads) { asm volatile("barrier.cta.sync %0, %1;" ::"r"(id), "r"(threads) : "memory"); }
__device__ __forceinline__ bool bar_any(int id, int threads, bool v) {
  uint32_t r;
  asm volatile("{\n.reg .pred p, q;\nsetp.ne.u32 p, %3, 0;\nbarrier.cta.red.or.pred q, %1, %2, p;\nselp.u32 %0, 1, 0, q;\n}"
               : "=r"(r) : "r"(id), "r"(threads), "r"((uint32_t)v) : "memory");
  return r != 0;
}
// Reduces 16 values per lane over the 16 lanes of a half warp: every exchange with the lane w away (w = 8, 4, 2, 1) halves the values,
// so that lane i of the half ends up with the result of value half_slot(i).
template <typename Op>
__device__ __forceinline__ float half_reduce(float (&x)[16], int lane, Op op) {
#pragma unroll
  for (int w = 8; w >= 1; w >>= 1) {
    const bool hi = lane & w;
#pragma unroll
    for (int c = 0; c < w; ++c) {
      const float keep = hi ? x[w + c] : x[c], give = hi ? x[c] : x[w + c];
      x[c] = op(keep, __shfl_xor_sync(0xffffffffu, give, w));
    }
  }
  return x[0];
}
__device__ __forceinline__ int half_slot(int lane) { return lane & 15; }
template <int NC>
__device__ __forceinline__ void tmem_ld_cols(uint32_t addr, float (&v)[NC]) {
  uint32_t r[NC];
  if constexpr (NC == 32) tmem_ld_32x32(addr, r);
  else tmem_ld_32x16(addr, r);
  tmem_ld_wait();
#pragma unroll
  for (int i = 0; i < NC; ++i) v[i] = __uint_as_float(r[i]);
}

// NH heads (16 or 32) of one query. q [T * H, W] absorbed queries, pool rows of W columns. Products run on tcgen05 with keys or value
// columns as the rows of a tile and heads as its columns: S^T = K Q^T, 64 rows, which lie in lanes 0-15 of every warp's 32; and
// O^T += V^T P^T, 128 rows, V being the same shared memory read along its other dimension.
//   warps 0-3 : softmax. A thread holds the scores of one key with 16 heads and keeps each head's maximum and its own share of the
//               sums, so nothing crosses lanes unless a score outgrows a maximum by more than 2^8: then the new maxima are shared
//               and O^T is rescaled. O^T leaves through all lanes (lane = value column).
//   warp 4    : one thread issues the products, scores of the next tile and outputs of this one in the order in which their
//               operands are ready.
//   warp 5    : one thread fetches queries and tiles; a buffer is free when the output product of its tile has retired.
template <int NH>
__global__ void __launch_bounds__(LD_THREADS, 1)
latent_decode_kernel(const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmQ, const int* __restrict__ table,
                     int max_pages, int page_size, const int* __restrict__ seq_ids, const int* __restrict__ seq_lens, int H, int R, int W,
                     float scale2, int window, const HeadExtras ex, int num_splits, int split_tokens, float* __restrict__ part_acc,
                     float* __restrict__ part_ml, __nv_bfloat16* __restrict__ out, int* __restrict__ status) {
  constexpr uint32_t TMEM_O = 2 * NH, TMEM_COLS = NH == 16 ? 128 : 256;
  extern __shared__ uint8_t smem_raw[];
  const uint32_t base = (smem_u32(smem_raw) + 1023u) & ~1023u;
  uint8_t* smem = smem_raw + (base - smem_u32(smem_raw));
  const LatentSmem lay(W, NH);
  const uint32_t sq = base + lay.q, sp = base + lay.p, bars = base + lay.bars;
  // barriers: 0-1 tile arrived, 2-3 tile free, 4-5 scores, 6 weights, 7 outputs, 8 queries
  const uint32_t bFull = bars, bFree = bars + 16, bS = bars + 32, bP = bars + 48, bO = bars + 56, bQ = bars + 64;
  volatile uint32_t* tmem_slot = reinterpret_cast<volatile uint32_t*>(smem + lay.bars + 80);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(smem + lay.bars + 84);
  float* s_row = reinterpret_cast<float*>(smem + lay.row);      // [4][NH]: per warp, maxima and at the end sums
  float* s_mul = s_row + 4 * NH;                                // [NH]: factors of the outputs
  float* s_max = s_mul + NH;                                    // [NH]: maxima at the end
  pdl_trigger();
  pdl_wait();
  const int b = blockIdx.x, h0 = blockIdx.y * NH, split = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int len = seq_lens[b];
  const KeyTiles kt(len, window, 0, 0);
  const int tile0 = split * (split_tokens / TILE_KEYS);
  const int n = min(kt.total - tile0, split_tokens / TILE_KEYS);
  if (len <= 0 || n <= 0) {             // past the end of this sequence: nobody reads this split
    if (num_splits == 1)
      for (int i = tid; i < min(NH, H - h0) * R; i += LD_THREADS) out[((long long)b * H + h0) * R + i] = __float2bfloat16(0.f);
    return;
  }
  const int mtiles = (R + 127) >> 7;
  const int* pt = table + (long long)seq_ids[b] * max_pages;
  auto row_of = [&](int j) {
    const int k = kt.start(tile0 + min(j, n - 1));
    return pt[k / page_size] * page_size + k % page_size;
  };
  auto fetch = [&](int j, int row) {                    // one thread
    const uint32_t bar = bFull + 8 * (j & 1), to = base + (j & 1) * lay.stage;
    mbar_expect_tx(bar, lay.stage);
    tma_load_3d(to, &tmK, bar, 0, row, 0);
  };
  if (tid == 160) {                                     // warp 5: what it fetches first needs no one else
#pragma unroll
    for (int i = 0; i < 6; ++i) mbar_init(bars + 8 * i, 1);
    mbar_init(bP, 128);
    mbar_init(bO, 1);
    mbar_init(bQ, 1);
    *abort_flag = 0;
    mbar_fence_init();
    fetch(0, row_of(0));
    mbar_expect_tx(bQ, NH * W * 2);
    tma_load_3d(sq, &tmQ, bQ, 0, b * H + h0, 0);
    if (n > 1) fetch(1, row_of(1));
  }
  if (warp == 4) {
    tmem_alloc(smem_u32((const void*)tmem_slot), TMEM_COLS);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot;

  if (warp == 5) {
    if (tid == 160) {
      for (int j = 2; j < n; ++j) {
        const int row = row_of(j);
        if (!mbar_wait_bounded(bFree + 8 * (j & 1), ((j >> 1) - 1) & 1, abort_flag, status, ST_TIMEOUT_PRODUCER)) break;
        fetch(j, row);
      }
    }
  } else if (warp == 4) {
    if (elect_one()) {
      const uint32_t idesc_s = make_idesc_bf16(64, NH, 0, 0), idesc_o = make_idesc_bf16(128, NH, 1, 0);
      // descriptors of a tile further along are the base plus (byte offset >> 4)
      const uint64_t kd0 = make_smem_desc(base, 16, 1024), qd0 = make_smem_desc(sq, 16, 1024);
      const uint64_t vd0 = make_smem_desc(base, 8192, 1024), pd0 = make_smem_desc(sp, 16, 1024);
      bool ok = mbar_wait_bounded(bQ, 0, abort_flag, status, ST_TIMEOUT_PRODUCER);
      int s = 0, o = 0, polls = 0;                      // next score product, next output product
      long long t0 = clock64();
      while (ok && o < n) {
        bool idle = true;
        if (s < n && s <= o + 1 && mbar_test(bFull + 8 * (s & 1), (s >> 1) & 1)) {
          tc_fence_after();
          uint64_t kd = kd0 + (uint64_t)(((s & 1) * lay.stage) >> 4), qd = qd0;
          const uint32_t d = tmem + (s & 1) * NH;
          for (int c = 0; c < W / 64; ++c, kd += 8192 >> 4, qd += (NH * 128) >> 4) {
            umma_f16_ss(d, kd, qd, idesc_s, c != 0);
            umma_f16_ss(d, kd + 2, qd + 2, idesc_s, 1);
            umma_f16_ss(d, kd + 4, qd + 4, idesc_s, 1);
            umma_f16_ss(d, kd + 6, qd + 6, idesc_s, 1);
          }
          umma_commit(bS + 8 * (s & 1));
          ++s;
          idle = false;
        }
        if (o < s && mbar_test(bP, o & 1)) {
          tc_fence_after();
          uint64_t vd = vd0 + (uint64_t)(((o & 1) * lay.stage) >> 4);
          uint32_t d = tmem + TMEM_O;
          for (int mt = 0; mt < mtiles; ++mt, vd += 16384 >> 4, d += NH) {
            umma_f16_ss(d, vd, pd0, idesc_o, o != 0);
            umma_f16_ss(d, vd + (2048 >> 4), pd0 + 2, idesc_o, 1);
            umma_f16_ss(d, vd + (4096 >> 4), pd0 + 4, idesc_o, 1);
            umma_f16_ss(d, vd + (6144 >> 4), pd0 + 6, idesc_o, 1);
          }
          umma_commit(bO);
          if (o + 2 < n) umma_commit(bFree + 8 * (o & 1));
          ++o;
          idle = false;
        }
        if (!idle) {
          t0 = clock64();
        } else if ((++polls & 63) == 0) {
          if (*abort_flag) break;
          if (clock64() - t0 > SPIN_LIMIT_CYCLES) {
            *abort_flag = 1;
            if (status) atomicCAS(status, 0, (int)ST_TIMEOUT_MMA);
            break;
          }
        }
      }
    }
  } else {
    const uint32_t lanes = (uint32_t)(warp * 32) << 16;
    const int key = warp * 16 + (lane & 15);            // this thread's key of a tile
    const int hb = NH == 32 ? (lane & 16) : 0;          // and the first of its 16 heads: lanes 16-31 take the second half
    const bool active = NH == 32 || lane < 16;
    float m[16], l[16];
#pragma unroll
    for (int c = 0; c < 16; ++c) { m[c] = -INFINITY; l[c] = 0.f; }
    bool ok = true;
    for (int j = 0; j < n; ++j) {
      ok = mbar_wait_bounded(bS + 8 * (j & 1), (j >> 1) & 1, abort_flag, status, ST_TIMEOUT_EPILOGUE);
      ok = __all_sync(0xffffffffu, ok);
      tc_fence_after();
      float z[16];
      {
        float v[NH];
        tmem_ld_cols<NH>(tmem + lanes + (j & 1) * NH, v);
#pragma unroll
        for (int c = 0; c < 16; ++c) {
          z[c] = v[c];
          if constexpr (NH == 32) {
            const float other = __shfl_sync(0xffffffffu, v[16 + c], lane & 15);
            z[c] = lane < 16 ? z[c] : other;
          }
        }
      }
      const int t0 = kt.start(tile0 + j);
      if (t0 < kt.w_lo || t0 + TILE_KEYS > len) {       // a tile at an end: not all of its keys are visible
        const bool seen = t0 + key < len && t0 + key >= kt.w_lo;
#pragma unroll
        for (int c = 0; c < 16; ++c) z[c] = seen ? z[c] : -INFINITY;
      }
      float over = -INFINITY;                           // how far scores lie above the maxima, in log2 units
#pragma unroll
      for (int c = 0; c < 16; ++c) over = fmaxf(over, fmaf(z[c], scale2, -m[c]));
      if (bar_any(1, 128, (active && over > 8.f) || j == 0 || !ok)) {
        // every tile has a visible key, so the maxima are finite from the first one on
        float x[16];
#pragma unroll
        for (int c = 0; c < 16; ++c) x[c] = z[c] * scale2;
        const float top = half_reduce(x, lane, [](float a, float c) { return fmaxf(a, c); });
        if (active) s_row[warp * NH + hb + half_slot(lane)] = top;
        if (bar_any(2, 128, !ok)) { ok = false; break; }
#pragma unroll
        for (int c = 0; c < 16; ++c) {
          const float* r = s_row + hb + c;
          const float y = fmaxf(fmaxf(r[0], r[NH]), fmaxf(r[2 * NH], r[3 * NH]));
          const bool up = y > m[c] + 8.f;
          const float alpha = up ? quick_exp2(m[c] - y) : 1.f;
          if (up) m[c] = y;
          l[c] *= alpha;
          if (warp == 0 && (lane & 15) == 0 && active) s_mul[hb + c] = alpha;
        }
        if (j > 0) {
          ok = __all_sync(0xffffffffu, mbar_wait_bounded(bO, (j - 1) & 1, abort_flag, status, ST_TIMEOUT_EPILOGUE));
          tc_fence_after();
          if (bar_any(1, 128, !ok)) { ok = false; break; }
#pragma unroll 1
          for (int c = 0; c < mtiles * NH; c += 16) {
            uint32_t o[16];
            tmem_ld_32x16(tmem + lanes + TMEM_O + c, o);
            tmem_ld_wait();
#pragma unroll
            for (int i = 0; i < 16; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * s_mul[(c & (NH - 1)) + i]);
            tmem_st_32x16(tmem + lanes + TMEM_O + c, o);
          }
          tmem_st_wait();
        }
      }
#pragma unroll
      for (int c = 0; c < 16; ++c) {
        z[c] = quick_exp2(fmaf(z[c], scale2, -m[c]));
        l[c] += z[c];
      }
      // the outputs of the tile before have retired: the weights' buffer is free
      if (j > 0) ok = mbar_wait_bounded(bO, (j - 1) & 1, abort_flag, status, ST_TIMEOUT_EPILOGUE) && ok;
      if (active) {
        uint8_t* at = smem + lay.p + hb * 128 + (key & 7) * 2;
#pragma unroll
        for (int c = 0; c < 16; c += 2) {               // a pair of heads shares the conversion
          const uint32_t two = pack_bf16(z[c], z[c + 1]);
          *reinterpret_cast<uint16_t*>(at + c * 128 + ((((key >> 3) ^ c) & 7) << 4)) = (uint16_t)two;
          *reinterpret_cast<uint16_t*>(at + c * 128 + 128 + ((((key >> 3) ^ (c + 1)) & 7) << 4)) = (uint16_t)(two >> 16);
        }
      }
      fence_proxy_async_smem();
      tc_fence_before();
      mbar_arrive(bP);
    }
    bar_sync(1, 128);
    if (warp == 0 && (lane & 15) == 0 && active) {
#pragma unroll
      for (int c = 0; c < 16; ++c) s_max[hb + c] = m[c];
    }
    const float sum_l = half_reduce(l, lane, [](float a, float c) { return a + c; });
    if (active) s_row[warp * NH + hb + half_slot(lane)] = sum_l;
    bar_sync(2, 128);
    if (tid < NH) {
      const float sum = s_row[tid] + s_row[NH + tid] + s_row[2 * NH + tid] + s_row[3 * NH + tid], top = s_max[tid];
      const int h = h0 + tid;
      s_mul[tid] = num_splits > 1 || h >= H ? 1.f : 1.f / (sum + quick_exp2(ex.sink_of(h) * LOG2_E - top));
      if (num_splits > 1 && h < H) {
        float* ml = part_ml + (((long long)b * H + h) * num_splits + split) * 2;
        ml[0] = top * 0.6931471805599453f;              // natural units, as the merging kernel has them
        ml[1] = sum;
      }
    }
    ok = ok && mbar_wait_bounded(bO, (n - 1) & 1, abort_flag, status, ST_TIMEOUT_EPILOGUE);
    tc_fence_after();
    // O^T through shared memory (the tiles have been read) to rows of heads
    if (!bar_any(1, 128, !ok)) {
      float f[NH];
#pragma unroll
      for (int c = 0; c < NH; ++c) f[c] = s_mul[c];
      for (int mt = 0; mt < mtiles; ++mt) {
        float v[NH];
        tmem_ld_cols<NH>(tmem + lanes + TMEM_O + mt * NH, v);
        const int d = mt * 128 + warp * 32 + lane;
        if (d < R && num_splits == 1) {
          uint8_t* to = smem + d * 2;
#pragma unroll
          for (int c = 0; c < NH; ++c, to += R * 2 + 16) *reinterpret_cast<__nv_bfloat16*>(to) = __float2bfloat16(v[c] * f[c]);
        } else if (d < R) {
          uint8_t* to = smem + d * 4;
#pragma unroll
          for (int c = 0; c < NH; ++c, to += R * 4 + 16) *reinterpret_cast<float*>(to) = v[c];
        }
      }
    }
  }
  __syncthreads();
  if (!*abort_flag) {
    const int size = num_splits == 1 ? 2 : 4, vec = R * size / 16;      // 16-byte pieces of a head
    uint8_t* to = num_splits == 1 ? reinterpret_cast<uint8_t*>(out) : reinterpret_cast<uint8_t*>(part_acc);
    const long long first = ((long long)b * H + h0) * num_splits + (num_splits == 1 ? 0 : split), step = (long long)num_splits * R * size;
    to += first * R * size;
    for (int i = tid; i < min(NH, H - h0) * vec; i += LD_THREADS) {
      const int c = i / vec, k = i - c * vec;
      *reinterpret_cast<uint4*>(to + c * step + k * 16) = *reinterpret_cast<const uint4*>(smem + c * (R * size + 16) + k * 16);
    }
  }
  tc_fence_before();
  __syncthreads();
  if (*abort_flag) {
    for (int i = 0; i < 2000; ++i) __nanosleep(1000);   // copies in flight land before the CTA's memory goes away
  }
  if (warp == 4) {
    tc_fence_after();
    tmem_dealloc(tmem, TMEM_COLS);
  }
}

template <int NH>
int launch_latent_decode(const void* pool, long long pool_rows, const void* q, int T, int H, int R, int W, const int* table, int max_pages,
                         int page_size, const int* seq_ids, const int* seq_lens, float scale, int window, HeadExtras ex, int splits,
                         int split_tokens, float* pa, float* pml, __nv_bfloat16* out, int* status, cudaStream_t stream) {
  constexpr int LIMIT = 226 * 1024;
  static DeviceOnce once;
  if (once.first() && cudaFuncSetAttribute(latent_decode_kernel<NH>, cudaFuncAttributeMaxDynamicSharedMemorySize, LIMIT) != cudaSuccess)
    return -5;
  const int smem = LatentSmem(W, NH).total + 1024;
  if (smem > LIMIT) return -2;
  CUtensorMap tk, tq;
  if (tb_make_tmap_slabs_bf16(&tk, pool, (uint64_t)pool_rows, (uint64_t)W, (uint64_t)W, TILE_KEYS) ||
      tb_make_tmap_slabs_bf16(&tq, q, (uint64_t)T * H, (uint64_t)W, (uint64_t)W, NH))
    return -3;
  return launch_pdl(latent_decode_kernel<NH>, dim3(T, (H + NH - 1) / NH, splits), dim3(LD_THREADS), smem, stream, tk, tq, table, max_pages,
                    page_size, seq_ids, seq_lens, H, R, W, scale * LOG2_E, window, ex, splits, split_tokens, pa, pml, out, status) == cudaSuccess
             ? 0 : -5;
}

}  // namespace

#define RAGGED Ragged rb{cu, slot, pos0, ent, E, n}

// proj T [n, ldp]: H query heads of dim + rot columns, and at c_off the latent (R) and the shared key part (rot). The first rd of
// every rotated part turn by the tables cos / sin fp32 [positions, rd / 2] (queries in place); the latent is normed with w T [R]; pool
// T [rows, W] gets the latent and the key part.
TB_API int tb_latent_write(int dtype, void* proj, long long ldp, int H, int dim, int rot, int c_off, int R, const void* w, float eps,
                           const float* cos_t, const float* sin_t, int rd, const int* cu, const int* slot, const int* pos0, const int* ent,
                           int E, int n, const int* table, int max_pages, int page_size, int W, void* pool, cudaStream_t stream) {
  if (n <= 0) return 0;
  if (rd < 0 || rd % 2 || rd > rot || R <= 0 || W < R + rot) return -2;
  RAGGED;
  typedef __nv_bfloat16 bf;
  const bool vec = dtype == 0 && ldp % 8 == 0 && dim % 8 == 0 && rot % 8 == 0 && c_off % 8 == 0 && R % 8 == 0 && W % 8 == 0 && rd % 16 == 0;
#define RUN(T, V)                                                                                                                  \
  launch_pdl(latent_write_kernel<T, V>, dim3(n), dim3(192), 0, stream, (T*)proj, ldp, H, dim, rot, c_off, R, (const T*)w, eps, cos_t, \
             sin_t, rd, rb, table, max_pages, page_size, W, (T*)pool)
  return (dtype ? RUN(float, 1) : vec ? RUN(bf, 8) : RUN(bf, 1)) == cudaSuccess ? 0 : -5;
#undef RUN
}

// dst bf16 [blocks * 64, W] = cached rows of positions pos[i] .. pos[i] + 63 of the sequences slot[i] (pos multiples of 64)
TB_API int tb_latent_gather(const void* pool, const int* slot, const int* pos, int blocks, const int* table, int max_pages,
                            int page_size, int W, void* dst, cudaStream_t stream) {
  if (blocks <= 0) return 0;
  if (page_size % 64 || W % 8) return -2;
  return launch_pdl(latent_gather_kernel, dim3(blocks, 4), dim3(256), 0, stream, (const uint4*)pool, slot, pos, table, max_pages, page_size,
                    W / 8, (uint4*)dst) == cudaSuccess ? 0 : -5;
}

// x bf16: row xrows[t] (or t) at ldx, heads x_heads apart; w bf16 [H, K, N] (wn) or [H, N, K]; out likewise. wn: the `tail` columns
// behind x's K go behind out's N, then zeros up to `pad` columns. Everything a multiple of 8; K at most 512.
TB_API int tb_head_product(int wn, const void* x, long long ldx, int x_heads, const int* xrows, const void* w, int H, int K, int N, void* out,
                           long long ldo, int o_heads, const int* orows, int T, int tail, int pad, cudaStream_t stream) {
  if (T <= 0 || H <= 0 || N <= 0) return 0;
  if (K <= 0 || K > 512 || K % 8 || N % 8 || tail % 8 || pad % 8 || ldx % 8 || x_heads % 8 || ldo % 8 || o_heads % 8 ||
      ((uintptr_t)x & 15) || ((uintptr_t)w & 15) || ((uintptr_t)out & 15))
    return -2;
  typedef __nv_bfloat16 bf;
  const int smem = (HP_ROWS + HP_COLS) * ((K + 63) & ~63) * 2;
  const dim3 grid((N + HP_COLS - 1) / HP_COLS, H, (T + HP_ROWS - 1) / HP_ROWS);
  if (grid.z > 65535 || H > 65535) return -2;
  static DeviceOnce once;
  if (once.first() &&
      (cudaFuncSetAttribute(head_product_kernel<true>, cudaFuncAttributeMaxDynamicSharedMemorySize, 96 * 1024) != cudaSuccess ||
       cudaFuncSetAttribute(head_product_kernel<false>, cudaFuncAttributeMaxDynamicSharedMemorySize, 96 * 1024) != cudaSuccess))
    return -5;
  const cudaError_t err =
      wn ? launch_pdl(head_product_kernel<true>, grid, dim3(128), smem, stream, (const bf*)x, ldx, x_heads, xrows, (const bf*)w, K, N, (bf*)out,
                      ldo, o_heads, orows, T, tail, pad)
         : launch_pdl(head_product_kernel<false>, grid, dim3(128), smem, stream, (const bf*)x, ldx, x_heads, xrows, (const bf*)w, K, N, (bf*)out,
                      ldo, o_heads, orows, T, 0, 0);
  return err == cudaSuccess ? 0 : -5;
}

// q bf16 [T, H, W] absorbed queries, one per entry of seq_ids (page-table row) / seq_lens (keys it sees at most, 0: none); pool bf16
// [pool_rows, W]: keys, and in their first R columns values. window <= 0: none. sinks fp32 [H] or null. out bf16 [T, H, R]. Workspace
// as for tb_paged_decode with splits = ceil(tiles / (split_tokens / 64)), `tiles` the most tiles of 64 keys that a query walks.
TB_API int tb_latent_decode(const void* q, const void* pool, long long pool_rows, const int* table, int max_pages, int page_size,
                            const int* seq_ids, const int* seq_lens, int T, int H, int R, int W, int tiles, float scale, int window,
                            const float* sinks, int split_tokens, float* part_acc, float* part_ml, void* out, int* status,
                            cudaStream_t stream) {
  if (T <= 0 || H <= 0) return 0;
  if (W % 64 || R % 8 || R <= 0 || R > 512 || R > W || page_size % TILE_KEYS || split_tokens <= 0 || split_tokens % TILE_KEYS || tiles <= 0)
    return -2;
  const int per = split_tokens / TILE_KEYS, splits = (tiles + per - 1) / per;
  const HeadExtras ex{-INFINITY, sinks, nullptr, 0};
#define RUN(NH)                                                                                                                       \
  launch_latent_decode<NH>(pool, pool_rows, q, T, H, R, W, table, max_pages, page_size, seq_ids, seq_lens, scale, window, ex, splits, \
                           split_tokens, part_acc, part_ml, (__nv_bfloat16*)out, status, stream)
  const int rc = H > 16 ? RUN(32) : RUN(16);
#undef RUN
  if (rc || splits == 1) return rc;
  return launch_pdl(paged_decode_combine_kernel, dim3(T, H), dim3(128), 0, stream, (const float*)part_acc, (const float*)part_ml, seq_lens, H,
                    R, splits, split_tokens, window, 0, 0, 1.f, R, ex, (__nv_bfloat16*)out, (long long)H * R) == cudaSuccess ? 0 : -5;
}
