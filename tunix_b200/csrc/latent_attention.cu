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
//   latent_decode : that attention. One CTA per (query token, up to 32 heads, split of the context): tiles of 64 rows come by TMA
//                   and serve as keys and, in their first R columns, as values; the heads are the rows of mma.sync tiles. Eight
//                   warps cut the scores into 16 keys x half of the contraction and the output into columns.
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

// The layout of a CTA's shared memory: two stages of 64 cached rows, the queries, the weights of a tile, its scores (the two halves
// of the contraction), and what the rows of heads are rescaled by.
struct LatentSmem {
  int stage, q, p, s, row, total;
  __host__ __device__ LatentSmem(int W, int rows)
      : stage(64 * W * 2), q(2 * stage), p(q + rows * W * 2), s(p + rows * 128), row(s + 2 * rows * 68 * 4), total(row + 3 * rows * 4) {}
};

// CB blocks of 16 output columns per warp, MT tiles of 16 heads. q [T, H, W] absorbed queries, pool rows of W columns.
template <int CB, int MT>
__global__ void __launch_bounds__(256, 1)
latent_decode_kernel(const __grid_constant__ CUtensorMap tmK, const __nv_bfloat16* __restrict__ q, const int* __restrict__ table,
                     int max_pages, int page_size, const int* __restrict__ seq_ids, const int* __restrict__ seq_lens, int H, int R, int W,
                     float scale, int window, const HeadExtras ex, int num_splits, int split_tokens, float* __restrict__ part_acc,
                     float* __restrict__ part_ml, __nv_bfloat16* __restrict__ out, int* __restrict__ status) {
  constexpr int ROWS = MT * 16, TPR = 256 / ROWS, KPT = 64 / TPR;     // threads per row of scores, keys per thread
  extern __shared__ uint8_t smem_raw[];
  __shared__ __align__(8) unsigned long long full_bars[2];
  __shared__ int abort_flag;
  uint8_t* smem = smem_raw + ((1024u - (smem_u32(smem_raw) & 1023u)) & 1023u);
  const LatentSmem lay(W, ROWS);
  pdl_trigger();
  pdl_wait();
  const int b = blockIdx.x, h0 = blockIdx.y * ROWS, split = blockIdx.z;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, li = lane >> 3, lr = lane & 7;
  const int len = seq_lens[b];
  const KeyTiles kt(len, window, 0, 0);
  const int tile0 = split * (split_tokens / TILE_KEYS);
  const int n_tiles = min(kt.total - tile0, split_tokens / TILE_KEYS);
  if (len <= 0 || n_tiles <= 0) {       // past the end of this sequence: nobody reads this split
    if (num_splits == 1)
      for (int i = tid; i < min(ROWS, H - h0) * R; i += 256) out[((long long)b * H + h0) * R + i] = __float2bfloat16(0.f);
    return;
  }
  const int* pt = table + (long long)seq_ids[b] * max_pages;
  const uint32_t base = smem_u32(smem), sq = base + lay.q, sp = base + lay.p;
  float* s_s = reinterpret_cast<float*>(smem + lay.s);          // [2][ROWS][68]
  float* s_alpha = reinterpret_cast<float*>(smem + lay.row);    // [ROWS], then the rows' maxima and sums
  if (tid == 0) {
    mbar_init(smem_u32(&full_bars[0]), 1);
    mbar_init(smem_u32(&full_bars[1]), 1);
    abort_flag = 0;
    mbar_fence_init();
  }
  __syncthreads();
  auto issue = [&](int tile) {
    const int k = kt.start(tile0 + tile), buf = tile & 1;
    const int row = pt[k / page_size] * page_size + k % page_size;
    const uint32_t bar = smem_u32(&full_bars[buf]);
    mbar_expect_tx(bar, lay.stage);
    for (int s = 0; s < W / 64; ++s) tma_load_2d(base + buf * lay.stage + s * 8192, &tmK, bar, s * 64, row);
  };
  if (tid == 0) {
    issue(0);
    if (n_tiles > 1) issue(1);
  }
  const int cpr = W >> 3;
  for (int i = tid; i < ROWS * cpr; i += 256) {
    const int r = i / cpr, c = i - r * cpr;
    uint4 u = make_uint4(0u, 0u, 0u, 0u);
    if (h0 + r < H) u = *reinterpret_cast<const uint4*>(q + ((long long)b * H + h0 + r) * W + c * 8);
    *reinterpret_cast<uint4*>(smem + lay.q + (c >> 3) * (ROWS * 128) + r * 128 + (((c ^ r) & 7) << 4)) = u;
  }
  __syncthreads();

  const int kg = warp & 3, kh = warp >> 2, steps = W / 32;      // this warp's 16 keys and half of the contraction
  const int srow = tid / TPR, skey = (tid % TPR) * KPT;         // this thread's row of scores and its keys
  float m = -INFINITY, l = 0.f;
  float o[MT][CB][8];
#pragma unroll
  for (int x = 0; x < MT; ++x)
#pragma unroll
    for (int i = 0; i < CB; ++i)
#pragma unroll
      for (int k = 0; k < 8; ++k) o[x][i][k] = 0.f;

  for (int tile = 0; tile < n_tiles; ++tile) {
    const uint32_t kb = base + (tile & 1) * lay.stage;
    if (!mbar_wait_bounded(smem_u32(&full_bars[tile & 1]), (tile >> 1) & 1, &abort_flag, status, ST_TIMEOUT_PRODUCER)) break;
    {
      float s[MT][2][4];
#pragma unroll
      for (int x = 0; x < MT; ++x)
#pragma unroll
        for (int k = 0; k < 4; ++k) s[x][0][k] = s[x][1][k] = 0.f;
#pragma unroll 4
      for (int ks = kh * steps; ks < (kh + 1) * steps; ++ks) {
        uint32_t kf[4];
        {
          const int r = kg * 16 + (li >> 1) * 8 + lr, c = ks * 2 + (li & 1);
          ldsm_x4(kf, kb + (c >> 3) * 8192 + r * 128 + (((c ^ r) & 7) << 4));
        }
#pragma unroll
        for (int x = 0; x < MT; ++x) {
          uint32_t a[4];
          const int r = x * 16 + (li & 1) * 8 + lr, c = ks * 2 + (li >> 1);
          ldsm_x4(a, sq + (c >> 3) * (ROWS * 128) + r * 128 + (((c ^ r) & 7) << 4));
          mma_16816(s[x][0], a, kf[0], kf[1]);
          mma_16816(s[x][1], a, kf[2], kf[3]);
        }
      }
#pragma unroll
      for (int x = 0; x < MT; ++x)
#pragma unroll
        for (int nb = 0; nb < 2; ++nb) {
          float* d = s_s + (kh * ROWS + x * 16 + (lane >> 2)) * 68 + kg * 16 + nb * 8 + 2 * (lane & 3);
          *reinterpret_cast<float2*>(d) = make_float2(s[x][nb][0], s[x][nb][1]);
          *reinterpret_cast<float2*>(d + 8 * 68) = make_float2(s[x][nb][2], s[x][nb][3]);
        }
    }
    __syncthreads();
    {
      const int t0 = kt.start(tile0 + tile) + skey;
      float v[KPT], mx = -INFINITY;
#pragma unroll
      for (int k = 0; k < KPT; k += 4) {
        const float4 a = *reinterpret_cast<const float4*>(s_s + srow * 68 + skey + k);
        const float4 c = *reinterpret_cast<const float4*>(s_s + (ROWS + srow) * 68 + skey + k);
        v[k] = a.x + c.x; v[k + 1] = a.y + c.y; v[k + 2] = a.z + c.z; v[k + 3] = a.w + c.w;
      }
#pragma unroll
      for (int k = 0; k < KPT; ++k) {
        v[k] = t0 + k < len && t0 + k >= kt.w_lo ? v[k] * scale : -INFINITY;
        mx = fmaxf(mx, v[k]);
      }
#pragma unroll
      for (int x = TPR / 2; x >= 1; x >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, x));
      const float mn = fmaxf(m, mx), c = m == -INFINITY ? 0.f : quick_exp(m - mn);
      float ps = 0.f;
#pragma unroll
      for (int k = 0; k < KPT; ++k) {
        v[k] = v[k] == -INFINITY ? 0.f : quick_exp(v[k] - mn);
        ps += v[k];
      }
      l = l * c + ps;
      m = mn;
      if (tid % TPR == 0) s_alpha[srow] = c;
      uint8_t* d = smem + lay.p + srow * 128 + ((((skey >> 3) ^ srow) & 7) << 4) + (skey & 7) * 2;
      if (KPT == 8)
        *reinterpret_cast<uint4*>(d) = make_uint4(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]), pack_bf16(v[KPT - 4], v[KPT - 3]), pack_bf16(v[KPT - 2], v[KPT - 1]));
      else
        *reinterpret_cast<uint2*>(d) = make_uint2(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]));
    }
    __syncthreads();
#pragma unroll
    for (int x = 0; x < MT; ++x) {
      const float a0 = s_alpha[x * 16 + (lane >> 2)], a1 = s_alpha[x * 16 + (lane >> 2) + 8];
#pragma unroll
      for (int i = 0; i < CB; ++i) {
        o[x][i][0] *= a0; o[x][i][1] *= a0; o[x][i][4] *= a0; o[x][i][5] *= a0;
        o[x][i][2] *= a1; o[x][i][3] *= a1; o[x][i][6] *= a1; o[x][i][7] *= a1;
      }
    }
#pragma unroll
    for (int kk = 0; kk < 4; ++kk) {
      uint32_t a[MT][4];
#pragma unroll
      for (int x = 0; x < MT; ++x) {
        const int r = x * 16 + (li & 1) * 8 + lr, c = kk * 2 + (li >> 1);
        ldsm_x4(a[x], sp + r * 128 + (((c ^ r) & 7) << 4));
      }
#pragma unroll
      for (int i = 0; i < CB; ++i) {
        const int nb = warp + 8 * i;
        if (nb * 16 < R) {                                      // the whole warp
          uint32_t vf[4];
          const int r = kk * 16 + (li & 1) * 8 + lr, c = nb * 2 + (li >> 1);
          ldsm_x4_t(vf, kb + (c >> 3) * 8192 + r * 128 + (((c ^ r) & 7) << 4));
#pragma unroll
          for (int x = 0; x < MT; ++x) {
            float(&lo)[4] = *reinterpret_cast<float(*)[4]>(&o[x][i][0]);
            float(&hi)[4] = *reinterpret_cast<float(*)[4]>(&o[x][i][4]);
            mma_16816(lo, a[x], vf[0], vf[1]);
            mma_16816(hi, a[x], vf[2], vf[3]);
          }
        }
      }
    }
    __syncthreads();
    if (tid == 0 && tile + 2 < n_tiles) issue(tile + 2);        // into the buffer that everyone has just left
  }
#pragma unroll
  for (int x = TPR / 2; x >= 1; x >>= 1) l += __shfl_xor_sync(0xffffffffu, l, x);
  if (tid % TPR == 0) {
    s_alpha[ROWS + srow] = m;
    s_alpha[2 * ROWS + srow] = l;
    const int h = h0 + srow;
    if (num_splits > 1 && h < H) {
      float* ml = part_ml + (((long long)b * H + h) * num_splits + split) * 2;
      ml[0] = m;
      ml[1] = l;
    }
  }
  __syncthreads();
#pragma unroll
  for (int x = 0; x < MT; ++x)
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int r = x * 16 + (lane >> 2) + 8 * half, h = h0 + r;
      if (h >= H) continue;
      const float inv = 1.f / (s_alpha[2 * ROWS + r] + quick_exp(ex.sink_of(h) - s_alpha[ROWS + r]));
#pragma unroll
      for (int i = 0; i < CB; ++i)
#pragma unroll
        for (int g = 0; g < 2; ++g) {
          const int d = (warp + 8 * i) * 16 + g * 8 + 2 * (lane & 3);
          if (d >= R) continue;
          const float v0 = o[x][i][4 * g + 2 * half], v1 = o[x][i][4 * g + 2 * half + 1];
          if (num_splits == 1)
            *reinterpret_cast<uint32_t*>(out + ((long long)b * H + h) * R + d) = pack_bf16(v0 * inv, v1 * inv);
          else
            *reinterpret_cast<float2*>(part_acc + (((long long)b * H + h) * num_splits + split) * R + d) = make_float2(v0, v1);
        }
    }
}

template <int CB, int MT>
int launch_latent_decode(const CUtensorMap& tm, dim3 grid, cudaStream_t stream, const __nv_bfloat16* q, const int* table, int max_pages,
                         int page_size, const int* seq_ids, const int* seq_lens, int H, int R, int W, float scale, int window,
                         HeadExtras ex, int splits, int split_tokens, float* pa, float* pml, __nv_bfloat16* out, int* status) {
  static DeviceOnce once;
  if (once.first() && cudaFuncSetAttribute(latent_decode_kernel<CB, MT>, cudaFuncAttributeMaxDynamicSharedMemorySize, 226 * 1024) != cudaSuccess)
    return -5;
  const int smem = LatentSmem(W, MT * 16).total + 1024;
  if (smem > 226 * 1024) return -2;
  return launch_pdl(latent_decode_kernel<CB, MT>, grid, dim3(256), smem, stream, tm, q, table, max_pages, page_size, seq_ids, seq_lens, H, R,
                    W, scale, window, ex, splits, split_tokens, pa, pml, out, status) == cudaSuccess ? 0 : -5;
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
  CUtensorMap tm;
  if (tb_make_tmap_2d_bf16(&tm, pool, (uint64_t)pool_rows, (uint64_t)W, (uint64_t)W, TILE_KEYS, 64, 1)) return -3;
  const int per = split_tokens / TILE_KEYS, splits = (tiles + per - 1) / per;
  const HeadExtras ex{-INFINITY, sinks, nullptr, 0};
  const bool two = H > 16;
  const dim3 grid(T, (H + (two ? 31 : 15)) / (two ? 32 : 16), splits);
  typedef __nv_bfloat16 bf;
  int rc;
#define RUN(CB, MT)                                                                                                                   \
  launch_latent_decode<CB, MT>(tm, grid, stream, (const bf*)q, table, max_pages, page_size, seq_ids, seq_lens, H, R, W, scale, window, ex, \
                               splits, split_tokens, part_acc, part_ml, (bf*)out, status)
  if (R <= 128) rc = two ? RUN(1, 2) : RUN(1, 1);
  else if (R <= 256) rc = two ? RUN(2, 2) : RUN(2, 1);
  else rc = two ? RUN(4, 2) : RUN(4, 1);
#undef RUN
  if (rc || splits == 1) return rc;
  return launch_pdl(paged_decode_combine_kernel, dim3(T, H), dim3(128), 0, stream, (const float*)part_acc, (const float*)part_ml, seq_lens, H,
                    R, splits, split_tokens, window, 0, 0, 1.f, R, ex, (bf*)out, (long long)H * R) == cudaSuccess ? 0 : -5;
}
