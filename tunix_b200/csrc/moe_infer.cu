// Mixture-of-experts feed-forwards of layer-stack models (forward only). T is the activation type (bf16 or float).
//
//   moe_route        : softmax over the experts' logits in fp32, the `top` experts by score (+ a correction that takes part in the
//                      choice only), their scores as weights; how many tokens of every block chose which expert.
//   moe_plan, moe_place : a row segment per expert (multiples of 128 rows) for the grouped tcgen05 GEMM (gemm.cu), and the row of
//                      every (token, choice). Padding rows of a segment are never read back, so nothing zeroes them.
//   moe_route_lists  : the same choice in one CTA for a decode step, with the choices sorted by expert.
//   expert_rows      : few rows per expert: a CTA streams 32 weight rows of one expert (16 gate and 16 up rows, or 32 down rows)
//                      past the rows that chose it, up to 64 at a time on mma.sync.
//   expert_plain     : any sizes, also 32-bit: a warp per choice and output.
//   moe_sum          : the sum over a token's choices.
// A choice is numbered token * top + j. Tokens of idle slots choose nothing (expert -1).
//
// This file is compiled without fast-math: the same kernels serve the 32-bit mode.
#include "mma.cuh"
#include "precise.cuh"

using namespace tb;

namespace {

typedef __nv_bfloat16 bf;
constexpr int BLOCK_TOKENS = 128;      // tokens per block of moe_route / moe_place
constexpr int MAX_EXPERTS = 1024;

// One warp routes one token: z [E] logits. Lane l holds experts l, l + 32, ...
template <typename T, int NE>
__device__ __forceinline__ void route_token(const float* z, const T* correction, int E, int top, int* idx, float* wts, int* hist) {
  const int lane = threadIdx.x & 31;
  float s[NE], c[NE], m = -INFINITY, sum = 0.f;
#pragma unroll
  for (int i = 0; i < NE; ++i) {
    const int e = lane + 32 * i;
    s[i] = e < E ? z[e] : -INFINITY;
    m = fmaxf(m, s[i]);
  }
  m = warp_max(m);
#pragma unroll
  for (int i = 0; i < NE; ++i) {
    s[i] = expf(s[i] - m);
    sum += s[i];
  }
  sum = warp_sum(sum);
#pragma unroll
  for (int i = 0; i < NE; ++i) {
    const int e = lane + 32 * i;
    s[i] /= sum;
    c[i] = e < E ? s[i] + (correction ? to_f(correction[e]) : 0.f) : -INFINITY;
  }
  for (int j = 0; j < top; ++j) {
    float best = -INFINITY, weight = 0.f;
    int at = E;
#pragma unroll
    for (int i = 0; i < NE; ++i)
      if (c[i] > best) { best = c[i]; at = lane + 32 * i; weight = s[i]; }
#pragma unroll
    for (int w = 16; w >= 1; w >>= 1) {
      const float b = __shfl_xor_sync(0xffffffffu, best, w), wt = __shfl_xor_sync(0xffffffffu, weight, w);
      const int a = __shfl_xor_sync(0xffffffffu, at, w);
      if (b > best || (b == best && a < at)) { best = b; at = a; weight = wt; }
    }
#pragma unroll
    for (int i = 0; i < NE; ++i)
      if (lane + 32 * i == at) c[i] = -INFINITY;
    if (lane == 0) {
      const bool ok = at < E;                          // false only where the logits are not numbers
      idx[j] = ok ? at : -1;
      wts[j] = ok ? weight : 0.f;
      if (ok) atomicAdd(hist + at, 1);
    }
  }
}

__device__ __forceinline__ void skip_token(int top, int* idx, float* wts) {
  for (int j = threadIdx.x & 31; j < top; j += 32) {
    idx[j] = -1;
    wts[j] = 0.f;
  }
}

template <typename T, int NE>
__global__ void __launch_bounds__(512)
moe_route_kernel(const float* __restrict__ z, const T* __restrict__ correction, Ragged rb, int E, int top, int* __restrict__ idx,
                 float* __restrict__ wts, int* __restrict__ hist) {
  __shared__ int h[MAX_EXPERTS];
  pdl_trigger();
  pdl_wait();
  for (int e = threadIdx.x; e < E; e += blockDim.x) h[e] = 0;
  __syncthreads();
  const int t0 = blockIdx.x * BLOCK_TOKENS, t1 = min(t0 + BLOCK_TOKENS, rb.n);
  for (int t = t0 + (threadIdx.x >> 5); t < t1; t += blockDim.x >> 5) {
    const long long o = (long long)t * top;
    if (rb.pos0[rb.ent[t]] < 0) skip_token(top, idx + o, wts + o);
    else route_token<T, NE>(z + (long long)t * E, correction, E, top, idx + o, wts + o, h);
  }
  __syncthreads();
  for (int e = threadIdx.x; e < E; e += blockDim.x) hist[(long long)blockIdx.x * E + e] = h[e];
}

// hist [blocks, E] -> first row of every (block, expert) in place, seg_off [E + 1]; one CTA, a thread per expert
__global__ void __launch_bounds__(MAX_EXPERTS)
moe_plan_kernel(int* __restrict__ hist, int blocks, int E, int* __restrict__ seg_off) {
  __shared__ int off[MAX_EXPERTS + 1];
  pdl_trigger();
  pdl_wait();
  const int e = threadIdx.x;
  int total = 0;
  if (e < E) {
#pragma unroll 8
    for (int b = 0; b < blocks; ++b) total += hist[(long long)b * E + e];
    off[e + 1] = (total + 127) & ~127;
  }
  __syncthreads();
  if (e == 0) {
    off[0] = 0;
    for (int i = 0; i < E; ++i) off[i + 1] += off[i];
  }
  __syncthreads();
  if (e <= E) seg_off[e] = off[e];
  if (e == 0) seg_off[E] = off[E];
  if (e < E) {
    int at = off[e];
    for (int b0 = 0; b0 < blocks; b0 += 8) {
      int v[8];
#pragma unroll
      for (int i = 0; i < 8; ++i) v[i] = b0 + i < blocks ? hist[(long long)(b0 + i) * E + e] : 0;
#pragma unroll
      for (int i = 0; i < 8; ++i)
        if (b0 + i < blocks) {
          hist[(long long)(b0 + i) * E + e] = at;
          at += v[i];
        }
    }
  }
}

__global__ void __launch_bounds__(512)
moe_place_kernel(const int* __restrict__ idx, const int* __restrict__ base, int n, int E, int top, int* __restrict__ pos) {
  __shared__ int next[MAX_EXPERTS];
  pdl_trigger();
  pdl_wait();
  for (int e = threadIdx.x; e < E; e += blockDim.x) next[e] = base[(long long)blockIdx.x * E + e];
  __syncthreads();
  const long long i0 = (long long)blockIdx.x * BLOCK_TOKENS * top, i1 = min(i0 + (long long)BLOCK_TOKENS * top, (long long)n * top);
  for (long long i = i0 + threadIdx.x; i < i1; i += blockDim.x) {
    const int e = idx[i];
    pos[i] = e < 0 ? -1 : atomicAdd(next + e, 1);      // the order inside a segment does not matter: rows are independent
  }
}

template <typename T, int NE>
__global__ void __launch_bounds__(1024)
moe_route_lists_kernel(const float* __restrict__ z, const T* __restrict__ correction, Ragged rb, int E, int top, int* __restrict__ idx,
                       float* __restrict__ wts, int* __restrict__ off, int* __restrict__ list) {
  __shared__ int h[MAX_EXPERTS];
  pdl_trigger();
  pdl_wait();
  for (int e = threadIdx.x; e < E; e += blockDim.x) h[e] = 0;
  __syncthreads();
  for (int t = threadIdx.x >> 5; t < rb.n; t += blockDim.x >> 5) {
    const long long o = (long long)t * top;
    if (rb.pos0[rb.ent[t]] < 0) skip_token(top, idx + o, wts + o);
    else route_token<T, NE>(z + (long long)t * E, correction, E, top, idx + o, wts + o, h);
  }
  __syncthreads();
  if (threadIdx.x < 32) {                              // exclusive sums over the experts, 32 at a time
    int carry = 0;
    for (int e0 = 0; e0 < E; e0 += 32) {
      const int e = e0 + threadIdx.x, v = e < E ? h[e] : 0;
      int s = v;
#pragma unroll
      for (int w = 1; w < 32; w <<= 1) {
        const int u = __shfl_up_sync(0xffffffffu, s, w);
        if (threadIdx.x >= w) s += u;
      }
      if (e < E) {
        h[e] = carry + s - v;
        off[e] = carry + s - v;
      }
      carry += __shfl_sync(0xffffffffu, s, 31);
    }
    if (threadIdx.x == 0) off[E] = carry;
  }
  __syncthreads();
  const long long total = (long long)rb.n * top;
  for (long long i = threadIdx.x; i < total; i += blockDim.x) {
    const int e = idx[i];
    if (e >= 0) list[atomicAdd(h + e, 1)] = (int)i;
  }
}

// Rows of one expert, up to 64 at a time, times 32 of its weight rows. GLU: x rows belong to tokens, out[choice, f] = silu(gate) *
// up for 16 f, T. Otherwise x rows belong to choices, out[choice, d] = weight * product for 32 d, fp32. The warps of a CTA split
// the contraction and meet in shared memory; both operands of a product see the same permutation of k, so nothing is shuffled.
__host__ __device__ constexpr int row_warps(bool glu) { return glu ? 8 : 4; }      // shorter contractions: fewer warps, more CTAs
template <bool GLU, int MT, int RW>
__device__ __forceinline__ void expert_pass(const bf* x, long long ldx, const bf* const (&wr)[4], int K, int N, const int* list, int left,
                                            const float* wts, int top, int n0, float (&part)[RW][16][33], void* out) {
  constexpr int TILE = GLU ? 16 : 32;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, q8 = (lane & 3) * 8;
  const bf* xr[MT][2];
  float acc[MT][4][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int c = list[min(m * 16 + h * 8 + g, left - 1)];
      xr[m][h] = x + (GLU ? c / top : c) * ldx;
#pragma unroll
      for (int j = 0; j < 4; ++j) acc[m][j][2 * h] = acc[m][j][2 * h + 1] = 0.f;
    }
#pragma unroll (MT == 1 ? 4 : MT == 2 ? 2 : 1)
  for (int kb = warp * 32; kb < K; kb += RW * 32) {             // whole warps stay together for the products
    const int k = kb + q8;                                      // K is a multiple of 8: a lane's 8 elements are in or out
    const uint4 zero = make_uint4(0u, 0u, 0u, 0u);
    uint4 w[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) w[j] = k < K ? __ldg(reinterpret_cast<const uint4*>(wr[j] + k)) : zero;
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      const uint4 a = k < K ? *reinterpret_cast<const uint4*>(xr[m][0] + k) : zero, b = k < K ? *reinterpret_cast<const uint4*>(xr[m][1] + k) : zero;
      const uint32_t s0[4] = {a.x, b.x, a.y, b.y}, s1[4] = {a.z, b.z, a.w, b.w};
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        mma_16816(acc[m][j], s0, w[j].x, w[j].y);
        mma_16816(acc[m][j], s1, w[j].z, w[j].w);
      }
    }
  }
  const int c2 = 2 * (lane & 3);
#pragma unroll
  for (int m = 0; m < MT; ++m) {
#pragma unroll
    for (int j = 0; j < 4; ++j)
#pragma unroll
      for (int i = 0; i < 4; ++i) part[warp][g + (i >> 1) * 8][j * 8 + c2 + (i & 1)] = acc[m][j][i];
    __syncthreads();
    for (int i = threadIdx.x; i < 16 * TILE; i += 32 * RW) {
      const int r = i / TILE, c = i % TILE, col = n0 + c;
      if (m * 16 + r < left && col < N) {
        const int choice = list[m * 16 + r];
        float v = 0.f, u = 0.f;
#pragma unroll
        for (int j = 0; j < RW; ++j) {
          v += part[j][r][c];
          if (GLU) u += part[j][r][16 + c];
        }
        if (GLU) static_cast<bf*>(out)[(long long)choice * N + col] = __float2bfloat16(v * quick_sigmoid(v) * u);
        else static_cast<float*>(out)[(long long)choice * N + col] = wts[choice] * v;
      }
    }
    __syncthreads();
  }
}

template <bool GLU>
__global__ void __launch_bounds__(32 * row_warps(GLU), 16 / row_warps(GLU))
expert_rows_kernel(const bf* __restrict__ x, long long ldx, const bf* __restrict__ w, int K, int N, const int* __restrict__ off,
                   const int* __restrict__ list, const float* __restrict__ wts, int top, void* __restrict__ out) {
  constexpr int RW = row_warps(GLU);
  __shared__ float part[RW][16][33];
  pdl_trigger();
  pdl_wait();
  const int e = blockIdx.y, i0 = off[e], i1 = off[e + 1];
  if (i0 >= i1) return;
  const int g = (threadIdx.x & 31) >> 2, n0 = blockIdx.x * (GLU ? 16 : 32);
  // this lane's four weight rows: GLU gate n0 + g, + 8, then up; otherwise n0 + g + 8 j. Rows past N repeat the last one.
  const bf* wr[4];
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const int r = GLU ? min(n0 + (j & 1) * 8 + g, N - 1) + (j >> 1) * N : min(n0 + j * 8 + g, N - 1);
    wr[j] = w + ((long long)e * (GLU ? 2 * N : N) + r) * K;
  }
  for (int r0 = i0; r0 < i1;) {
    const int left = i1 - r0;
    if (left > 32) {
      expert_pass<GLU, 4, RW>(x, ldx, wr, K, N, list + r0, left, wts, top, n0, part, out);
      r0 += 64;
    } else if (left > 16) {
      expert_pass<GLU, 2, RW>(x, ldx, wr, K, N, list + r0, left, wts, top, n0, part, out);
      r0 += 32;
    } else {
      expert_pass<GLU, 1, RW>(x, ldx, wr, K, N, list + r0, left, wts, top, n0, part, out);
      r0 += 16;
    }
  }
}

// A warp per (choice, output). GLU: w [E, 2 N, K], gate rows before up rows; otherwise w [E, N, K].
template <typename T, bool GLU>
__global__ void __launch_bounds__(256)
expert_plain_kernel(const T* __restrict__ x, long long ldx, const T* __restrict__ w, int K, int N, const int* __restrict__ idx,
                    const float* __restrict__ wts, int top, long long choices, void* __restrict__ out) {
  pdl_trigger();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const long long total = choices * N, step = (long long)gridDim.x * (blockDim.x >> 5);
  for (long long i = (long long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5); i < total; i += step) {
    const long long c = i / N;
    const int o = (int)(i - c * N), e = idx[c];
    if (e < 0) continue;
    const T* xr = x + (GLU ? c / top : c) * ldx;
    const T* w0 = w + ((long long)e * (GLU ? 2 * N : N) + o) * K;
    float v = 0.f, u = 0.f;
    for (int k = lane; k < K; k += 32) {
      const float xv = to_f(xr[k]);
      v += xv * to_f(w0[k]);
      if (GLU) u += xv * to_f(w0[(long long)N * K + k]);
    }
    v = warp_sum(v);
    if (GLU) u = warp_sum(u);
    if (lane == 0) {
      if (GLU) static_cast<T*>(out)[i] = from_f<T>(v * sigmoid(v) * u);
      else static_cast<float*>(out)[i] = wts[c] * v;
    }
  }
}

// out[t] = sum over the token's choices of y fp32 [choices, D]
template <typename T, int V>
__global__ void __launch_bounds__(256)
moe_sum_kernel(const float* __restrict__ y, const int* __restrict__ idx, int n, int top, int D, T* __restrict__ out) {
  pdl_trigger();
  pdl_wait();
  const long long per = D / V, total = (long long)n * per;
  for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const long long t = i / per;
    const int d = (int)(i - t * per) * V;
    float acc[V];
#pragma unroll
    for (int q = 0; q < V; ++q) acc[q] = 0.f;
    for (int j = 0; j < top; ++j) {
      if (idx[t * top + j] < 0) continue;
      float v[V];
      load_v<V>(y + (t * top + j) * D + d, v);
#pragma unroll
      for (int q = 0; q < V; ++q) acc[q] += v[q];
    }
    store_v<V>(out + t * D + d, acc);
  }
}

dim3 blocks_for(long long work) {
  const long long want = (work + 255) / 256;
  return dim3((unsigned)(want < 148 * 16 ? want : 148 * 16));
}

}  // namespace

#define BY_EXPERTS(RUN, T) \
  (E <= 32 ? RUN(T, 1) : E <= 64 ? RUN(T, 2) : E <= 128 ? RUN(T, 4) : E <= 256 ? RUN(T, 8) : RUN(T, 32))

// z fp32 [n, E] router logits, correction T [E] or null -> idx int32 [n, top], wts fp32 [n, top], pos int32 [n, top] (row of the
// permuted buffer, -1: none), seg_off int32 [E + 1]. hist: int32 [ceil(n / 128), E] workspace.
TB_API int tb_moe_route(int dtype, const float* z, const void* correction, const int* cu, const int* slot, const int* pos0,
                        const int* ent, int Eb, int n, int E, int top, int* idx, float* wts, int* hist, int* seg_off, int* pos,
                        cudaStream_t stream) {
  if (n <= 0) return 0;
  if (E < 1 || E > MAX_EXPERTS || top < 1 || top > E) return -2;
  Ragged rb{cu, slot, pos0, ent, Eb, n};
  const int blocks = (n + BLOCK_TOKENS - 1) / BLOCK_TOKENS;
#define RT(T, NE) launch_pdl(moe_route_kernel<T, NE>, dim3(blocks), dim3(512), 0, stream, z, (const T*)correction, rb, E, top, idx, wts, hist)
  if ((dtype == 0 ? BY_EXPERTS(RT, bf) : BY_EXPERTS(RT, float)) != cudaSuccess) return -5;
#undef RT
  const int threads = ((E + 1 + 31) / 32) * 32;
  if (launch_pdl(moe_plan_kernel, dim3(1), dim3(threads < MAX_EXPERTS ? threads : MAX_EXPERTS), 0, stream, hist, blocks, E, seg_off) != cudaSuccess) return -5;
  return launch_pdl(moe_place_kernel, dim3(blocks), dim3(512), 0, stream, (const int*)idx, (const int*)hist, n, E, top, pos) == cudaSuccess ? 0 : -5;
}

// The same choice with off int32 [E + 1] and list int32 [n * top]: the choices of expert e are list[off[e]] .. list[off[e + 1] - 1].
TB_API int tb_moe_route_lists(int dtype, const float* z, const void* correction, const int* cu, const int* slot, const int* pos0,
                              const int* ent, int Eb, int n, int E, int top, int* idx, float* wts, int* off, int* list,
                              cudaStream_t stream) {
  if (n <= 0) return 0;
  if (E < 1 || E > MAX_EXPERTS || top < 1 || top > E) return -2;
  Ragged rb{cu, slot, pos0, ent, Eb, n};
#define RL(T, NE) launch_pdl(moe_route_lists_kernel<T, NE>, dim3(1), dim3(1024), 0, stream, z, (const T*)correction, rb, E, top, idx, wts, off, list)
  return (dtype == 0 ? BY_EXPERTS(RL, bf) : BY_EXPERTS(RL, float)) == cudaSuccess ? 0 : -5;
#undef RL
}

// x T [n, ldx]; wgu T [E, 2 F, D] (gate rows, then up rows), wd T [E, D, F]; act T [n * top, F] and y fp32 [n * top, D] workspaces;
// out T [n, D]. rows: bf16 with D and F multiples of 8 and ldx a multiple of 8, by expert lists; otherwise choice by choice.
TB_API int tb_moe_experts(int dtype, int rows, const void* x, long long ldx, const void* wgu, const void* wd, int n, int D, int F, int E,
                          int top, const int* idx, const float* wts, const int* off, const int* list, void* act, float* y, void* out,
                          cudaStream_t stream) {
  if (n <= 0) return 0;
  const long long choices = (long long)n * top;
  cudaError_t err;
  if (rows) {
    if (dtype != 0 || D % 8 || F % 8 || ldx % 8 || E > 65535 || ((uintptr_t)x & 15) || ((uintptr_t)wgu & 15) || ((uintptr_t)wd & 15)) return -2;
    err = launch_pdl(expert_rows_kernel<true>, dim3((F + 15) / 16, E), dim3(32 * row_warps(true)), 0, stream, (const bf*)x, ldx, (const bf*)wgu, D, F,
                     off, list, wts, top, act);
    if (err != cudaSuccess) return -5;
    err = launch_pdl(expert_rows_kernel<false>, dim3((D + 31) / 32, E), dim3(32 * row_warps(false)), 0, stream, (const bf*)act, (long long)F,
                     (const bf*)wd, F, D, off, list, wts, top, (void*)y);
    if (err != cudaSuccess) return -5;
  } else {
    const dim3 g1 = blocks_for(choices * F * 32), g2 = blocks_for(choices * D * 32);
#define PL(T)                                                                                                                  \
  (launch_pdl(expert_plain_kernel<T, true>, g1, dim3(256), 0, stream, (const T*)x, ldx, (const T*)wgu, D, F, idx, wts, top,     \
              choices, act) != cudaSuccess ||                                                                                  \
   launch_pdl(expert_plain_kernel<T, false>, g2, dim3(256), 0, stream, (const T*)act, (long long)F, (const T*)wd, F, D, idx,     \
              wts, top, choices, (void*)y) != cudaSuccess)
    if (dtype == 0 ? PL(bf) : PL(float)) return -5;
#undef PL
  }
  const bool vec = D % 4 == 0;
  const dim3 g = blocks_for((long long)n * D / (vec ? 4 : 1));
#define SM(T, V) launch_pdl(moe_sum_kernel<T, V>, g, dim3(256), 0, stream, (const float*)y, idx, n, top, D, (T*)out)
  err = dtype == 0 ? (vec ? SM(bf, 4) : SM(bf, 1)) : (vec ? SM(float, 4) : SM(float, 1));
#undef SM
  return err == cudaSuccess ? 0 : -5;
}
