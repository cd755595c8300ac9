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

}  // namespace

#define RAGGED Ragged rb{cu, slot, pos0, ent, E, n}

// x and y are columns x_off.. and y_off.. of proj [n, ldp]. u / A / B: workspaces [n, W] (T, fp32, fp32).
// state fp32 [slots, W], ring fp32 [slots, K, W]; out T [n, W].
TB_API int tb_rglru(int dtype, const void* proj, long long ldp, int x_off, int y_off, const void* conv_w, const void* conv_b,
                    const void* ra, const void* rab, const void* ri, const void* rib, const void* lam, const int* cu,
                    const int* slot, const int* pos0, const int* ent, int E, int n, int W, int K, int blocks, float* state,
                    float* ring, void* u, float* A, float* B, void* out, cudaStream_t stream) {
  if (n <= 0 || E <= 0) return 0;
  if (blocks <= 0 || W % blocks || K < 1 || n > 65535 * GT) return -2;
  const int bs = W / blocks;
  RAGGED;
  const dim3 gconv((W + 127) / 128, n), ggate((bs + GC - 1) / GC, blocks, (n + GT - 1) / GT), gscan((W + 63) / 64, E);
  if (n > 65535 || ggate.z > 65535 || E > 65535) return -2;
  const size_t smem = (size_t)GT * bs * 4;
#define RUN(T)                                                                                                              \
  {                                                                                                                         \
    static DeviceOnce once;                                                                                                 \
    if (smem > 200 * 1024) return -2;                                                                                       \
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
TB_API int tb_mlstm_seq(int dtype, const void* proj, long long ldp, int q_off, int k_off, int v_off, const float* gates,
                        const void* ib, const void* fb, float cap, const int* cu, const int* slot, const int* pos0,
                        const int* ent, int E, int n, int heads, int dk, int dv, float* S, float* N, float* M, float* out,
                        cudaStream_t stream) {
  if (n <= 0 || E <= 0) return 0;
  if (E > 65535 || heads > 65535) return -2;
  RAGGED;
  const size_t smem = ((size_t)dk * (MV + 3) + MV * 9) * 4;
  if (smem > 200 * 1024) return -2;
  const dim3 grid(tb_mlstm_slices(dv), heads, E);
#define RUN(T)                                                                                                              \
  {                                                                                                                         \
    static DeviceOnce once;                                                                                                 \
    if (once.first() && cudaFuncSetAttribute(mlstm_seq_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize,              \
                                             200 * 1024) != cudaSuccess) return -5;                                         \
    cudaError_t err = launch_pdl(mlstm_seq_kernel<T>, grid, dim3(MTHREADS), smem, stream, (const T*)proj, ldp, q_off, k_off, \
                                 v_off, gates, (const T*)ib, (const T*)fb, cap, rb, heads, dk, dv, S, N, M, out);            \
    return err == cudaSuccess ? 0 : -5;                                                                                     \
  }
  if (dtype == 0) RUN(__nv_bfloat16) else RUN(float)
#undef RUN
}
