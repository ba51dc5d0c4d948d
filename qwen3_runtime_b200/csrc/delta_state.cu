// The gated delta rule with a decay per key channel, on a matrix state S [D, Dv] per (sequence, head):
//
//   S <- diag(g_t) S;   u = beta_t (v_t - S^T k_t);   S <- S + k_t u^T;   o_t = S^T q_t
//
// and what surrounds it: a short causal convolution with silu on every channel of q, k and v, unit vectors for q
// and k per head, g = exp(neg_a_h * softplus(z + dt_bias)), beta = sigmoid(b).  q and k have G heads, v and the
// state H = a multiple of G; head h reads q/k head h / (H / G).  The state, decays, steps, unit vectors and all
// sums are fp32.
//
// The convolution's past inputs live in a ring of `taps` rows per state slot (fp32 [taps, C]; the input of
// position p sits in row p mod taps), so a step that brings one token writes its row beside the rows that are
// still read.  Rows of positions before the sequence's start are never read: they count as zeros.
//
//   delta_prepare    every token of a step: convolution, silu, unit vectors, decays and steps as rows in memory
//   ring_update      the last rows of every sequence's portion into the ring (after delta_prepare has read it)
//   delta_scan       the recurrence over every sequence's tokens of the step, from delta_prepare's rows
//   delta_chunk_*    the same in chunks of 16 tokens, for prompts
//   delta_step       all of it for steps in which every sequence brings one token, with the decay's and the
//                    gate's second low-rank products and the heads' output norm and gate: one kernel
#include "common.cuh"

#define DELTA_MAX_TAPS 16
#define UNIT_EPS 1e-6f

static inline bool ds_aligned(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

__device__ __forceinline__ float softplus_f(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }
__device__ __forceinline__ float sigmoid_f(float x) { return 1.f / (1.f + expf(-x)); }

// E (1 or 8) consecutive channels' convolution at token t of the step, n rows into its sequence's portion, at
// position p; ring: the slot's rows.  w: fp32 [taps, C].
template <typename T, int E>
__device__ __forceinline__ void conv_silu(const T* __restrict__ xrow, long x_stride, const float* __restrict__ w,
                                          int taps, const float* __restrict__ ring, int C, int n, int p, int c,
                                          float (&y)[E]) {
#pragma unroll
  for (int e = 0; e < E; ++e) y[e] = 0.f;
#pragma unroll 4
  for (int j = 0; j < taps; ++j) {
    const int back = taps - 1 - j;
    if (p - back < 0) continue;
    float u[E], wv[E];
    if constexpr (E == 8) {
      if (n - back >= 0) load8(xrow - (long)back * x_stride + c, u);
      else load8(ring + (long)((p - back) % taps) * C + c, u);
      load8(w + (long)j * C + c, wv);
    } else {
      u[0] = n - back >= 0 ? to_f32(xrow[-(long)back * x_stride + c]) : ring[(long)((p - back) % taps) * C + c];
      wv[0] = w[(long)j * C + c];
    }
#pragma unroll
    for (int e = 0; e < E; ++e) y[e] = fmaf(wv[e], u[e], y[e]);
  }
#pragma unroll
  for (int e = 0; e < E; ++e) y[e] = y[e] * sigmoid_f(y[e]);
}

// Warps of a block take the token's work items: groups of q and k heads (a warp holds 32 / lph heads, lph lanes of E
// elements each and, for E = 1, up to 8 strided elements), then groups of 32 * E value channels, then groups of
// 32 * E decays, then the steps.  v is kept in the activation type; q and k are normalised from the convolution's
// fp32 values.
template <typename T, int E>
__global__ void __launch_bounds__(256)
delta_prepare_kernel(const T* __restrict__ x, long x_stride, const float* __restrict__ w, int taps,
                     const float* __restrict__ ring, const int* __restrict__ positions,
                     const int* __restrict__ token_seq, const int* __restrict__ cu_seqlens,
                     const int* __restrict__ state_slots, const float* __restrict__ z, const float* __restrict__ dt_bias,
                     const float* __restrict__ neg_a, const T* __restrict__ b, long b_stride, float q_scale,
                     float* __restrict__ qn, float* __restrict__ kn, T* __restrict__ vc, float* __restrict__ g,
                     float* __restrict__ beta, int G, int H, int D, int Dv, int lph) {
  pdl_wait();
  pdl_launch_dependents();
  const int t = blockIdx.x, lane = threadIdx.x & 31;
  int item = blockIdx.y * (blockDim.x >> 5) + (threadIdx.x >> 5);
  const int seq = token_seq[t], p = positions[t], n = t - cu_seqlens[seq];
  const int C = 2 * G * D + H * Dv;
  const T* xrow = x + (long)t * x_stride;
  const float* rows = taps > 1 ? ring + (long)state_slots[seq] * taps * C : nullptr;
  const int per_warp = 32 / lph;
  const int qk_items = (2 * G + per_warp - 1) / per_warp, v_items = (H * Dv + 32 * E - 1) / (32 * E),
            g_items = (H * D + 32 * E - 1) / (32 * E);
  if (item < qk_items) {
    const int head = item * per_warp + lane / lph;  // q heads, then k heads
    const bool live_head = head < 2 * G;
    constexpr int M = E == 8 ? 1 : 8;               // strided groups of a lane (E = 1: elements lane + 32 m)
    float y[M][E];
    float ss = 0.f;
#pragma unroll
    for (int m = 0; m < M; ++m) {
      const int d = E == 8 ? (lane % lph) * 8 : lane + 32 * m;
#pragma unroll
      for (int e = 0; e < E; ++e) y[m][e] = 0.f;
      if (live_head && d < D) conv_silu<T, E>(xrow, x_stride, w, taps, rows, C, n, p, head * D + d, y[m]);
#pragma unroll
      for (int e = 0; e < E; ++e) ss += y[m][e] * y[m][e];
    }
    for (int o = lph >> 1; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if (!live_head) return;
    const float inv = rsqrtf(ss + UNIT_EPS) * (head < G ? q_scale : 1.f);
    float* dst = head < G ? qn + ((long)t * G + head) * D : kn + ((long)t * G + head - G) * D;
#pragma unroll
    for (int m = 0; m < M; ++m) {
      const int d = E == 8 ? (lane % lph) * 8 : lane + 32 * m;
      if (d >= D) continue;
#pragma unroll
      for (int e = 0; e < E; ++e) y[m][e] *= inv;
      if constexpr (E == 8) store8(dst + d, y[m]); else dst[d] = y[m][0];
    }
    return;
  }
  item -= qk_items;
  if (item < v_items) {
    const int c = (item * 32 + lane) * E;
    if (c >= H * Dv) return;
    float y[E];
    conv_silu<T, E>(xrow, x_stride, w, taps, rows, C, n, p, 2 * G * D + c, y);
    T* dst = vc + (long)t * H * Dv + c;
    if constexpr (E == 8) store8(dst, y); else dst[0] = from_f32<T>(y[0]);
    return;
  }
  item -= v_items;
  if (item < g_items) {
    const int c = (item * 32 + lane) * E;
    if (c >= H * D) return;
    float zz[E], bb[E];
    if constexpr (E == 8) {
      load8(z + (long)t * H * D + c, zz);
      load8(dt_bias + c, bb);
    } else {
      zz[0] = z[(long)t * H * D + c];
      bb[0] = dt_bias[c];
    }
    const float a = neg_a[c / D];
#pragma unroll
    for (int e = 0; e < E; ++e) zz[e] = expf(a * softplus_f(zz[e] + bb[e]));
    float* dst = g + (long)t * H * D + c;
    if constexpr (E == 8) store8(dst, zz); else dst[0] = zz[0];
    return;
  }
  item -= g_items;
  const int h = item * 32 + lane;
  if (h < H) beta[(long)t * H + h] = sigmoid_f(to_f32(b[(long)t * b_stride + h]));
}

// x: [T, C] rows (q heads | k heads | v heads), w fp32 [taps, C], ring fp32 [slots, taps, C]; z fp32 [T, H * D];
// neg_a fp32 [H] (-exp of the stored logarithm); b [T, H] rows b_stride apart; qn, kn fp32 [T, G, D]; vc [T, H, Dv];
// g fp32 [T, H, D]; beta fp32 [T, H].
Q3_EXPORT int q3_delta_prepare(int dtype, const void* x, long x_stride, const float* w, int taps, const float* ring,
                               const int* positions, const int* token_seq, const int* cu_seqlens,
                               const int* state_slots, const float* z, const float* dt_bias, const float* neg_a,
                               const void* b, long b_stride, float q_scale, float* qn, float* kn, void* vc, float* g,
                               float* beta, int num_tokens, int G, int H, int D, int Dv, cudaStream_t stream) {
  if (!x || !w || !positions || !token_seq || !cu_seqlens || !state_slots || !z || !dt_bias || !neg_a || !b || !qn || !kn ||
      !vc || !g || !beta)
    return Q3_ERR_ARGUMENT;
  if (G < 1 || H < 1 || H % G || D < 1 || Dv < 1 || taps < 1 || (taps > 1 && !ring)) return Q3_ERR_ARGUMENT;
  if (D > 256 || taps > DELTA_MAX_TAPS) return Q3_ERR_UNSUPPORTED;
  if (num_tokens == 0) return Q3_OK;
  const bool vec = D % 8 == 0 && Dv % 8 == 0 && x_stride % 8 == 0 && ds_aligned(x) && ds_aligned(w) && ds_aligned(ring) &&
                   ds_aligned(z) && ds_aligned(dt_bias) && ds_aligned(qn) && ds_aligned(kn) && ds_aligned(vc) &&
                   ds_aligned(g);
  const int E = vec ? 8 : 1;
  int lph = 32;
  if (vec) {
    lph = 1;
    while (lph * 8 < D) lph <<= 1;
  }
  const int items = (2 * G + 32 / lph - 1) / (32 / lph) + (H * Dv + 32 * E - 1) / (32 * E) +
                    (H * D + 32 * E - 1) / (32 * E) + (H + 31) / 32;
  const dim3 grid(num_tokens, (items + 7) / 8);
  if (grid.y > 65535) return Q3_ERR_UNSUPPORTED;
  cudaError_t e;
#define Q3_DELTA_PREPARE(T, EE)                                                                                      \
  e = launch_pdl(delta_prepare_kernel<T, EE>, grid, dim3(256), 0, stream, (const T*)x, x_stride, w, taps, ring, positions, \
                 token_seq, cu_seqlens, state_slots, z, dt_bias, neg_a, (const T*)b, b_stride, q_scale, qn, kn, (T*)vc, g, \
                 beta, G, H, D, Dv, lph)
  if (dtype == Q3_DTYPE_F32) {
    if (vec) Q3_DELTA_PREPARE(float, 8); else Q3_DELTA_PREPARE(float, 1);
  } else if (dtype == Q3_DTYPE_BF16) {
    if (vec) Q3_DELTA_PREPARE(bf16, 8); else Q3_DELTA_PREPARE(bf16, 1);
  } else {
    return Q3_ERR_ARGUMENT;
  }
#undef Q3_DELTA_PREPARE
  return e == cudaSuccess ? Q3_OK : Q3_ERR_LAUNCH;
}

// The last taps rows of every sequence's portion into its ring (rows of earlier positions stay where they are).
template <typename T>
__global__ void ring_update_kernel(const T* __restrict__ x, long x_stride, float* __restrict__ ring,
                                   const int* __restrict__ positions, const int* __restrict__ cu_seqlens,
                                   const int* __restrict__ state_slots, int taps, int C, long total) {
  pdl_wait();
  pdl_launch_dependents();
  const long idx = (long)blockIdx.x * blockDim.x + threadIdx.x;
  if (idx >= total) return;
  const int seq = (int)(idx / C), c = (int)(idx - (long)seq * C);
  const int t0 = cu_seqlens[seq], t1 = cu_seqlens[seq + 1];
  float* rows = ring + (long)state_slots[seq] * taps * C;
  for (int t = max(t0, t1 - taps); t < t1; ++t) rows[(long)(positions[t] % taps) * C + c] = to_f32(x[(long)t * x_stride + c]);
}

Q3_EXPORT int q3_ring_update(int dtype, const void* x, long x_stride, float* ring, const int* positions,
                             const int* cu_seqlens, const int* state_slots, int taps, int C, int num_seqs,
                             cudaStream_t stream) {
  if (!x || !ring || !positions || !cu_seqlens || !state_slots || C < 1 || taps < 1) return Q3_ERR_ARGUMENT;
  const long total = (long)num_seqs * C;
  if (total == 0) return Q3_OK;
  const unsigned blocks = (unsigned)((total + 255) / 256);
  cudaError_t e;
  if (dtype == Q3_DTYPE_F32)
    e = launch_pdl(ring_update_kernel<float>, dim3(blocks), dim3(256), 0, stream, (const float*)x, x_stride, ring,
                   positions, cu_seqlens, state_slots, taps, C, total);
  else if (dtype == Q3_DTYPE_BF16)
    e = launch_pdl(ring_update_kernel<bf16>, dim3(blocks), dim3(256), 0, stream, (const bf16*)x, x_stride, ring, positions,
                   cu_seqlens, state_slots, taps, C, total);
  else
    return Q3_ERR_ARGUMENT;
  return e == cudaSuccess ? Q3_OK : Q3_ERR_LAUNCH;
}

// ---- the recurrence, token by token ------------------------------------------------------------------
// One block per (VT value columns, head, sequence).  A thread owns R key rows of one value column of the state in
// registers; the RG row groups of a column are neighbouring lanes of a warp, so the two sums a token needs -- the
// decayed state times k and times q -- are shuffle sums that run side by side: with them and k . q,
// o = (g S)^T q + u (k . q), so the output does not wait for the state's update.  Tokens come CT at a time through a
// double buffer in shared memory whose next half is fetched into registers while this one is worked on.
#define DS_CT 16
template <typename T, int RG, int R, int VT>
__global__ void __launch_bounds__(RG * VT)
delta_scan_kernel(const float* __restrict__ qn, const float* __restrict__ kn, const T* __restrict__ vc,
                  const float* __restrict__ g, const float* __restrict__ beta, float* __restrict__ state,
                  const int* __restrict__ cu_seqlens, const int* __restrict__ state_slots, float* __restrict__ out, int G,
                  int H, int D, int Dv) {
  constexpr int THREADS = RG * VT, DP = RG * R, CPW = 32 / RG;
  constexpr int EPT = DS_CT * DP / THREADS;
  constexpr int VPT = (DS_CT * VT + THREADS - 1) / THREADS;
  extern __shared__ __align__(16) float ds_smem[];
  float* qs = ds_smem;                           // [2][CT][DP]
  float* ks = qs + 2 * DS_CT * DP;
  float* gs = ks + 2 * DS_CT * DP;
  float* vs = gs + 2 * DS_CT * DP;               // [2][CT][VT]
  float* bs = vs + 2 * DS_CT * VT;               // [2][CT]
  pdl_wait();
  pdl_launch_dependents();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int rg = lane % RG, col = warp * CPW + lane / RG;
  const int h = blockIdx.y, seq = blockIdx.z, gh = h / (H / G);
  const int j = blockIdx.x * VT + col;
  const int t0 = cu_seqlens[seq], t1 = cu_seqlens[seq + 1];
  if (t1 <= t0) return;
  float* Sg = state + ((long)state_slots[seq] * H + h) * (long)D * Dv;
  float S[R];
#pragma unroll
  for (int r = 0; r < R; ++r) {
    const int i = rg * R + r;
    S[r] = (i < D && j < Dv) ? Sg[(long)i * Dv + j] : 0.f;
  }
  float qr[EPT], kr[EPT], gr[EPT], br = 0.f;
  float vr[VPT];
  auto fetch = [&](int c0) {
#pragma unroll
    for (int m = 0; m < EPT; ++m) {
      const int x = tid + m * THREADS, c = x / DP, i = x - c * DP;
      const long t = c0 + c;
      const bool live = t < t1 && i < D;
      qr[m] = live ? qn[(t * G + gh) * D + i] : 0.f;
      kr[m] = live ? kn[(t * G + gh) * D + i] : 0.f;
      gr[m] = live ? g[(t * H + h) * D + i] : 0.f;
    }
#pragma unroll
    for (int m = 0; m < VPT; ++m) {
      const int x = tid + m * THREADS, c = x / VT, jj = blockIdx.x * VT + x % VT;
      const long t = c0 + c;
      vr[m] = (x < DS_CT * VT && t < t1 && jj < Dv) ? to_f32(vc[(t * H + h) * Dv + jj]) : 0.f;
    }
    if (tid < DS_CT) br = c0 + tid < t1 ? beta[(long)(c0 + tid) * H + h] : 0.f;
  };
  auto stage = [&](int buf) {
#pragma unroll
    for (int m = 0; m < EPT; ++m) {
      const int x = tid + m * THREADS;
      qs[buf * DS_CT * DP + x] = qr[m];
      ks[buf * DS_CT * DP + x] = kr[m];
      gs[buf * DS_CT * DP + x] = gr[m];
    }
#pragma unroll
    for (int m = 0; m < VPT; ++m) {
      const int x = tid + m * THREADS;
      if (x < DS_CT * VT) vs[buf * DS_CT * VT + x] = vr[m];
    }
    if (tid < DS_CT) bs[buf * DS_CT + tid] = br;
  };
  fetch(t0);
  stage(0);
  __syncthreads();
  int buf = 0;
  for (int c0 = t0; c0 < t1; c0 += DS_CT, buf ^= 1) {
    const int n = min(DS_CT, t1 - c0);
    const bool more = c0 + DS_CT < t1;
    if (more) fetch(c0 + DS_CT);
    for (int c = 0; c < n; ++c) {
      const float* qc = qs + (buf * DS_CT + c) * DP + rg * R;
      const float* kc = ks + (buf * DS_CT + c) * DP + rg * R;
      const float* gc = gs + (buf * DS_CT + c) * DP + rg * R;
      float sk = 0.f, sq = 0.f, kq = 0.f, kk[R];
#pragma unroll
      for (int r = 0; r < R; r += 4) {
        const float4 a = *reinterpret_cast<const float4*>(gc + r);
        const float4 k4 = *reinterpret_cast<const float4*>(kc + r);
        const float4 q4 = *reinterpret_cast<const float4*>(qc + r);
        kk[r] = k4.x; kk[r + 1] = k4.y; kk[r + 2] = k4.z; kk[r + 3] = k4.w;
        S[r] *= a.x; S[r + 1] *= a.y; S[r + 2] *= a.z; S[r + 3] *= a.w;
        sk = fmaf(S[r], k4.x, sk); sq = fmaf(S[r], q4.x, sq); kq = fmaf(k4.x, q4.x, kq);
        sk = fmaf(S[r + 1], k4.y, sk); sq = fmaf(S[r + 1], q4.y, sq); kq = fmaf(k4.y, q4.y, kq);
        sk = fmaf(S[r + 2], k4.z, sk); sq = fmaf(S[r + 2], q4.z, sq); kq = fmaf(k4.z, q4.z, kq);
        sk = fmaf(S[r + 3], k4.w, sk); sq = fmaf(S[r + 3], q4.w, sq); kq = fmaf(k4.w, q4.w, kq);
      }
#pragma unroll
      for (int o = 1; o < RG; o <<= 1) {
        sk += __shfl_xor_sync(0xffffffffu, sk, o);
        sq += __shfl_xor_sync(0xffffffffu, sq, o);
        kq += __shfl_xor_sync(0xffffffffu, kq, o);
      }
      const float u = bs[buf * DS_CT + c] * (vs[(buf * DS_CT + c) * VT + col] - sk);
#pragma unroll
      for (int r = 0; r < R; ++r) S[r] = fmaf(kk[r], u, S[r]);
      if (rg == 0 && j < Dv) out[((long)(c0 + c) * H + h) * Dv + j] = fmaf(u, kq, sq);
    }
    if (more) stage(buf ^ 1);
    __syncthreads();
  }
#pragma unroll
  for (int r = 0; r < R; ++r) {
    const int i = rg * R + r;
    if (i < D && j < Dv) Sg[(long)i * Dv + j] = S[r];
  }
}

template <typename T, int RG, int R, int VT>
static cudaError_t launch_delta_scan(cudaStream_t stream, int num_seqs, const float* qn, const float* kn, const void* vc,
                                     const float* g, const float* beta, float* state, const int* cu_seqlens,
                                     const int* state_slots, float* out, int G, int H, int D, int Dv) {
  constexpr size_t smem = (size_t)(6 * DS_CT * RG * R + 2 * DS_CT * VT + 2 * DS_CT) * sizeof(float);
  auto kernel = delta_scan_kernel<T, RG, R, VT>;
  if (smem > 48 * 1024) cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  return launch_pdl(kernel, dim3((Dv + VT - 1) / VT, H, num_seqs), dim3(RG * VT), smem, stream, qn, kn, (const T*)vc, g,
                    beta, state, cu_seqlens, state_slots, out, G, H, D, Dv);
}

// qn, kn, vc, g, beta: delta_prepare's rows; state fp32 [slots, H, D, Dv]; out fp32 [T, H, Dv].
Q3_EXPORT int q3_delta_scan(int dtype, const float* qn, const float* kn, const void* vc, const float* g,
                            const float* beta, float* state, const int* cu_seqlens, const int* state_slots, float* out,
                            int num_seqs, int G, int H, int D, int Dv, cudaStream_t stream) {
  if (!qn || !kn || !vc || !g || !beta || !state || !cu_seqlens || !state_slots || !out) return Q3_ERR_ARGUMENT;
  if (G < 1 || H < 1 || H % G || D < 1 || Dv < 1 || H > 65535 || num_seqs > 65535) return Q3_ERR_ARGUMENT;
  if (D > 256 || (dtype != Q3_DTYPE_F32 && dtype != Q3_DTYPE_BF16)) return Q3_ERR_UNSUPPORTED;
  if (num_seqs == 0) return Q3_OK;
  cudaError_t e;
#define Q3_DELTA_SCAN(T, RG, R, VT)                                                                                  \
  e = launch_delta_scan<T, RG, R, VT>(stream, num_seqs, qn, kn, vc, g, beta, state, cu_seqlens, state_slots, out, G, H, \
                                      D, Dv)
#define Q3_DELTA_SIZES(T)                                                                                            \
  if (D <= 16) Q3_DELTA_SCAN(T, 4, 4, 16); else if (D <= 32) Q3_DELTA_SCAN(T, 8, 4, 16);                              \
  else if (D <= 64) Q3_DELTA_SCAN(T, 8, 8, 16); else if (D <= 128) Q3_DELTA_SCAN(T, 16, 8, 16);                       \
  else Q3_DELTA_SCAN(T, 32, 8, 16)
  if (dtype == Q3_DTYPE_F32) { Q3_DELTA_SIZES(float); } else { Q3_DELTA_SIZES(bf16); }
#undef Q3_DELTA_SIZES
#undef Q3_DELTA_SCAN
  return e == cudaSuccess ? Q3_OK : Q3_ERR_LAUNCH;
}

// ---- the recurrence in chunks of 16 tokens ------------------------------------------------------------
// With G_i the product of a chunk's decays up to token i and S the state before the chunk, the recurrence is, in
// matrices whose rows are the chunk's tokens (the WY form of a product of rank-one updates):
//   A_ij = sum_d k_i k_j prod_(j < m <= i) g_m  (j < i)        B_ij = sum_d q_i k_j prod_(j < m <= i) g_m  (j <= i)
//   W = (I + diag(beta) A)^(-1) diag(beta)
//   U = W (V - (G k) S)      O = (G q) S + B U      S <- G_last S + sum_j (prod_(m > j) g_m k_j) u_j^T
// Only products of decays occur, never quotients, so strong decays lose nothing.  All of it is fp32 FMA.
//
// delta_chunk_rows: everything that does not depend on the state, a record of DC_REC floats per (chunk, head):
// [DP][32] (G k | G q, transposed), [16][DP] the decayed-to-the-end keys, [DP] G_last, W and B [16][16].  Chunks of
// sequence b start at place cu_seqlens[b] / 16 + b; tokens beyond a portion's end are k = q = 0, g = 1, beta = 0.
// delta_chunk_scan: one block per (16 value columns, head, sequence); the state's columns stay in registers (and, for
// the products with it, in shared memory), the next chunk's record is on its way while one is worked on.
#define DC_C 16
#define DC_REC(DP) ((DP) * 49 + 2 * DC_C * DC_C)

template <int DP>
__global__ void __launch_bounds__(256)
delta_chunk_rows_kernel(const float* __restrict__ qn, const float* __restrict__ kn, const float* __restrict__ g,
                        const float* __restrict__ beta, const int* __restrict__ cu_seqlens, int num_seqs,
                        float* __restrict__ records, int G, int H, int D) {
  __shared__ __align__(16) float ks[DC_C][DP], qs[DC_C][DP], gs[DC_C][DP];
  __shared__ float as[DC_C][DC_C + 1], bs[DC_C][DC_C + 1], be[DC_C];
  __shared__ int s_t0, s_n;
  pdl_wait();
  pdl_launch_dependents();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int place = blockIdx.x, h = blockIdx.y, gh = h / (H / G);
  if (tid == 0) {
    int n = 0, t0 = 0;
    for (int b = 0; b < num_seqs; ++b) {
      const int c0 = cu_seqlens[b], c1 = cu_seqlens[b + 1], base = c0 / DC_C + b;
      if (place >= base && place < c1 / DC_C + b + 1) {
        t0 = c0 + (place - base) * DC_C;
        n = c1 - t0;
        break;
      }
    }
    s_t0 = t0;
    s_n = n > DC_C ? DC_C : n;
  }
  __syncthreads();
  const int n = s_n;
  const long t0 = s_t0;
  if (n <= 0) return;
  for (int x = tid; x < DC_C * DP; x += 256) {
    const int c = x / DP, i = x - c * DP;
    const bool live = c < n && i < D;
    ks[c][i] = live ? kn[((t0 + c) * G + gh) * D + i] : 0.f;
    qs[c][i] = live ? qn[((t0 + c) * G + gh) * D + i] : 0.f;
    gs[c][i] = live ? g[((t0 + c) * H + h) * D + i] : 1.f;
  }
  if (tid < DC_C) be[tid] = tid < n ? beta[(t0 + tid) * H + h] : 0.f;
  __syncthreads();
  float* rec = records + ((long)place * H + h) * DC_REC(DP);
  if (tid < DP) {  // the keys and queries decayed from the chunk's start, a channel's 32 values side by side
    float* dst = rec + tid * 32;
    float run = 1.f;
#pragma unroll
    for (int c = 0; c < DC_C; c += 4) {
      float a[4], b[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        run *= gs[c + e][tid];
        a[e] = run * ks[c + e][tid];
        b[e] = run * qs[c + e][tid];
      }
      *reinterpret_cast<float4*>(dst + c) = make_float4(a[0], a[1], a[2], a[3]);
      *reinterpret_cast<float4*>(dst + DC_C + c) = make_float4(b[0], b[1], b[2], b[3]);
    }
    rec[48 * DP + tid] = run;
  } else if (tid < 2 * DP) {  // the keys decayed to the chunk's end
    const int i = tid - DP;
    float run = 1.f;
#pragma unroll
    for (int c = DC_C - 1; c >= 0; --c) {
      rec[32 * DP + c * DP + i] = run * ks[c][i];
      run *= gs[c][i];
    }
  }
  constexpr int E = DP / 32;
#pragma unroll
  for (int half = 0; half < 2; ++half) {  // rows i and 15 - i: every warp the same work
    const int i = half ? DC_C - 1 - warp : warp;
    float wk[E], wq[E];
#pragma unroll
    for (int e = 0; e < E; ++e) {
      wk[e] = ks[i][lane + 32 * e];
      wq[e] = qs[i][lane + 32 * e];
    }
    for (int j = i; j >= 0; --j) {
      float a = 0.f, b = 0.f;
#pragma unroll
      for (int e = 0; e < E; ++e) {
        const float kj = ks[j][lane + 32 * e];
        a = fmaf(wk[e], kj, a);
        b = fmaf(wq[e], kj, b);
        const float gj = gs[j][lane + 32 * e];
        wk[e] *= gj;
        wq[e] *= gj;
      }
      a = warp_sum(a);
      b = warp_sum(b);
      if (lane == 0) {
        as[i][j] = a;  // (the diagonal is not used)
        bs[i][j] = b;
      }
    }
  }
  __syncthreads();
  if (tid < DC_C) {  // column tid of W by forward substitution
    float x[DC_C];
#pragma unroll
    for (int i = 0; i < DC_C; ++i) {
      float acc = i == tid ? 1.f : 0.f;
#pragma unroll
      for (int j = 0; j < i; ++j) acc = fmaf(-as[i][j], x[j], acc);
      x[i] = be[i] * acc;
      rec[49 * DP + i * DC_C + tid] = x[i];
    }
  } else if (tid >= 64 && tid < 64 + DC_C * 4) {
    const int i = (tid - 64) >> 2, j0 = ((tid - 64) & 3) * 4;
#pragma unroll
    for (int e = 0; e < 4; ++e) rec[49 * DP + DC_C * DC_C + i * DC_C + j0 + e] = j0 + e <= i ? bs[i][j0 + e] : 0.f;
  }
}

__device__ __forceinline__ void ds_copy16(float* dst, const float* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src));
}

template <typename T, int DP>
__global__ void __launch_bounds__(256)
delta_chunk_scan_kernel(const float* __restrict__ records, const T* __restrict__ vc, float* __restrict__ state,
                        const int* __restrict__ cu_seqlens, const int* __restrict__ state_slots, float* __restrict__ out,
                        int H, int D, int Dv) {
  constexpr int VT = 16, REC = DC_REC(DP), RD = DP / 64, PS = 20;  // PS: row pitch of the partial sums
  extern __shared__ __align__(16) float dc_smem[];
  float* Ss = dc_smem + 2 * REC;       // [DP][VT]
  float* part = Ss + DP * VT;          // [8][32][PS]
  float* ys = part + 8 * 32 * PS;      // [16][VT]
  float* us = ys + DC_C * VT;          // [16][VT]
  pdl_wait();
  pdl_launch_dependents();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int h = blockIdx.y, b = blockIdx.z, col0 = blockIdx.x * VT;
  const int t0 = cu_seqlens[b], t1 = cu_seqlens[b + 1];
  if (t1 <= t0) return;
  const int chunks = (t1 - t0 + DC_C - 1) / DC_C;
  const float* rec0 = records + ((long)(t0 / DC_C + b) * H + h) * REC;
  auto load = [&](int c) {
    const float* src = rec0 + (long)c * H * REC;
    float* dst = dc_smem + (c & 1) * REC;
    for (int x = tid * 4; x < REC; x += 1024) ds_copy16(dst + x, src + x);
    asm volatile("cp.async.commit_group;\n" ::);
  };
  load(0);
  // this thread's rows and columns of the state
  const int d0 = (tid >> 2) * RD, c0 = (tid & 3) * 4;
  float* Sg = state + ((long)state_slots[b] * H + h) * (long)D * Dv;
  float S[RD][4];
#pragma unroll
  for (int r = 0; r < RD; ++r) {
#pragma unroll
    for (int e = 0; e < 4; ++e)
      S[r][e] = d0 + r < D && col0 + c0 + e < Dv ? Sg[(long)(d0 + r) * Dv + col0 + c0 + e] : 0.f;
    *reinterpret_cast<float4*>(Ss + (d0 + r) * VT + c0) = make_float4(S[r][0], S[r][1], S[r][2], S[r][3]);
  }
  const int row = tid >> 4, col = tid & 15;  // the chunk's token and the value column of the small products
  const bool col_in = col0 + col < Dv;
  auto value = [&](int c) {
    const long t = t0 + c * DC_C + row;
    return col_in && t < t1 ? to_f32(vc[(t * H + h) * Dv + col0 + col]) : 0.f;
  };
  float v_next = value(0);
  const int rt = (lane >> 2) * 4, ct = (lane & 3) * 4;
  for (int c = 0; c < chunks; ++c) {
    asm volatile("cp.async.wait_group 0;\n" ::);
    __syncthreads();  // the record and the state in shared memory are complete; nobody reads the other record
    const float* rec = dc_smem + (c & 1) * REC;
    const float v = v_next;
    if (c + 1 < chunks) {
      load(c + 1);
      v_next = value(c + 1);
    }
    {  // [G k; G q] S, an eighth of the channels a warp, 4 x 4 sums a thread
      float acc[4][4];
#pragma unroll
      for (int i = 0; i < 4; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
#pragma unroll
      for (int dd = 0; dd < DP / 8; ++dd) {
        const int d = warp * (DP / 8) + dd;
        const float4 a = *reinterpret_cast<const float4*>(rec + d * 32 + rt);
        const float4 s = *reinterpret_cast<const float4*>(Ss + d * VT + ct);
        const float av[4] = {a.x, a.y, a.z, a.w};
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          acc[i][0] = fmaf(av[i], s.x, acc[i][0]);
          acc[i][1] = fmaf(av[i], s.y, acc[i][1]);
          acc[i][2] = fmaf(av[i], s.z, acc[i][2]);
          acc[i][3] = fmaf(av[i], s.w, acc[i][3]);
        }
      }
#pragma unroll
      for (int i = 0; i < 4; ++i)
        *reinterpret_cast<float4*>(part + (warp * 32 + rt + i) * PS + ct) =
            make_float4(acc[i][0], acc[i][1], acc[i][2], acc[i][3]);
    }
    __syncthreads();
    float pk = 0.f, o = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) {
      pk += part[(w * 32 + row) * PS + col];
      o += part[(w * 32 + 16 + row) * PS + col];
    }
    ys[row * VT + col] = v - pk;
    __syncthreads();
    {
      const float* W = rec + 49 * DP + row * DC_C;
      float u = 0.f;
#pragma unroll
      for (int j = 0; j < DC_C; j += 4) {  // (W is zero beyond the diagonal)
        const float4 w4 = *reinterpret_cast<const float4*>(W + j);
        u = fmaf(w4.x, ys[j * VT + col], u);
        u = fmaf(w4.y, ys[(j + 1) * VT + col], u);
        u = fmaf(w4.z, ys[(j + 2) * VT + col], u);
        u = fmaf(w4.w, ys[(j + 3) * VT + col], u);
      }
      us[row * VT + col] = u;
    }
    __syncthreads();
    {
      const float* B = rec + 49 * DP + DC_C * DC_C + row * DC_C;
#pragma unroll
      for (int j = 0; j < DC_C; j += 4) {
        const float4 b4 = *reinterpret_cast<const float4*>(B + j);
        o = fmaf(b4.x, us[j * VT + col], o);
        o = fmaf(b4.y, us[(j + 1) * VT + col], o);
        o = fmaf(b4.z, us[(j + 2) * VT + col], o);
        o = fmaf(b4.w, us[(j + 3) * VT + col], o);
      }
      const long t = t0 + c * DC_C + row;
      if (col_in && t < t1) out[(t * H + h) * Dv + col0 + col] = o;
    }
    const float* kend = rec + 32 * DP;
#pragma unroll
    for (int r = 0; r < RD; ++r) {
      const float gl = rec[48 * DP + d0 + r];
#pragma unroll
      for (int e = 0; e < 4; ++e) S[r][e] *= gl;
    }
#pragma unroll
    for (int j = 0; j < DC_C; ++j) {
      const float4 u4 = *reinterpret_cast<const float4*>(us + j * VT + c0);
#pragma unroll
      for (int r = 0; r < RD; ++r) {
        const float kk = kend[j * DP + d0 + r];
        S[r][0] = fmaf(kk, u4.x, S[r][0]);
        S[r][1] = fmaf(kk, u4.y, S[r][1]);
        S[r][2] = fmaf(kk, u4.z, S[r][2]);
        S[r][3] = fmaf(kk, u4.w, S[r][3]);
      }
    }
#pragma unroll
    for (int r = 0; r < RD; ++r)
      *reinterpret_cast<float4*>(Ss + (d0 + r) * VT + c0) = make_float4(S[r][0], S[r][1], S[r][2], S[r][3]);
  }
#pragma unroll
  for (int r = 0; r < RD; ++r)
#pragma unroll
    for (int e = 0; e < 4; ++e)
      if (d0 + r < D && col0 + c0 + e < Dv) Sg[(long)(d0 + r) * Dv + col0 + c0 + e] = S[r][e];
}

template <typename T, int DP>
static int launch_delta_chunks(cudaStream_t stream, int num_tokens, int num_seqs, const float* qn, const float* kn,
                               const void* vc, const float* g, const float* beta, float* records, float* state,
                               const int* cu_seqlens, const int* state_slots, float* out, int G, int H, int D, int Dv) {
  const int places = num_tokens / DC_C + num_seqs;
  if (launch_pdl(delta_chunk_rows_kernel<DP>, dim3(places, H), dim3(256), 0, stream, qn, kn, g, beta, cu_seqlens, num_seqs,
                 records, G, H, D) != cudaSuccess)
    return Q3_ERR_LAUNCH;
  constexpr size_t smem = sizeof(float) * (2 * DC_REC(DP) + DP * 16 + 8 * 32 * 20 + 2 * DC_C * 16);
  auto kernel = delta_chunk_scan_kernel<T, DP>;
  static bool configured_on[Q3_MAX_DEVICES];
  bool& configured = configured_on[q3_current_device()];
  if (!configured) {
    if (cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
      return Q3_ERR_LAUNCH;
    configured = true;
  }
  return launch_pdl(kernel, dim3((Dv + 15) / 16, H, num_seqs), dim3(256), smem, stream, (const float*)records, (const T*)vc,
                    state, cu_seqlens, state_slots, out, H, D, Dv) == cudaSuccess
             ? Q3_OK
             : Q3_ERR_LAUNCH;
}

// The same as q3_delta_scan for key sizes up to 128, in chunks; records: (num_tokens / 16 + num_seqs) * H * (49 * DP +
// 512) floats with DP = 64 (D <= 64) or 128.
Q3_EXPORT int q3_delta_chunk_scan(int dtype, const float* qn, const float* kn, const void* vc, const float* g,
                                  const float* beta, float* records, float* state, const int* cu_seqlens,
                                  const int* state_slots, float* out, int num_tokens, int num_seqs, int G, int H, int D,
                                  int Dv, cudaStream_t stream) {
  if (!qn || !kn || !vc || !g || !beta || !records || !state || !cu_seqlens || !state_slots || !out) return Q3_ERR_ARGUMENT;
  if (G < 1 || H < 1 || H % G || D < 1 || Dv < 1 || H > 65535 || num_seqs > 65535) return Q3_ERR_ARGUMENT;
  if (D > 128 || (dtype != Q3_DTYPE_F32 && dtype != Q3_DTYPE_BF16) || !ds_aligned(records)) return Q3_ERR_UNSUPPORTED;
  if (num_seqs == 0 || num_tokens == 0) return Q3_OK;
#define Q3_DELTA_CHUNKS(T, DP)                                                                                       \
  return launch_delta_chunks<T, DP>(stream, num_tokens, num_seqs, qn, kn, vc, g, beta, records, state, cu_seqlens,   \
                                    state_slots, out, G, H, D, Dv)
  if (dtype == Q3_DTYPE_F32) {
    if (D <= 64) Q3_DELTA_CHUNKS(float, 64);
    Q3_DELTA_CHUNKS(float, 128);
  }
  if (D <= 64) Q3_DELTA_CHUNKS(bf16, 64);
  Q3_DELTA_CHUNKS(bf16, 128);
#undef Q3_DELTA_CHUNKS
}

// ---- steps in which every sequence brings one token, in one kernel ------------------------------------
// One block per (head, sequence).  The head's state is fetched into registers before the projection it waits for is
// finished; then the block convolves its q, k and v channels (and writes the token's inputs into the ring), makes the
// decays and the output gate from the low-rank products' first halves, updates the state, norms and gates the head's
// output.  A thread holds up to 32 key rows of one value column; the NT / DVP row groups of a column meet in shared
// memory.  DVP: the value size rounded up to a power of two (32 at least).
template <typename T>
__global__ void __launch_bounds__(512)
delta_step_kernel(const T* __restrict__ x, long x_stride, const float* __restrict__ w, int taps, float* ring,
                  const int* __restrict__ positions, const int* __restrict__ cu_seqlens,
                  const int* __restrict__ state_slots, const T* __restrict__ low_a, const T* __restrict__ low_g,
                  const T* __restrict__ a2, int a_rank, const T* __restrict__ g2, int g_rank,
                  const float* __restrict__ dt_bias, const float* __restrict__ neg_a, const T* __restrict__ b,
                  float q_scale, float* state, const float* __restrict__ norm_w, float eps, T* __restrict__ out,
                  long out_stride, int G, int H, int D, int Dv, int dvp_shift) {
  extern __shared__ __align__(16) float st_smem[];
  const int NT = blockDim.x, tid = threadIdx.x, DVP = 1 << dvp_shift, RG = NT >> dvp_shift;
  const int RP = (((D + RG - 1) / RG) + 3) & ~3;  // rows of a thread: at most 32
  const int DP = (RP * RG + 3) & ~3;
  float* qs = st_smem;              // [DP] q, then k, then decays; zero beyond D
  float* ks = qs + DP;
  float* gs = ks + DP;
  float* vs = gs + DP;              // [Dv] values, then gates
  float* gate = vs + ((Dv + 3) & ~3);
  float* la = gate + ((Dv + 3) & ~3);  // low-rank rows
  float* lg = la + ((a_rank + 3) & ~3);
  float* part = lg + ((g_rank + 3) & ~3);  // [2][RG][DVP]
  __shared__ float red[33], sums[3];
  const int h = blockIdx.x, seq = blockIdx.y, rep = H / G, gh = h / rep;
  const int j = tid & (DVP - 1), rg = tid >> dvp_shift, i0 = rg * RP;
  const int slot = state_slots[seq];
  float* Sg = state + ((long)slot * H + h) * (long)D * Dv;
  float S[32];
#pragma unroll
  for (int r = 0; r < 32; ++r) S[r] = (r < RP && i0 + r < D && j < Dv) ? Sg[(long)(i0 + r) * Dv + j] : 0.f;
  pdl_wait();
  pdl_launch_dependents();
  const int t = cu_seqlens[seq], p = positions[t];
  const T* xrow = x + (long)t * x_stride;
  const int C = 2 * G * D + H * Dv;
  float* rows = taps > 1 ? ring + (long)slot * taps * C : nullptr;
  for (int c = tid; c < a_rank; c += NT) la[c] = to_f32(low_a[(long)t * x_stride + c]);
  for (int c = tid; c < g_rank; c += NT) lg[c] = to_f32(low_g[(long)t * x_stride + c]);
  for (int c = tid; c < 2 * D + Dv; c += NT) {
    const int ch = c < D ? gh * D + c : (c < 2 * D ? G * D + gh * D + c - D : 2 * G * D + h * Dv + c - 2 * D);
    float y[1];
    conv_silu<T, 1>(xrow, x_stride, w, taps, rows, C, 0, p, ch, y);
    (c < D ? qs[c] : (c < 2 * D ? ks[c - D] : vs[c - 2 * D])) = y[0];
    if (rows && (c >= 2 * D || h == gh * rep)) rows[(long)(p % taps) * C + ch] = to_f32(xrow[ch]);
  }
  for (int i = D + tid; i < DP; i += NT) qs[i] = ks[i] = gs[i] = 0.f;
  __syncthreads();
  // decays (outputs 0 .. D - 1) and gates (D ..): four lanes an output
  {
    const int lane4 = tid & 3;
    for (int o0 = 0; o0 < D + Dv; o0 += NT >> 2) {
      const int o = o0 + (tid >> 2);
      const bool live = o < D + Dv, is_a = o < D;
      const int rank = is_a ? a_rank : g_rank;
      const T* wr = live ? (is_a ? a2 + ((long)h * D + o) * a_rank : g2 + ((long)h * Dv + o - D) * g_rank) : a2;
      const float* lo = is_a ? la : lg;
      float acc = 0.f;
      if (live) {
        if ((rank & 7) == 0) {
          for (int r = lane4 * 8; r < rank; r += 32) {
            float v8[8];
            load8(wr + r, v8);
#pragma unroll
            for (int e = 0; e < 8; ++e) acc = fmaf(v8[e], lo[r + e], acc);
          }
        } else {
          for (int r = lane4; r < rank; r += 4) acc = fmaf(to_f32(wr[r]), lo[r], acc);
        }
      }
      acc += __shfl_xor_sync(0xffffffffu, acc, 1);
      acc += __shfl_xor_sync(0xffffffffu, acc, 2);
      if (live && lane4 == 0) {
        if (is_a) gs[o] = expf(neg_a[h] * softplus_f(acc + dt_bias[h * D + o]));
        else gate[o - D] = sigmoid_f(acc);
      }
    }
  }
  if (tid < 96) {  // |q|^2, |k|^2 and k . q, a warp each
    const float* p1 = tid < 32 ? qs : ks;
    const float* p2 = tid < 32 || tid >= 64 ? qs : ks;
    float acc = 0.f;
    for (int i = tid & 31; i < D; i += 32) acc = fmaf(p1[i], p2[i], acc);
    acc = warp_sum(acc);
    if ((tid & 31) == 0) sums[tid >> 5] = acc;
  }
  __syncthreads();
  const float inv_q = rsqrtf(sums[0] + UNIT_EPS) * q_scale, inv_k = rsqrtf(sums[1] + UNIT_EPS);
  const float kq = sums[2] * inv_q * inv_k;
  float sk = 0.f, sq = 0.f;
#pragma unroll
  for (int r = 0; r < 32; r += 4) {
    if (r < RP) {
      const float4 a = *reinterpret_cast<const float4*>(gs + i0 + r);
      const float4 k4 = *reinterpret_cast<const float4*>(ks + i0 + r);
      const float4 q4 = *reinterpret_cast<const float4*>(qs + i0 + r);
      S[r] *= a.x; S[r + 1] *= a.y; S[r + 2] *= a.z; S[r + 3] *= a.w;
      sk = fmaf(S[r], k4.x, sk); sq = fmaf(S[r], q4.x, sq);
      sk = fmaf(S[r + 1], k4.y, sk); sq = fmaf(S[r + 1], q4.y, sq);
      sk = fmaf(S[r + 2], k4.z, sk); sq = fmaf(S[r + 2], q4.z, sq);
      sk = fmaf(S[r + 3], k4.w, sk); sq = fmaf(S[r + 3], q4.w, sq);
    }
  }
  part[rg * DVP + j] = sk;
  part[(RG + rg) * DVP + j] = sq;
  __syncthreads();
  sk = sq = 0.f;
  for (int r = 0; r < RG; ++r) sk += part[r * DVP + j];
  const float beta = sigmoid_f(to_f32(b[(long)t * x_stride + h]));
  const float u = j < Dv ? beta * (vs[j] - sk * inv_k) : 0.f;
  const float uk = u * inv_k;
#pragma unroll
  for (int r = 0; r < 32; ++r)
    if (r < RP && i0 + r < D && j < Dv) Sg[(long)(i0 + r) * Dv + j] = fmaf(ks[i0 + r], uk, S[r]);
  float o = 0.f;
  if (rg == 0 && j < Dv) {
    for (int r = 0; r < RG; ++r) sq += part[(RG + r) * DVP + j];
    o = fmaf(u, kq, sq * inv_q);
  }
  const float rstd = rsqrtf(block_sum(o * o, red) / (float)Dv + eps);
  if (rg == 0 && j < Dv) out[(long)t * out_stride + (long)h * Dv + j] = from_f32<T>((o * rstd) * norm_w[j] * gate[j]);
}

// x, low_a, low_g and b are columns of one product: rows x_stride apart.  ring fp32 [slots, taps, C] (or null with one
// tap); a2 [H * D, a_rank], g2 [H * Dv, g_rank] of the activation type; norm_w fp32 [Dv]; out rows out_stride apart,
// head h at column h * Dv.  Value sizes up to 256 with D * (Dv rounded up to a power of two) at most 16384.
Q3_EXPORT int q3_delta_step(int dtype, const void* x, long x_stride, const float* w, int taps, float* ring,
                            const int* positions, const int* cu_seqlens, const int* state_slots, const void* low_a,
                            const void* low_g, const void* a2, int a_rank, const void* g2, int g_rank,
                            const float* dt_bias, const float* neg_a, const void* b, float q_scale, float* state,
                            const float* norm_w, float eps, void* out, long out_stride, int num_seqs, int G, int H, int D,
                            int Dv, cudaStream_t stream) {
  if (!x || !w || !positions || !cu_seqlens || !state_slots || !low_a || !low_g || !a2 || !g2 || !dt_bias || !neg_a || !b ||
      !state || !norm_w || !out)
    return Q3_ERR_ARGUMENT;
  if (G < 1 || H < 1 || H % G || D < 1 || Dv < 1 || taps < 1 || (taps > 1 && !ring) || a_rank < 1 || g_rank < 1)
    return Q3_ERR_ARGUMENT;
  int shift = 5;
  while ((1 << shift) < Dv) ++shift;
  const int DVP = 1 << shift;
  if (D > 256 || DVP > 256 || D * DVP > 16384 || taps > DELTA_MAX_TAPS || num_seqs > 65535) return Q3_ERR_UNSUPPORTED;
  if (((a_rank & 7) == 0 && !ds_aligned(a2)) || ((g_rank & 7) == 0 && !ds_aligned(g2))) return Q3_ERR_UNSUPPORTED;
  if (num_seqs == 0) return Q3_OK;
  int NT = 128;
  while (NT < 512 && (long)NT * 32 < (long)D * DVP) NT <<= 1;
  if (NT < DVP) NT = DVP;
  const int RG = NT / DVP, RP = (((D + RG - 1) / RG) + 3) & ~3;
  if (RP > 32) return Q3_ERR_UNSUPPORTED;
  const size_t smem = sizeof(float) * (size_t)(3 * ((RP * RG + 3) & ~3) + 2 * ((Dv + 3) & ~3) + ((a_rank + 3) & ~3) +
                                               ((g_rank + 3) & ~3) + 2 * RG * DVP);
  if (smem > 48 * 1024) return Q3_ERR_UNSUPPORTED;
  cudaError_t e;
#define Q3_DELTA_STEP(T)                                                                                               e = launch_pdl(delta_step_kernel<T>, dim3(H, num_seqs), dim3(NT), smem, stream, (const T*)x, x_stride, w, taps, ring,                  positions, cu_seqlens, state_slots, (const T*)low_a, (const T*)low_g, (const T*)a2, a_rank,                          (const T*)g2, g_rank, dt_bias, neg_a, (const T*)b, q_scale, state, norm_w, eps, (T*)out, out_stride, G, H,                  D, Dv, shift)
  if (dtype == Q3_DTYPE_F32) Q3_DELTA_STEP(float);
  else if (dtype == Q3_DTYPE_BF16) Q3_DELTA_STEP(bf16);
  else return Q3_ERR_ARGUMENT;
#undef Q3_DELTA_STEP
  return e == cudaSuccess ? Q3_OK : Q3_ERR_LAUNCH;
}
