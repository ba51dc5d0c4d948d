// Sums of several sublayer outputs folded into the residual stream, with an optional average over the depth,
// and the norm that reads the result; everything in fp32, one rounding at the store.
//
//   v = resid[r] + sum_k y_k         y_k = x_k, or (x_k * rsqrt(mean(x_k^2) + eps_k)) * w_k   (an output norm)
//         x_k: rows of the output's type, or fp32 planes (partial sums of a product, added in order)
//   without depth weights:   s = v
//   with depth weights:      points[n][r] = v,  s = sum_(j < n) dw[j] * points[j][r] + dw[n] * v
//   resid_out[r] = s         out[i] = (s * rsqrt(mean(s^2) + eps)) * w     (no w: out = s, rounded)
//
// `points` holds the stream's values between the layers, [*, rows, H]: the embedding output and every layer's
// result before its average.  `rows` picks the source rows (the final norm on the rows whose logits are wanted;
// nothing is written back then).  One block per row; every reduction is a fixed tree over the row, so a row's
// bits do not depend on the rows around it.
//
// embed_norm: out[r] = (t * rsqrt(mean(t^2) + eps)) * w with t = table[ids[r]], as fp32 rows.
#include "common.cuh"

#define SN_MAX 4  // outputs folded at a time

struct SumItems {
  const void* x[SN_MAX];
  const float* w[SN_MAX];   // output norm, or null
  long plane[SN_MAX];       // distance of an fp32 item's planes
  int parts[SN_MAX];        // 0: rows of the output's type; else fp32 planes
  float eps[SN_MAX];
  int count;
};

// eight consecutive values of item k at column i of source row `src`
template <typename T>
__device__ __forceinline__ void item8(const SumItems& it, int k, long src, int H, int i, float (&v)[8]) {
  if (it.parts[k] == 0) {
    load8(static_cast<const T*>(it.x[k]) + src * H + i, v);
    return;
  }
  const float* p = static_cast<const float*>(it.x[k]) + src * H + i;
  load8(p, v);
  for (int q = 1; q < it.parts[k]; q += 2) {  // two planes' loads in flight; added in order
    float a[8], b[8];
    const bool two = q + 1 < it.parts[k];
    load8(p + q * it.plane[k], a);
    if (two) load8(p + (q + 1) * it.plane[k], b);
#pragma unroll
    for (int e = 0; e < 8; ++e) v[e] += a[e];
    if (two) {
#pragma unroll
      for (int e = 0; e < 8; ++e) v[e] += b[e];
    }
  }
}

template <typename T>
__device__ __forceinline__ float item1(const SumItems& it, int k, long src, int H, int i) {
  if (it.parts[k] == 0) return to_f32(static_cast<const T*>(it.x[k])[src * H + i]);
  const float* p = static_cast<const float*>(it.x[k]) + src * H + i;
  float v = p[0];
  for (int q = 1; q < it.parts[k]; ++q) v += p[q * it.plane[k]];
  return v;
}

// sums of `n` values per thread over the block, all at once; red: 32 * SN_MAX floats
__device__ __forceinline__ void block_sums(float (&v)[SN_MAX], int n, float* red) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarp = blockDim.x >> 5;
#pragma unroll
  for (int k = 0; k < SN_MAX; ++k)
    if (k < n) v[k] = warp_sum(v[k]);
  __syncthreads();
  if (lane == 0) {
#pragma unroll
    for (int k = 0; k < SN_MAX; ++k)
      if (k < n) red[k * 32 + warp] = v[k];
  }
  __syncthreads();
#pragma unroll
  for (int k = 0; k < SN_MAX; ++k)
    if (k < n) v[k] = warp_sum(lane < nwarp ? red[k * 32 + lane] : 0.f);
}

// Eight values a thread, a thread for every eight values of the row (H <= 8192): items and sum stay in registers.
template <typename T>
__global__ void __launch_bounds__(1024)
sum_norm_vec_kernel(SumItems it, const float* __restrict__ resid, float* resid_out, float* points, long point_stride,
                    int num_points, const float* __restrict__ dw, const int* __restrict__ rows,
                    const float* __restrict__ w, T* __restrict__ out, int H, float eps, int write) {
  __shared__ float red[32 * SN_MAX];
  pdl_wait();
  pdl_launch_dependents();
  const int r = blockIdx.x;
  const long src = rows ? rows[r] : r;
  const int i = threadIdx.x * 8;
  const bool live = i < H;
  float x[SN_MAX][8], s[8];
  float ss[SN_MAX];
#pragma unroll
  for (int e = 0; e < 8; ++e) s[e] = 0.f;
  if (live) load8(resid + src * H + i, s);
#pragma unroll
  for (int k = 0; k < SN_MAX; ++k) {
    ss[k] = 0.f;
#pragma unroll
    for (int e = 0; e < 8; ++e) x[k][e] = 0.f;
    if (k < it.count && live) {
      item8<T>(it, k, src, H, i, x[k]);
#pragma unroll
      for (int e = 0; e < 8; ++e) ss[k] += x[k][e] * x[k][e];
    }
  }
  bool any = false;
#pragma unroll
  for (int k = 0; k < SN_MAX; ++k) any |= k < it.count && it.w[k] != nullptr;
  if (any) block_sums(ss, it.count, red);
#pragma unroll
  for (int k = 0; k < SN_MAX; ++k) {
    if (k >= it.count || !live) continue;
    if (it.w[k]) {
      const float rstd = rsqrtf(ss[k] / (float)H + it.eps[k]);
      float ww[8];
      load8(it.w[k] + i, ww);
#pragma unroll
      for (int e = 0; e < 8; ++e) s[e] += (x[k][e] * rstd) * ww[e];
    } else {
#pragma unroll
      for (int e = 0; e < 8; ++e) s[e] += x[k][e];
    }
  }
  if (dw && live) {
    if (write) store8(points + num_points * point_stride + src * H + i, s);
    const float wn = dw[num_points];
    float acc[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) acc[e] = 0.f;
    for (int j0 = 0; j0 < num_points; j0 += 4) {  // four points' loads in flight at a time; added in order
      float p[4][8];
#pragma unroll
      for (int u = 0; u < 4; ++u)
        if (j0 + u < num_points) load8(points + (j0 + u) * point_stride + src * H + i, p[u]);
#pragma unroll
      for (int u = 0; u < 4; ++u)
        if (j0 + u < num_points) {
          const float wj = dw[j0 + u];
#pragma unroll
          for (int e = 0; e < 8; ++e) acc[e] = fmaf(wj, p[u][e], acc[e]);
        }
    }
#pragma unroll
    for (int e = 0; e < 8; ++e) s[e] = fmaf(wn, s[e], acc[e]);
  }
  if (write && live) store8(resid_out + src * H + i, s);
  if (!w) {
    if (live) store8(out + (long)r * H + i, s);
    return;
  }
  float tot[SN_MAX];
  tot[0] = 0.f;
#pragma unroll
  for (int e = 0; e < 8; ++e) tot[0] += s[e] * s[e];
  block_sums(tot, 1, red);
  if (!live) return;
  const float rstd = rsqrtf(tot[0] / (float)H + eps);
  float ww[8];
  load8(w + i, ww);
#pragma unroll
  for (int e = 0; e < 8; ++e) s[e] = (s[e] * rstd) * ww[e];
  store8(out + (long)r * H + i, s);
}

// Any width: one element at a time, the row's sum in shared memory.
template <typename T>
__global__ void sum_norm_kernel(SumItems it, const float* __restrict__ resid, float* resid_out, float* points,
                                long point_stride, int num_points, const float* __restrict__ dw,
                                const int* __restrict__ rows, const float* __restrict__ w, T* __restrict__ out, int H,
                                float eps, int write) {
  extern __shared__ float sn_vals[];  // H
  __shared__ float red[32 * SN_MAX];
  pdl_wait();
  pdl_launch_dependents();
  const int r = blockIdx.x;
  const long src = rows ? rows[r] : r;
  float ss[SN_MAX];
#pragma unroll
  for (int k = 0; k < SN_MAX; ++k) {
    ss[k] = 0.f;
    if (k < it.count && it.w[k])
      for (int i = threadIdx.x; i < H; i += blockDim.x) {
        const float x = item1<T>(it, k, src, H, i);
        ss[k] += x * x;
      }
  }
  block_sums(ss, it.count, red);
  float tot[SN_MAX];
  tot[0] = 0.f;
  for (int i = threadIdx.x; i < H; i += blockDim.x) {
    float s = resid[src * H + i];
#pragma unroll
    for (int k = 0; k < SN_MAX; ++k)
      if (k < it.count) {
        const float x = item1<T>(it, k, src, H, i);
        s += it.w[k] ? (x * rsqrtf(ss[k] / (float)H + it.eps[k])) * it.w[k][i] : x;
      }
    if (dw) {
      if (write) points[num_points * point_stride + src * H + i] = s;
      float acc = 0.f;
      for (int j = 0; j < num_points; ++j) acc = fmaf(dw[j], points[j * point_stride + src * H + i], acc);
      s = fmaf(dw[num_points], s, acc);
    }
    if (write) resid_out[src * H + i] = s;
    if (!w) out[(long)r * H + i] = from_f32<T>(s);
    sn_vals[i] = s;
    tot[0] += s * s;
  }
  if (!w) return;
  block_sums(tot, 1, red);
  const float rstd = rsqrtf(tot[0] / (float)H + eps);
  for (int i = threadIdx.x; i < H; i += blockDim.x) out[(long)r * H + i] = from_f32<T>((sn_vals[i] * rstd) * w[i]);
}

static inline bool sn_aligned(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

template <typename T>
static int launch_sum_norm(const SumItems& it, const float* resid, float* resid_out, float* points, long point_stride,
                           int num_points, const float* dw, const int* rows, const float* w, void* out, int num_rows,
                           int H, float eps, int write, cudaStream_t stream) {
  bool vec = H % 8 == 0 && H <= 8192 && sn_aligned(resid) && sn_aligned(resid_out) && sn_aligned(points) &&
             point_stride % 4 == 0 && sn_aligned(w) && sn_aligned(out);
  for (int k = 0; k < it.count; ++k)
    vec = vec && sn_aligned(it.x[k]) && sn_aligned(it.w[k]) && (it.parts[k] == 0 || it.plane[k] % 4 == 0);
  cudaError_t e;
  if (vec) {
    const int threads = ((H / 8 + 31) / 32) * 32;
    e = launch_pdl(sum_norm_vec_kernel<T>, dim3(num_rows), dim3(threads), 0, stream, it, resid, resid_out, points,
                   point_stride, num_points, dw, rows, w, (T*)out, H, eps, write);
  } else {
    const size_t smem = (size_t)H * sizeof(float);
    if (smem > 200 * 1024) return Q3_ERR_UNSUPPORTED;
    if (smem > 48 * 1024)
      cudaFuncSetAttribute(sum_norm_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    const int threads = H >= 2048 ? 512 : (H >= 512 ? 256 : 128);
    e = launch_pdl(sum_norm_kernel<T>, dim3(num_rows), dim3(threads), smem, stream, it, resid, resid_out, points,
                   point_stride, num_points, dw, rows, w, (T*)out, H, eps, write);
  }
  return e == cudaSuccess ? Q3_OK : Q3_ERR_LAUNCH;
}

// x0..x3: the outputs to fold (the first `count`); parts 0: `dtype` [*, H]; parts > 0: fp32 planes plane_k elements
// apart; w_k: fp32 [H] output norm with eps_k, or null.  resid, resid_out fp32 [*, H] (may be the same rows without
// depth weights); points fp32 [num_points + 1, *, H], point_stride apart, with dw fp32 [num_points + 1], or both
// null; w fp32 [H] or null; write: store resid_out (and the new point).
Q3_EXPORT int q3_sum_norm(int dtype, int count, const void* x0, int parts0, long plane0, const float* w0, float eps0,
                          const void* x1, int parts1, long plane1, const float* w1, float eps1, const void* x2,
                          int parts2, long plane2, const float* w2, float eps2, const void* x3, int parts3, long plane3,
                          const float* w3, float eps3, const float* resid, float* resid_out, float* points,
                          long point_stride, int num_points, const float* dw, const int* rows, const float* w, void* out,
                          int num_rows, int H, float eps, int write, cudaStream_t stream) {
  if (count < 0 || count > SN_MAX || !resid || !out || H < 1 || (write && !resid_out)) return Q3_ERR_ARGUMENT;
  if (dw && (!points || num_points < 1)) return Q3_ERR_ARGUMENT;
  SumItems it = {{x0, x1, x2, x3}, {w0, w1, w2, w3}, {plane0, plane1, plane2, plane3},
                 {parts0, parts1, parts2, parts3}, {eps0, eps1, eps2, eps3}, count};
  for (int k = 0; k < count; ++k)
    if (!it.x[k] || it.parts[k] < 0) return Q3_ERR_ARGUMENT;
  if (num_rows == 0) return Q3_OK;
  if (dtype == Q3_DTYPE_F32)
    return launch_sum_norm<float>(it, resid, resid_out, points, point_stride, num_points, dw, rows, w, out, num_rows, H,
                                  eps, write, stream);
  if (dtype == Q3_DTYPE_BF16)
    return launch_sum_norm<bf16>(it, resid, resid_out, points, point_stride, num_points, dw, rows, w, out, num_rows, H,
                                 eps, write, stream);
  return Q3_ERR_ARGUMENT;
}

template <typename T, bool VEC>
__global__ void embed_norm_kernel(const int* __restrict__ ids, const T* __restrict__ table, int vocab,
                                  const float* __restrict__ w, float* __restrict__ out, int H, float eps) {
  __shared__ float red[33];
  pdl_wait();
  pdl_launch_dependents();
  int id = ids[blockIdx.x];
  id = id < 0 ? 0 : (id >= vocab ? vocab - 1 : id);
  const T* row = table + (long)id * H;
  float* dst = out + (long)blockIdx.x * H;
  constexpr int E = VEC ? 8 : 1;
  float ss = 0.f;
  for (int i = threadIdx.x * E; i < H; i += blockDim.x * E) {
    if (VEC) {
      float v[8];
      load8(row + i, v);
#pragma unroll
      for (int e = 0; e < 8; ++e) ss += v[e] * v[e];
    } else {
      const float v = to_f32(row[i]);
      ss += v * v;
    }
  }
  const float rstd = rsqrtf(block_sum(ss, red) / (float)H + eps);
  for (int i = threadIdx.x * E; i < H; i += blockDim.x * E) {
    if (VEC) {
      float v[8], ww[8];
      load8(row + i, v);
      load8(w + i, ww);
#pragma unroll
      for (int e = 0; e < 8; ++e) v[e] = (v[e] * rstd) * ww[e];
      store8(dst + i, v);
    } else {
      dst[i] = (to_f32(row[i]) * rstd) * w[i];
    }
  }
}

// ids int32 [num_rows]; table `dtype` [vocab, H]; w fp32 [H]; out fp32 [num_rows, H].
Q3_EXPORT int q3_embed_norm(int dtype, const int* ids, const void* table, int vocab, const float* w, float* out,
                            int num_rows, int H, float eps, cudaStream_t stream) {
  if (!ids || !table || !w || !out || H < 1 || vocab < 1) return Q3_ERR_ARGUMENT;
  if (num_rows == 0) return Q3_OK;
  const bool vec = H % 8 == 0 && sn_aligned(table) && sn_aligned(w) && sn_aligned(out);
  int threads = (((vec ? H / 8 : H) + 31) / 32) * 32;
  threads = threads > 512 ? 512 : threads;
  cudaError_t e;
  if (dtype == Q3_DTYPE_F32)
    e = launch_pdl(vec ? embed_norm_kernel<float, true> : embed_norm_kernel<float, false>, dim3(num_rows), dim3(threads),
                   0, stream, ids, (const float*)table, vocab, w, out, H, eps);
  else if (dtype == Q3_DTYPE_BF16)
    e = launch_pdl(vec ? embed_norm_kernel<bf16, true> : embed_norm_kernel<bf16, false>, dim3(num_rows), dim3(threads), 0,
                   stream, ids, (const bf16*)table, vocab, w, out, H, eps);
  else
    return Q3_ERR_ARGUMENT;
  return e == cudaSuccess ? Q3_OK : Q3_ERR_LAUNCH;
}
