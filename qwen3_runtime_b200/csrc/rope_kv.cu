// Per-head q/k RMSNorm, rotary position encoding and the write of keys and values
// into their cache pages, in one pass over the QKV projection's output.
//
// One warp handles one (token, head).  For a q or k head (models/qwen3.py:101-103):
//   y = (x * rsqrt(mean(x^2) + eps)) * w          over the head's D values, fp32
//   rotation of the first 2*rot_half dims by cos/sin[position][i]; which two elements form
//   pair i is the position part's choice: `pairing` 0 = halves, (i, i + rot_half)
//   (layers/rope.py:7-11, what Qwen3 uses); 1 = interleaved, (2i, 2i + 1)
// q is written back in place (the attention kernels read it from the QKV buffer);
// k goes to its slot of the key pages; v heads are copied to the value pages
// unchanged (kv/paged.py:74-84).  Slot of position p: page = block_table[seq][p / ps],
// row p % ps.  Page layout [pages, kv_heads, page_size, D].
//
// A position outside the rotation tables (p < 0 or p >= max_pos) is never rotated with another
// position's angles: the (token, head) is left untouched and `error_word` (if given) is set to
// Q3_ERR_POSITION, which the host reads with the step's other error reports.
#include "common.cuh"
#include "rotary.cuh"

#define Q3_ERR_POSITION 16

template <typename T, int WARPS>
__global__ void qk_norm_rope_store_kernel(T* __restrict__ qkv, int row_stride, int nq, int nkv, int D,
                                          const float* __restrict__ q_w, const float* __restrict__ k_w,
                                          float eps, const float* __restrict__ cos_t,
                                          const float* __restrict__ sin_t, int rot_half, int max_pos,
                                          const int* __restrict__ positions, const int* __restrict__ token_seq,
                                          const int* __restrict__ block_table, int max_pages,
                                          T* __restrict__ kpages, T* __restrict__ vpages, int ps,
                                          int num_tokens, int write_kv, int pairing, int* __restrict__ error_word) {
  extern __shared__ float stage[];  // WARPS * D
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int heads = write_kv ? nq + 2 * nkv : nq;
  const long item = (long)blockIdx.x * WARPS + warp;
  if (item >= (long)num_tokens * heads) return;
  const int t = (int)(item / heads);
  const int hi = (int)(item - (long)t * heads);
  T* x = qkv + (long)t * row_stride + (long)hi * D;
  const int p = positions[t];
  if (cos_t && hi < nq + nkv && (p < 0 || p >= max_pos)) {
    if (error_word && lane == 0) atomicExch(error_word, Q3_ERR_POSITION);
    return;
  }
  long cache_row = 0;
  if (hi >= nq) {
    const int kvh = hi < nq + nkv ? hi - nq : hi - nq - nkv;
    if (p < 0 || p / ps >= max_pages) return;  // no page in the table for this position: write nothing
    const int page = block_table[(long)token_seq[t] * max_pages + p / ps];
    if (page < 0) return;
    cache_row = (((long)page * nkv + kvh) * ps + (p % ps)) * D;
  }
  if (hi >= nq + nkv) {  // value head: plain copy
    T* dst = vpages + cache_row;
    for (int d = lane; d < D; d += 32) dst[d] = x[d];
    return;
  }
  float* xs = stage + warp * D;
  float ss = 0.f;
  for (int d = lane; d < D; d += 32) {
    const float v = to_f32(x[d]);
    xs[d] = v;
    ss += v * v;
  }
  const float* w = hi < nq ? q_w : k_w;
  const float rstd = w ? rsqrtf(warp_sum(ss) / (float)D + eps) : 1.f;
  __syncwarp();
  const float* cs = cos_t ? cos_t + (long)p * rot_half : nullptr;
  const float* sn = cos_t ? sin_t + (long)p * rot_half : nullptr;
  T* dst = hi < nq ? x : kpages + cache_row;
  for (int d = lane; d < D; d += 32) {
    float y = w ? (xs[d] * rstd) * w[d] : xs[d];
    if (cs && d < 2 * rot_half) {
      const bool first = pairing ? (d & 1) == 0 : d < rot_half;  // the pair's first element
      const int i = pairing ? d >> 1 : (first ? d : d - rot_half);
      const int pd = pairing ? d ^ 1 : (first ? d + rot_half : d - rot_half);
      const float yp = w ? (xs[pd] * rstd) * w[pd] : xs[pd];
      y = first ? y * cs[i] - yp * sn[i] : y * cs[i] + yp * sn[i];
    }
    dst[d] = from_f32<T>(y);
  }
}

// The same with 16-byte accesses, for head sizes 16, 32, 64, 128, 256 with the rotation over
// the whole head (or none): D/16 threads per (token, head); a thread owns elements
// [8c, 8c+8) and [8c + D/2, 8c + D/2 + 8): with the halves pairing each element's partner is in
// the other chunk, with the interleaved pairing it is its neighbour in the same chunk.
template <typename T>
__global__ void qk_norm_rope_store_vec_kernel(T* __restrict__ qkv, int row_stride, int nq, int nkv, int D,
                                              const float* __restrict__ q_w, const float* __restrict__ k_w,
                                              float eps, const float* __restrict__ cos_t,
                                              const float* __restrict__ sin_t, int max_pos,
                                              const int* __restrict__ positions,
                                              const int* __restrict__ token_seq,
                                              const int* __restrict__ block_table, int max_pages,
                                              T* __restrict__ kpages, T* __restrict__ vpages, int ps,
                                              int tph_shift, int write_kv, int pairing,
                                              int* __restrict__ error_word) {
  // grid (tokens, blocks over one token's heads): no division finds a thread's token and head
  const int tph = D / 16;  // threads per head: a power of two, at most 16
  const int heads = write_kv ? nq + 2 * nkv : nq;
  pdl_wait();
  pdl_launch_dependents();
  const int u = blockIdx.y * blockDim.x + threadIdx.x;
  const int t = blockIdx.x;
  const int hi_raw = u >> tph_shift;
  const int c = u & (tph - 1);
  const bool live = hi_raw < heads;
  const int hi = live ? hi_raw : 0;
  const int half = D / 2;
  T* x = qkv + (long)t * row_stride + (long)hi * D;
  const int p = positions[t];
  long cache_row = -1;
  if (live && hi >= nq && p >= 0 && p / ps < max_pages) {
    const int kvh = hi < nq + nkv ? hi - nq : hi - nq - nkv;
    const int page = block_table[(long)token_seq[t] * max_pages + p / ps];
    if (page >= 0) cache_row = (((long)page * nkv + kvh) * ps + (p % ps)) * D;
  }
  float a[8], b[8];
  if (live) {
    load8(x + 8 * c, a);
    load8(x + half + 8 * c, b);
  } else {
#pragma unroll
    for (int e = 0; e < 8; ++e) a[e] = b[e] = 0.f;
  }
  const bool is_v = hi >= nq + nkv;
  const float* w = hi < nq ? q_w : k_w;
  float ss = 0.f;
#pragma unroll
  for (int e = 0; e < 8; ++e) ss += a[e] * a[e] + b[e] * b[e];
  for (int o = tph >> 1; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  if (!live) return;
  if (is_v) {
    if (cache_row >= 0) {
      store8(vpages + cache_row + 8 * c, a);
      store8(vpages + cache_row + half + 8 * c, b);
    }
    return;
  }
  if (w) {
    const float rstd = rsqrtf(ss / (float)D + eps);
    float wa[8], wb[8];
    load8(w + 8 * c, wa);
    load8(w + half + 8 * c, wb);
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      a[e] = (a[e] * rstd) * wa[e];
      b[e] = (b[e] * rstd) * wb[e];
    }
  }
  if (cos_t) {
    if (p < 0 || p >= max_pos) {
      if (error_word && c == 0) atomicExch(error_word, Q3_ERR_POSITION);
      return;
    }
    rotate_chunks(a, b, cos_t + (long)p * half, sin_t + (long)p * half, c, half, pairing);
  }
  if (hi < nq) {
    store8(x + 8 * c, a);
    store8(x + half + 8 * c, b);
  } else if (cache_row >= 0) {
    store8(kpages + cache_row + 8 * c, a);
    store8(kpages + cache_row + half + 8 * c, b);
  }
}

static inline bool rk_aligned16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

Q3_EXPORT int q3_qk_norm_rope_store(int dtype, void* qkv, int row_stride, int nq, int nkv, int D,
                                    const float* q_w, const float* k_w, float eps, const float* cos_t,
                                    const float* sin_t, int rot_half, int max_pos, const int* positions,
                                    const int* token_seq, const int* block_table, int max_pages, void* kpages,
                                    void* vpages, int ps, int num_tokens, int write_kv, int pairing,
                                    int* error_word, cudaStream_t stream) {
  if (!qkv || !positions || nq < 1 || nkv < 1 || D < 1 || pairing < 0 || pairing > 1) return Q3_ERR_ARGUMENT;
  if (cos_t && max_pos < 1) return Q3_ERR_ARGUMENT;
  if (write_kv && (!token_seq || !block_table || !kpages || !vpages || ps < 1)) return Q3_ERR_ARGUMENT;
  if (cos_t && (!sin_t || rot_half < 1 || 2 * rot_half > D)) return Q3_ERR_ARGUMENT;
  if (num_tokens == 0) return Q3_OK;
  const int tph = D / 16;
  const bool vec = D % 16 == 0 && tph >= 1 && tph <= 16 && (tph & (tph - 1)) == 0 && row_stride % 8 == 0 &&
                   (!cos_t || 2 * rot_half == D) && rk_aligned16(qkv) && rk_aligned16(kpages) &&
                   rk_aligned16(vpages) && rk_aligned16(q_w) && rk_aligned16(k_w) && rk_aligned16(cos_t) &&
                   rk_aligned16(sin_t);
  if (vec) {
    // a token's threads in blocks of 128 (Qwen3 sizes: 48 heads x 8 threads = 3 blocks, none idle)
    const int per_token = (write_kv ? nq + 2 * nkv : nq) * tph;
    int tph_shift = 0;
    while ((1 << tph_shift) < tph) ++tph_shift;
    const int vthreads = 128;
    const dim3 vgrid((unsigned)num_tokens, (unsigned)((per_token + vthreads - 1) / vthreads));
    if (vgrid.y > 65535) return Q3_ERR_UNSUPPORTED;
    cudaError_t err;
    if (dtype == Q3_DTYPE_F32)
      err = launch_pdl(qk_norm_rope_store_vec_kernel<float>, vgrid, dim3(vthreads), 0, stream, (float*)qkv,
                       row_stride, nq, nkv, D, q_w, k_w, eps, cos_t, sin_t, max_pos, positions, token_seq,
                       block_table, max_pages, (float*)kpages, (float*)vpages, ps, tph_shift, write_kv, pairing,
                       error_word);
    else if (dtype == Q3_DTYPE_BF16)
      err = launch_pdl(qk_norm_rope_store_vec_kernel<bf16>, vgrid, dim3(vthreads), 0, stream, (bf16*)qkv,
                       row_stride, nq, nkv, D, q_w, k_w, eps, cos_t, sin_t, max_pos, positions, token_seq,
                       block_table, max_pages, (bf16*)kpages, (bf16*)vpages, ps, tph_shift, write_kv, pairing,
                       error_word);
    else
      return Q3_ERR_ARGUMENT;
    return err == cudaSuccess ? Q3_OK : Q3_ERR_LAUNCH;
  }
  constexpr int WARPS = 4;
  const size_t smem = (size_t)WARPS * D * sizeof(float);
  if (smem > 48 * 1024) return Q3_ERR_UNSUPPORTED;
  const long items = (long)num_tokens * (write_kv ? nq + 2 * nkv : nq);
  const unsigned blocks = (unsigned)((items + WARPS - 1) / WARPS);
  if (dtype == Q3_DTYPE_F32)
    qk_norm_rope_store_kernel<float, WARPS><<<blocks, WARPS * 32, smem, stream>>>(
        (float*)qkv, row_stride, nq, nkv, D, q_w, k_w, eps, cos_t, sin_t, rot_half, max_pos, positions,
        token_seq, block_table, max_pages, (float*)kpages, (float*)vpages, ps, num_tokens, write_kv, pairing,
                       error_word);
  else if (dtype == Q3_DTYPE_BF16)
    qk_norm_rope_store_kernel<bf16, WARPS><<<blocks, WARPS * 32, smem, stream>>>(
        (bf16*)qkv, row_stride, nq, nkv, D, q_w, k_w, eps, cos_t, sin_t, rot_half, max_pos, positions,
        token_seq, block_table, max_pages, (bf16*)kpages, (bf16*)vpages, ps, num_tokens, write_kv, pairing,
                       error_word);
  else
    return Q3_ERR_ARGUMENT;
  return q3_launch_status();
}

// cos/sin tables [max_pos, half]: angle = float(p) * inv_freq[j], as an fp32 product
// (layers/rope.py:17-22); accurate cosf/sinf (this file is never built with fast math).
__global__ void rope_table_kernel(const float* __restrict__ inv_freq, float* __restrict__ cos_t,
                                  float* __restrict__ sin_t, int max_pos, int half) {
  const long idx = (long)blockIdx.x * blockDim.x + threadIdx.x;
  if (idx >= (long)max_pos * half) return;
  const int p = (int)(idx / half), j = (int)(idx % half);
  const float angle = (float)p * inv_freq[j];
  cos_t[idx] = cosf(angle);
  sin_t[idx] = sinf(angle);
}

Q3_EXPORT int q3_rope_table(const float* inv_freq, float* cos_t, float* sin_t, int max_pos, int half,
                            cudaStream_t stream) {
  if (!inv_freq || !cos_t || !sin_t || max_pos < 1 || half < 1) return Q3_ERR_ARGUMENT;
  const long total = (long)max_pos * half;
  rope_table_kernel<<<(unsigned)((total + 255) / 256), 256, 0, stream>>>(inv_freq, cos_t, sin_t, max_pos, half);
  return q3_launch_status();
}

// ---- per-head q/k RMSNorm, optional rotation and cache write, for rows whose k and v blocks start at
// columns of their own, whose values have a size and a head count of their own, and whose heads may be
// made of several maps ------------------------------------------------------------------------------
// One warp per (token, head).  q heads (columns h * D) are normalised in place; k heads (columns
// k_start + g * D) are normalised into their page rows; v heads (columns v_start + g * Dv) are copied
// (v_start may equal k_start: the values are then the keys as projected, since k is never changed in place).
// Key pages [pages, nkv, ps, D], value pages [pages, nv, ps, Dv].  A weight of null leaves q (or k) as it is.
// `maps`: a q or k head is `maps` consecutive parts of D / maps elements, each divided by its own root mean
// square and multiplied by the one weight of D / maps elements.  `inv_freq` (fp32 [rot_half]): the first
// 2 * rot_half elements of every part turn by angle = float(position) * inv_freq[i] (exact cosf/sinf, no
// table, so no position is out of reach), pair i = (i, i + rot_half) with pairing 0 and (2i, 2i + 1) with
// pairing 1; cos and sin are multiplied by `magnitude`.  `q_scale` (fp32 [num_tokens], or null): a token's queries are
// multiplied by its factor at the end.  `v_first` (rows v_first_stride apart with nv heads of Dv, or null): what is stored
// as a token's value is (1 - v_share) * v + v_share * v_first (fp32, one rounding).
template <typename T, int WARPS>
__global__ void qk_norm_store_kernel(T* __restrict__ proj, long row_stride, int nq, int nkv, int nv, int D, int Dv,
                                     int k_start, int v_start, const float* __restrict__ q_w,
                                     const float* __restrict__ k_w, float eps, int maps,
                                     const float* __restrict__ inv_freq, int rot_half, int pairing, float magnitude,
                                     const float* __restrict__ q_scale, const T* __restrict__ v_first,
                                     long v_first_stride, float v_share, const int* __restrict__ positions,
                                     const int* __restrict__ token_seq, const int* __restrict__ block_table,
                                     int max_pages, T* __restrict__ kpages, T* __restrict__ vpages, int ps,
                                     int num_tokens, int write_kv) {
  extern __shared__ float stage[];  // WARPS * D
  pdl_wait();
  pdl_launch_dependents();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int heads = write_kv ? nq + nkv + nv : nq;
  const long item = (long)blockIdx.x * WARPS + warp;
  if (item >= (long)num_tokens * heads) return;
  const int t = (int)(item / heads);
  const int hi = (int)(item - (long)t * heads);
  T* row = proj + (long)t * row_stride;
  const int p = positions[t];
  long slot = 0;  // the token's row among all (page, head, place) rows
  if (hi >= nq) {
    const bool is_k = hi < nq + nkv;
    const int kvh = is_k ? hi - nq : hi - nq - nkv;
    if (p < 0 || p / ps >= max_pages) return;  // no page in the table for this position: write nothing
    const int page = block_table[(long)token_seq[t] * max_pages + p / ps];
    if (page < 0) return;
    slot = ((long)page * (is_k ? nkv : nv) + kvh) * ps + (p % ps);
  }
  if (hi >= nq + nkv) {  // value head: a copy, or a blend with the first rows' head
    const int vh = hi - nq - nkv;
    const T* x = row + v_start + (long)vh * Dv;
    T* dst = vpages + slot * Dv;
    if (v_first) {
      const T* f = v_first + (long)t * v_first_stride + (long)vh * Dv;
      for (int d = lane; d < Dv; d += 32)
        dst[d] = from_f32<T>((1.f - v_share) * to_f32(x[d]) + v_share * to_f32(f[d]));
      return;
    }
    for (int d = lane; d < Dv; d += 32) dst[d] = x[d];
    return;
  }
  T* x = hi < nq ? row + (long)hi * D : row + k_start + (long)(hi - nq) * D;
  T* dst = hi < nq ? x : kpages + slot * D;
  const float* w = hi < nq ? q_w : k_w;
  const float factor = hi < nq && q_scale ? q_scale[t] : 1.f;
  if (!w && !inv_freq && factor == 1.f) {
    if (dst != x)
      for (int d = lane; d < D; d += 32) dst[d] = x[d];
    return;
  }
  float* xs = stage + warp * D;
  for (int d = lane; d < D; d += 32) xs[d] = to_f32(x[d]);
  __syncwarp();
  const int Dm = D / maps;
  if (w) {
    for (int m = 0; m < maps; ++m) {
      float ss = 0.f;
      for (int d = lane; d < Dm; d += 32) ss += xs[m * Dm + d] * xs[m * Dm + d];
      const float rstd = rsqrtf(warp_sum(ss) / (float)Dm + eps);
      for (int d = lane; d < Dm; d += 32) xs[m * Dm + d] = (xs[m * Dm + d] * rstd) * w[d];
    }
    __syncwarp();
  }
  for (int d = lane; d < D; d += 32) {
    float y = xs[d];
    const int dm = d % Dm;
    if (inv_freq && dm < 2 * rot_half) {
      const bool first = pairing ? (dm & 1) == 0 : dm < rot_half;  // the pair's first element
      const int i = pairing ? dm >> 1 : (first ? dm : dm - rot_half);
      const int pd = pairing ? dm ^ 1 : (first ? dm + rot_half : dm - rot_half);
      const float ang = (float)p * inv_freq[i];
      const float cs = cosf(ang) * magnitude, sn = sinf(ang) * magnitude;
      const float yp = xs[d - dm + pd];
      y = first ? y * cs - yp * sn : y * cs + yp * sn;
    }
    dst[d] = from_f32<T>(y * factor);
  }
}

// The same without maps and rotation, with 16-byte accesses: sizes multiples of 8 up to 256, rows, columns and pages
// 16-byte aligned.  1 << shift lanes per head, eight elements each; grid (tokens, blocks over one token's heads).
template <typename T>
__global__ void qk_norm_store_vec_kernel(T* __restrict__ proj, long row_stride, int nq, int nkv, int nv, int D, int Dv,
                                         int k_start, int v_start, const float* __restrict__ q_w,
                                         const float* __restrict__ k_w, float eps, const float* __restrict__ q_scale,
                                         const T* __restrict__ v_first, long v_first_stride, float v_share,
                                         const int* __restrict__ positions, const int* __restrict__ token_seq,
                                         const int* __restrict__ block_table, int max_pages, T* __restrict__ kpages,
                                         T* __restrict__ vpages, int ps, int shift, int write_kv) {
  pdl_wait();
  pdl_launch_dependents();
  const int t = blockIdx.x;
  const int u = blockIdx.y * blockDim.x + threadIdx.x;
  const int lanes = 1 << shift;
  const int hi = u >> shift, c = (u & (lanes - 1)) * 8;
  const bool is_q = hi < nq, is_k = !is_q && hi < nq + nkv;
  const bool live = hi < (write_kv ? nq + nkv + nv : nq);
  T* row = proj + (long)t * row_stride;
  long slot = -1;  // the token's row among all (page, head, place) rows
  if (live && !is_q) {
    const int p = positions[t];
    if (p >= 0 && p / ps < max_pages) {
      const int page = block_table[(long)token_seq[t] * max_pages + p / ps];
      const int head = is_k ? hi - nq : hi - nq - nkv;
      if (page >= 0) slot = ((long)page * (is_k ? nkv : nv) + head) * ps + (p % ps);
    }
  }
  T* x = is_q ? row + (long)hi * D : row + k_start + (long)(hi - nq) * D;
  const bool mine = live && (is_q || is_k) && c < D;
  float a[8];
#pragma unroll
  for (int e = 0; e < 8; ++e) a[e] = 0.f;
  if (mine) load8(x + c, a);
  float ss = 0.f;
#pragma unroll
  for (int e = 0; e < 8; ++e) ss += a[e] * a[e];
  for (int o = lanes >> 1; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  if (mine) {
    const float* w = is_q ? q_w : k_w;
    if (w) {
      const float rstd = rsqrtf(ss / (float)D + eps);
      float wv[8];
      load8(w + c, wv);
#pragma unroll
      for (int e = 0; e < 8; ++e) a[e] = (a[e] * rstd) * wv[e];
    }
    if (is_q && q_scale) {
      const float factor = q_scale[t];
#pragma unroll
      for (int e = 0; e < 8; ++e) a[e] *= factor;
    }
    if (is_q)
      store8(x + c, a);
    else if (slot >= 0)
      store8(kpages + slot * D + c, a);
    return;
  }
  if (!live || is_q || is_k || slot < 0) return;
  const int vh = hi - nq - nkv;
  const T* v = row + v_start + (long)vh * Dv;
  const T* f = v_first ? v_first + (long)t * v_first_stride + (long)vh * Dv : nullptr;
  for (int d = c; d < Dv; d += lanes * 8) {
    float b[8];
    load8(v + d, b);
    if (f) {
      float fv[8];
      load8(f + d, fv);
#pragma unroll
      for (int e = 0; e < 8; ++e) b[e] = (1.f - v_share) * b[e] + v_share * fv[e];
    }
    store8(vpages + slot * Dv + d, b);
  }
}

template <typename T>
static int launch_qk_norm_store_vec(void* proj, long row_stride, int nq, int nkv, int nv, int D, int Dv, int k_start,
                                    int v_start, const float* q_w, const float* k_w, float eps, const float* q_scale,
                                    const void* v_first, long v_first_stride, float v_share, const int* positions,
                                    const int* token_seq, const int* block_table, int max_pages, void* kpages,
                                    void* vpages, int ps, int num_tokens, int write_kv, cudaStream_t stream) {
  int shift = 0;
  while ((8 << shift) < D) ++shift;
  const long threads = (long)(write_kv ? nq + nkv + nv : nq) << shift;
  const dim3 grid((unsigned)num_tokens, (unsigned)((threads + 127) / 128));
  if (grid.y > 65535) return Q3_ERR_UNSUPPORTED;
  return launch_pdl(qk_norm_store_vec_kernel<T>, grid, dim3(128), 0, stream, (T*)proj, row_stride, nq, nkv, nv, D, Dv,
                    k_start, v_start, q_w, k_w, eps, q_scale, (const T*)v_first, v_first_stride, v_share, positions,
                    token_seq, block_table, max_pages, (T*)kpages, (T*)vpages, ps, shift, write_kv) == cudaSuccess
             ? Q3_OK
             : Q3_ERR_LAUNCH;
}

Q3_EXPORT int q3_qk_norm_store(int dtype, void* proj, long row_stride, int nq, int nkv, int nv, int D, int Dv,
                               int k_start, int v_start, const float* q_w, const float* k_w, float eps, int maps,
                               const float* inv_freq, int rot_half, int pairing, float magnitude,
                               const float* q_scale, const void* v_first, long v_first_stride, float v_share,
                               const int* positions, const int* token_seq, const int* block_table, int max_pages,
                               void* kpages, void* vpages, int ps, int num_tokens, int write_kv,
                               cudaStream_t stream) {
  if (!proj || !positions || nq < 1 || nkv < 1 || nv < 1 || D < 1 || Dv < 1 || ps < 1) return Q3_ERR_ARGUMENT;
  if (maps < 1 || D % maps || pairing < 0 || pairing > 1) return Q3_ERR_ARGUMENT;
  if (inv_freq && (rot_half < 1 || 2 * rot_half > D / maps)) return Q3_ERR_ARGUMENT;
  if (v_first && v_first_stride < (long)nv * Dv) return Q3_ERR_ARGUMENT;
  if (write_kv && (!token_seq || !block_table || !kpages || !vpages || max_pages < 1)) return Q3_ERR_ARGUMENT;
  if (num_tokens == 0) return Q3_OK;
  if (maps == 1 && !inv_freq && D % 8 == 0 && Dv % 8 == 0 && D <= 256 && row_stride % 8 == 0 && k_start % 8 == 0 &&
      v_start % 8 == 0 && v_first_stride % 8 == 0 && rk_aligned16(proj) && rk_aligned16(kpages) && rk_aligned16(vpages) &&
      rk_aligned16(q_w) && rk_aligned16(k_w) && rk_aligned16(v_first)) {
    if (dtype == Q3_DTYPE_F32)
      return launch_qk_norm_store_vec<float>(proj, row_stride, nq, nkv, nv, D, Dv, k_start, v_start, q_w, k_w, eps, q_scale,
                                             v_first, v_first_stride, v_share, positions, token_seq, block_table, max_pages,
                                             kpages, vpages, ps, num_tokens, write_kv, stream);
    if (dtype == Q3_DTYPE_BF16)
      return launch_qk_norm_store_vec<bf16>(proj, row_stride, nq, nkv, nv, D, Dv, k_start, v_start, q_w, k_w, eps, q_scale,
                                            v_first, v_first_stride, v_share, positions, token_seq, block_table, max_pages,
                                            kpages, vpages, ps, num_tokens, write_kv, stream);
    return Q3_ERR_ARGUMENT;
  }
  constexpr int WARPS = 4;
  const size_t smem = (size_t)WARPS * D * sizeof(float);
  if (smem > 48 * 1024) return Q3_ERR_UNSUPPORTED;
  const long items = (long)num_tokens * (write_kv ? nq + nkv + nv : nq);
  const unsigned blocks = (unsigned)((items + WARPS - 1) / WARPS);
  cudaError_t e;
  if (dtype == Q3_DTYPE_F32)
    e = launch_pdl(qk_norm_store_kernel<float, WARPS>, dim3(blocks), dim3(WARPS * 32), smem, stream, (float*)proj,
                   row_stride, nq, nkv, nv, D, Dv, k_start, v_start, q_w, k_w, eps, maps, inv_freq, rot_half, pairing,
                   magnitude, q_scale, (const float*)v_first, v_first_stride, v_share, positions, token_seq,
                   block_table, max_pages, (float*)kpages, (float*)vpages, ps,
                   num_tokens, write_kv);
  else if (dtype == Q3_DTYPE_BF16)
    e = launch_pdl(qk_norm_store_kernel<bf16, WARPS>, dim3(blocks), dim3(WARPS * 32), smem, stream, (bf16*)proj,
                   row_stride, nq, nkv, nv, D, Dv, k_start, v_start, q_w, k_w, eps, maps, inv_freq, rot_half, pairing,
                   magnitude, q_scale, (const bf16*)v_first, v_first_stride, v_share, positions, token_seq,
                   block_table, max_pages, (bf16*)kpages, (bf16*)vpages, ps,
                   num_tokens, write_kv);
  else
    return Q3_ERR_ARGUMENT;
  return e == cudaSuccess ? Q3_OK : Q3_ERR_LAUNCH;
}

// ---- factors for the queries of a step's tokens, worked out once for all layers with the same constants ----
// factors[t] = 1 + coef * ln(floor((position + 1) / every) + 1)
__global__ void query_temperature_kernel(const int* __restrict__ positions, float coef, int every,
                                         float* __restrict__ factors, int num_tokens) {
  pdl_wait();
  pdl_launch_dependents();
  const int t = blockIdx.x * blockDim.x + threadIdx.x;
  if (t < num_tokens) factors[t] = 1.f + coef * logf((float)((positions[t] + 1) / every + 1));
}

Q3_EXPORT int q3_query_temperature(const int* positions, float coef, int every, float* factors, int num_tokens,
                                   cudaStream_t stream) {
  if (!positions || !factors || every < 1) return Q3_ERR_ARGUMENT;
  if (num_tokens == 0) return Q3_OK;
  return launch_pdl(query_temperature_kernel, dim3((unsigned)((num_tokens + 127) / 128)), dim3(128), 0, stream, positions,
                    coef, every, factors, num_tokens) == cudaSuccess
             ? Q3_OK
             : Q3_ERR_LAUNCH;
}

// ---- rotations of a step's tokens, worked out once for all layers that turn by the same frequencies ----
// turns [num_tokens, 2, n]: cos then sin of float(position) * inv_freq[m] (exact cosf / sinf).
__global__ void turn_table_kernel(const int* __restrict__ positions, const float* __restrict__ inv_freq, int n,
                                  float* __restrict__ turns, long total) {
  pdl_wait();
  pdl_launch_dependents();
  const long idx = (long)blockIdx.x * blockDim.x + threadIdx.x;
  if (idx >= total) return;
  const long t = idx / n;
  const int m = (int)(idx - t * n);
  const float ang = (float)positions[t] * inv_freq[m];
  turns[(2 * t) * n + m] = cosf(ang);
  turns[(2 * t + 1) * n + m] = sinf(ang);
}

Q3_EXPORT int q3_turn_table(const int* positions, const float* inv_freq, int n, float* turns, int num_tokens,
                            cudaStream_t stream) {
  if (!positions || !inv_freq || !turns || n < 1) return Q3_ERR_ARGUMENT;
  const long total = (long)num_tokens * n;
  if (total == 0) return Q3_OK;
  return launch_pdl(turn_table_kernel, dim3((unsigned)((total + 127) / 128)), dim3(128), 0, stream, positions, inv_freq,
                    n, turns, total) == cudaSuccess
             ? Q3_OK
             : Q3_ERR_LAUNCH;
}

// ---- biases, rotation of q, k and (optionally) v, and the cache write, from a step's turn tables --------
// A row of proj holds nq query heads of D from column 0, nkv key heads from k_start, nkv value heads of Dv from
// v_start; bias (fp32, one number per column, or null) is added first.  The first 2 * qn elements of q and k heads
// turn by qk_turns [T, 2, qn], the first 2 * vn of a value head by v_turns [T, 2, vn] (either may be null); the
// sums are fp32, rounded once.  q is changed in place, k and v go to the token's rows of their pages.
// A work unit is E pairs (or E elements that do not turn): E = 8 with 16-byte accesses (halves pairing, every
// size a multiple of 8), else one.  Grid (tokens, blocks of units).
template <typename T, int E>
__device__ __forceinline__ void turn_unit(const T* __restrict__ x, const float* __restrict__ bias, T* __restrict__ dst,
                                          int unit, int n, int pairing, const float* __restrict__ cs,
                                          const float* __restrict__ sn) {
  const int turning = n / E;
  if (unit >= turning) {  // elements beyond the rotation
    const int i = 2 * n + (unit - turning) * E;
    if (E == 8) {
      float a[8];
      load8(x + i, a);
      if (bias) {
        float b[8];
        load8(bias + i, b);
#pragma unroll
        for (int e = 0; e < 8; ++e) a[e] += b[e];
      }
      store8(dst + i, a);
    } else {
      dst[i] = from_f32<T>(to_f32(x[i]) + (bias ? bias[i] : 0.f));
    }
    return;
  }
  if (E == 8) {
    const int i = unit * 8;
    float u[8], v[8], c[8], s[8];
    load8(x + i, u);
    load8(x + n + i, v);
    load8(cs + i, c);
    load8(sn + i, s);
    if (bias) {
      float b[8];
      load8(bias + i, b);
#pragma unroll
      for (int e = 0; e < 8; ++e) u[e] += b[e];
      load8(bias + n + i, b);
#pragma unroll
      for (int e = 0; e < 8; ++e) v[e] += b[e];
    }
    float a[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      a[e] = u[e] * c[e] - v[e] * s[e];
      v[e] = v[e] * c[e] + u[e] * s[e];
    }
    store8(dst + i, a);
    store8(dst + n + i, v);
  } else {
    const int i0 = pairing ? 2 * unit : unit, i1 = pairing ? i0 + 1 : unit + n;
    const float u = to_f32(x[i0]) + (bias ? bias[i0] : 0.f), v = to_f32(x[i1]) + (bias ? bias[i1] : 0.f);
    const float c = cs[unit], s = sn[unit];
    dst[i0] = from_f32<T>(u * c - v * s);
    dst[i1] = from_f32<T>(v * c + u * s);
  }
}

template <typename T, int E>
__global__ void turn_store_kernel(T* __restrict__ proj, long row_stride, int nq, int nkv, int D, int Dv, int k_start,
                                  int v_start, const float* __restrict__ bias, const float* __restrict__ qk_turns, int qn,
                                  const float* __restrict__ v_turns, int vn, int pairing,
                                  const int* __restrict__ positions, const int* __restrict__ token_seq,
                                  const int* __restrict__ block_table, int max_pages, T* __restrict__ kpages,
                                  T* __restrict__ vpages, int ps, int write_kv) {
  const int t = blockIdx.x;
  int unit = blockIdx.y * blockDim.x + threadIdx.x;
  const int qu = bias ? qn / E + (D - 2 * qn) / E : qn / E;  // without a bias what does not turn stays as it is
  const int ku = qn / E + (D - 2 * qn) / E, vu = vn / E + (Dv - 2 * vn) / E;
  if (unit >= nq * qu + (write_kv ? nkv * (ku + vu) : 0)) return;
  pdl_wait();
  pdl_launch_dependents();
  T* row = proj + (long)t * row_stride;
  const float* qc = qk_turns ? qk_turns + (long)t * 2 * qn : nullptr;
  if (unit < nq * qu) {
    const int h = unit / qu;
    T* x = row + h * D;
    turn_unit<T, E>(x, bias ? bias + h * D : nullptr, x, unit - h * qu, qn, pairing, qc, qc + qn);
    return;
  }
  unit -= nq * qu;
  const int p = positions[t];
  if (p < 0 || p / ps >= max_pages) return;  // no page in the table for this position: write nothing
  const int page = block_table[(long)token_seq[t] * max_pages + p / ps];
  if (page < 0) return;
  if (unit < nkv * ku) {
    const int g = unit / ku;
    const int col = k_start + g * D;
    turn_unit<T, E>(row + col, bias ? bias + col : nullptr, kpages + (((long)page * nkv + g) * ps + p % ps) * D,
                    unit - g * ku, qn, pairing, qc, qc + qn);
    return;
  }
  unit -= nkv * ku;
  const int g = unit / vu;
  const int col = v_start + g * Dv;
  const float* vc = v_turns ? v_turns + (long)t * 2 * vn : nullptr;
  turn_unit<T, E>(row + col, bias ? bias + col : nullptr, vpages + (((long)page * nkv + g) * ps + p % ps) * Dv,
                  unit - g * vu, vn, pairing, vc, vc + vn);
}

Q3_EXPORT int q3_turn_store(int dtype, void* proj, long row_stride, int nq, int nkv, int D, int Dv, int k_start,
                            int v_start, const float* bias, const float* qk_turns, int qn, const float* v_turns, int vn,
                            int pairing, const int* positions, const int* token_seq, const int* block_table,
                            int max_pages, void* kpages, void* vpages, int ps, int num_tokens, int write_kv,
                            cudaStream_t stream) {
  if (!proj || !positions || nq < 1 || nkv < 1 || D < 1 || Dv < 1 || ps < 1) return Q3_ERR_ARGUMENT;
  if (pairing < 0 || pairing > 1 || qn < 0 || vn < 0 || 2 * qn > D || 2 * vn > Dv) return Q3_ERR_ARGUMENT;
  if ((qn > 0) != (qk_turns != nullptr) || (vn > 0) != (v_turns != nullptr)) return Q3_ERR_ARGUMENT;
  if (write_kv && (!token_seq || !block_table || !kpages || !vpages || max_pages < 1)) return Q3_ERR_ARGUMENT;
  if (num_tokens == 0) return Q3_OK;
  const bool vec = (pairing == 0 || (qn == 0 && vn == 0)) && D % 8 == 0 && Dv % 8 == 0 && qn % 8 == 0 && vn % 8 == 0 &&
                   k_start % 8 == 0 && v_start % 8 == 0 && row_stride % 8 == 0 && rk_aligned16(proj) &&
                   rk_aligned16(bias) && rk_aligned16(qk_turns) && rk_aligned16(v_turns) && rk_aligned16(kpages) &&
                   rk_aligned16(vpages);
  const int E = vec ? 8 : 1;
  const int units = nq * (bias ? (D - qn) / E : qn / E) + (write_kv ? nkv * ((D - qn) / E + (Dv - vn) / E) : 0);
  if (units == 0) return Q3_OK;
  const dim3 grid((unsigned)num_tokens, (unsigned)((units + 127) / 128));
  if (grid.y > 65535) return Q3_ERR_UNSUPPORTED;
  cudaError_t e;
#define Q3_TURN_STORE(T, EE)                                                                                         \
  e = launch_pdl(turn_store_kernel<T, EE>, grid, dim3(128), 0, stream, (T*)proj, row_stride, nq, nkv, D, Dv, k_start,  \
                 v_start, bias, qk_turns, qn, v_turns, vn, pairing, positions, token_seq, block_table, max_pages,    \
                 (T*)kpages, (T*)vpages, ps, write_kv)
  if (dtype == Q3_DTYPE_F32) {
    if (vec) Q3_TURN_STORE(float, 8); else Q3_TURN_STORE(float, 1);
  } else if (dtype == Q3_DTYPE_BF16) {
    if (vec) Q3_TURN_STORE(bf16, 8); else Q3_TURN_STORE(bf16, 1);
  } else {
    return Q3_ERR_ARGUMENT;
  }
#undef Q3_TURN_STORE
  return e == cudaSuccess ? Q3_OK : Q3_ERR_LAUNCH;
}
