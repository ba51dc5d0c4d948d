// Attention over the paged cache in bfloat16 for keys and values of sizes of their own, under a chunked mask, with
// values that may be turned by their positions.  A token at position p sees keys lo .. p with lo = floor(p / chunk) *
// chunk (chunk > 0; chunks counted from the sequence's first token) or 0.  With turn tables the cached values are
// turned by their own positions, and a head's sum is turned back by the token's angles before it is stored.  With
// sinks (fp32, one score per head) each softmax's denominator has one more term, exp(sink_h), that stands for no key.
// Key pages [pages, nkv, ps, D], value pages [pages, nkv, ps, DV]; D and DV multiples of 8 up to 256.  The kernels
// are made for DP, DVP in {64, 128, 256}; columns between a size and its DP are zeros in shared memory.
//
//   chunk_prefill   prompt portions on the tensor cores: a work item is (sequence, kv head, block of 128 (token, head
//                   of the group) rows), keys and values in tiles of 64 through a cp.async ring into XOR-swizzled
//                   shared memory, S = Q K^T and O += P V as m16n8k16 MMAs with fp32 accumulators, an online softmax
//                   in fp32 (exp2 with the scale folded in).  Tiles before the block's first visible key are never
//                   loaded.
//   chunk_decode    sequences that bring one token: a block per (slice of the visible keys, kv head, sequence), the
//                   group's queries as the 16 rows of an MMA tile, 4 warps with 16 keys of a tile each; the slices'
//                   partial results are merged by whichever block of a (sequence, kv head) finishes last.
#include "common.cuh"
#include "mma_tiles.cuh"

namespace {

constexpr int TILE = 64;

__device__ __forceinline__ int first_seen(int p, int chunk) { return chunk > 0 ? p / chunk * chunk : 0; }

// Element d of a row of fp32 values in shared memory, turned back by cs = [cos(pairs) | sin(pairs)] (null: as it is).
__device__ __forceinline__ float turned_back(const float* row, int d, const float* cs, int pairs, int pairing) {
  const float v = row[d];
  if (!cs || d >= 2 * pairs) return v;
  const bool first = pairing ? (d & 1) == 0 : d < pairs;
  const int m = pairing ? d >> 1 : (first ? d : d - pairs);
  const float other = row[pairing ? d ^ 1 : (first ? d + pairs : d - pairs)];
  return first ? v * cs[m] + other * cs[pairs + m] : v * cs[m] - other * cs[pairs + m];
}

constexpr int BLOCK_M = 128;
constexpr int PF_WARPS = BLOCK_M / 16;
constexpr int PF_THREADS = PF_WARPS * 32;

template <int DP, int DVP> __host__ __device__ constexpr int prefill_stages() { return DP + DVP > 256 ? 2 : 3; }

template <int DP, int DVP>
__global__ void __launch_bounds__(PF_THREADS, 1)
chunk_prefill_kernel(const bf16* __restrict__ q, int q_stride, const bf16* __restrict__ kpages,
                     const bf16* __restrict__ vpages, const int* __restrict__ block_table, int max_pages,
                     const int* __restrict__ kv_lens, const int* __restrict__ cu_seqlens, bf16* __restrict__ out,
                     long out_stride, int num_seqs, int nq, int nkv, int D, int DV, int ps, float scale_log2, int chunk,
                     int skip_single, const float* __restrict__ turns, int pairs, int pairing,
                     const float* __restrict__ sinks) {
  constexpr int STAGES = prefill_stages<DP, DVP>();
  constexpr int KCH = DP / 8, VCH = DVP / 8;
  constexpr int K_BYTES = TILE * DP * 2, V_BYTES = TILE * DVP * 2;
  extern __shared__ __align__(128) unsigned char smem[];
  unsigned char* q_s = smem;                      // [BLOCK_M][DP]
  unsigned char* kv_s = smem + BLOCK_M * DP * 2;  // STAGES x (K tile, V tile); later O rows in fp32
  __shared__ int s_item[2];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int kvh = blockIdx.y;
  const int G = nq / nkv;
  if (tid == 0) {
    int acc = 0, found = -1, rb = 0;
    const int w = gridDim.x - 1 - blockIdx.x;  // long rows first
    for (int s = 0; s < num_seqs; ++s) {
      const int ql = cu_seqlens[s + 1] - cu_seqlens[s];
      if (ql <= 0 || (skip_single && ql == 1)) continue;
      const int nb = (ql * G + BLOCK_M - 1) / BLOCK_M;
      if (w < acc + nb) {
        found = s;
        rb = w - acc;
        break;
      }
      acc += nb;
    }
    s_item[0] = found;
    s_item[1] = rb;
  }
  __syncthreads();
  const int seq = s_item[0];
  if (seq < 0) return;
  const int row0 = s_item[1] * BLOCK_M;
  const int tok0 = cu_seqlens[seq];
  const int q_len = cu_seqlens[seq + 1] - tok0;
  const int rows = q_len * G;
  const int base_pos = kv_lens[seq] - q_len;
  const int* bt = block_table + (long)seq * max_pages;
  for (int c = tid; c < BLOCK_M * KCH; c += PF_THREADS) {
    const int r = c / KCH, ch = c % KCH;
    const int R = row0 + r;
    uint4 v = make_uint4(0, 0, 0, 0);
    if (R < rows && ch * 8 < D) {
      const int tk = R / G, hd = kvh * G + (R - tk * G);
      v = *reinterpret_cast<const uint4*>(q + (long)(tok0 + tk) * q_stride + (long)hd * D + ch * 8);
    }
    *reinterpret_cast<uint4*>(q_s + swz<DP>(r, ch)) = v;
  }
  const int last_row = min(rows, row0 + BLOCK_M) - 1;
  const int p_min = base_pos + row0 / G, p_max = base_pos + last_row / G;
  const int k_lo = first_seen(p_min, chunk);  // the first key any row of the block sees
  const int t_begin = k_lo / TILE, num_tiles = p_max / TILE - t_begin + 1;

  auto load_tile = [&](int tile, int stage) {
    unsigned char* k_dst = kv_s + (size_t)stage * (K_BYTES + V_BYTES);
    unsigned char* v_dst = k_dst + K_BYTES;
    const int base = (t_begin + tile) * TILE;
    constexpr int MCH = KCH > VCH ? KCH : VCH;
    for (int c = tid; c < TILE * MCH; c += PF_THREADS) {
      const int r = c / MCH, ch = c % MCH;
      const int j = base + r;
      const bool valid = j >= k_lo && j <= p_max;
      long row = 0;
      if (valid) row = ((long)bt[j / ps] * nkv + kvh) * ps + (j % ps);
      if (ch < KCH) {
        const bool in = valid && ch * 8 < D;
        cp_async16(smem_u32(k_dst + swz<DP>(r, ch)), kpages + (in ? row * D + ch * 8 : 0), in ? 16 : 0);
      }
      if (ch < VCH) {
        const bool in = valid && ch * 8 < DV;
        cp_async16(smem_u32(v_dst + swz<DVP>(r, ch)), vpages + (in ? row * DV + ch * 8 : 0), in ? 16 : 0);
      }
    }
  };
  for (int s = 0; s < STAGES - 1; ++s) {
    if (s < num_tiles) load_tile(s, s);
    cp_async_commit();
  }
  __syncthreads();  // q_s complete

  constexpr bool Q_REGS = DP <= 128 && DVP <= 128;  // the warp's queries stay in registers where there is room
  uint32_t qreg[Q_REGS ? DP / 16 : 1][4];
  if (Q_REGS) {
#pragma unroll
    for (int ks = 0; ks < DP / 16; ++ks)
      ldmatrix_x4(qreg[Q_REGS ? ks : 0], smem_u32(q_s + swz<DP>(warp * 16 + (lane & 15), 2 * ks + (lane >> 4))));
  }
  int pos[2], lo[2];
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int R = row0 + warp * 16 + (lane >> 2) + r * 8;
    pos[r] = R < rows ? base_pos + R / G : -1;
    lo[r] = pos[r] >= 0 ? first_seen(pos[r], chunk) : 0;
  }
  const int Rw0 = row0 + warp * 16, Rw1 = min(rows, Rw0 + 16) - 1;
  const bool warp_live = Rw0 < rows;
  const int wp_min = base_pos + Rw0 / G, wp_max = warp_live ? base_pos + Rw1 / G : -1;
  const int wlo_min = first_seen(wp_min, chunk), wlo_max = warp_live ? first_seen(wp_max, chunk) : 0;

  float o[DVP / 8][4];
#pragma unroll
  for (int i = 0; i < DVP / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.f, 0.f};

  for (int tile = 0; tile < num_tiles; ++tile) {
    cp_async_wait<STAGES - 2>();
    __syncthreads();
    {
      const int nxt = tile + STAGES - 1;
      if (nxt < num_tiles) load_tile(nxt, nxt % STAGES);
      cp_async_commit();
    }
    const int key0 = (t_begin + tile) * TILE;
    if (!warp_live || key0 > wp_max || key0 + TILE - 1 < wlo_min) continue;  // nothing for this warp
    const unsigned char* k_t = kv_s + (size_t)(tile % STAGES) * (K_BYTES + V_BYTES);
    const unsigned char* v_t = k_t + K_BYTES;
    float s[TILE / 8][4];
#pragma unroll
    for (int n = 0; n < TILE / 8; ++n) s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.f;
#pragma unroll
    for (int ks = 0; ks < DP / 16; ++ks) {
      if (ks * 16 >= D) break;  // padding columns
      uint32_t qa[4];
      if (Q_REGS) {
#pragma unroll
        for (int e = 0; e < 4; ++e) qa[e] = qreg[Q_REGS ? ks : 0][e];
      } else {
        ldmatrix_x4(qa, smem_u32(q_s + swz<DP>(warp * 16 + (lane & 15), 2 * ks + (lane >> 4))));
      }
#pragma unroll
      for (int nn = 0; nn < TILE / 16; ++nn) {
        uint32_t kb[4];
        const int row = nn * 16 + (lane & 7) + ((lane >> 4) << 3);
        ldmatrix_x4(kb, smem_u32(k_t + swz<DP>(row, 2 * ks + ((lane >> 3) & 1))));
        mma_bf16(s[2 * nn], qa, kb[0], kb[1]);
        mma_bf16(s[2 * nn + 1], qa, kb[2], kb[3]);
      }
    }
    if (key0 + TILE - 1 > wp_min || key0 < wlo_max) {  // the diagonal or a chunk's start crosses the tile
#pragma unroll
      for (int n = 0; n < TILE / 8; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int j = key0 + n * 8 + 2 * (lane & 3) + (e & 1);
          if (j > pos[e >> 1] || j < lo[e >> 1]) s[n][e] = -INFINITY;
        }
    }
    float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
    for (int n = 0; n < TILE / 8; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) mx[e >> 1] = fmaxf(mx[e >> 1], s[n][e]);
    float corr[2], m_use[2];
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
      mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
      const float m_new = fmaxf(m_run[r], mx[r]);
      m_use[r] = m_new == -INFINITY ? 0.f : m_new;
      corr[r] = exp2f((m_run[r] - m_use[r]) * scale_log2);
      m_run[r] = m_new;
      l_run[r] *= corr[r];
    }
#pragma unroll
    for (int n = 0; n < TILE / 8; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        s[n][e] = exp2f((s[n][e] - m_use[e >> 1]) * scale_log2);
        l_run[e >> 1] += s[n][e];
      }
    if (__any_sync(0xffffffffu, corr[0] != 1.f || corr[1] != 1.f)) {
#pragma unroll
      for (int i = 0; i < DVP / 8; ++i) {
        o[i][0] *= corr[0]; o[i][1] *= corr[0];
        o[i][2] *= corr[1]; o[i][3] *= corr[1];
      }
    }
#pragma unroll
    for (int kk = 0; kk < TILE / 16; ++kk) {
      uint32_t pa[4];
      pa[0] = pack_bf16(s[2 * kk][0], s[2 * kk][1]);
      pa[1] = pack_bf16(s[2 * kk][2], s[2 * kk][3]);
      pa[2] = pack_bf16(s[2 * kk + 1][0], s[2 * kk + 1][1]);
      pa[3] = pack_bf16(s[2 * kk + 1][2], s[2 * kk + 1][3]);
#pragma unroll
      for (int i = 0; i < DVP / 16; ++i) {
        if (i * 16 >= DV) break;
        uint32_t vb[4];
        const int row = kk * 16 + (lane & 7) + (((lane >> 3) & 1) << 3);
        ldmatrix_x4_trans(vb, smem_u32(v_t + swz<DVP>(row, 2 * i + (lane >> 4))));
        mma_bf16(o[2 * i], pa, vb[0], vb[1]);
        mma_bf16(o[2 * i + 1], pa, vb[2], vb[3]);
      }
    }
  }
  cp_async_wait<0>();
  float inv[2];
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    l_run[r] += __shfl_xor_sync(0xffffffffu, l_run[r], 1);
    l_run[r] += __shfl_xor_sync(0xffffffffu, l_run[r], 2);
    const int R = row0 + warp * 16 + (lane >> 2) + r * 8;
    if (sinks && R < rows) l_run[r] += exp2f(sinks[kvh * G + R % G] * LOG2_E - m_run[r] * scale_log2);
    inv[r] = l_run[r] > 0.f ? 1.f / l_run[r] : 0.f;
  }
  if (!turns) {
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int R = row0 + warp * 16 + (lane >> 2) + r * 8;
      if (R >= rows) continue;
      const int tk = R / G, hd = kvh * G + (R - tk * G);
      bf16* dst = out + (long)(tok0 + tk) * out_stride + (long)hd * DV + 2 * (lane & 3);
#pragma unroll
      for (int i = 0; i < DVP / 8; ++i)
        if (i * 8 < DV) *reinterpret_cast<uint32_t*>(dst + i * 8) = pack_bf16(o[i][2 * r] * inv[r], o[i][2 * r + 1] * inv[r]);
    }
    return;
  }
  // the sums as fp32 rows where the ring was, each warp its own 16 rows, then turned back
  __syncthreads();
  constexpr int OS = DVP + 8;
  float* o_s = reinterpret_cast<float*>(smem) + (size_t)warp * 16 * OS;
#pragma unroll
  for (int i = 0; i < DVP / 8; ++i)
#pragma unroll
    for (int r = 0; r < 2; ++r)
      *reinterpret_cast<float2*>(o_s + ((lane >> 2) + r * 8) * OS + i * 8 + 2 * (lane & 3)) =
          make_float2(o[i][2 * r] * inv[r], o[i][2 * r + 1] * inv[r]);
  __syncwarp();
  for (int r = 0; r < 16; ++r) {
    const int R = Rw0 + r;
    if (R >= rows) break;
    const int tk = R / G, hd = kvh * G + (R - tk * G);
    const float* cs = turns + (long)(tok0 + tk) * 2 * pairs;
    bf16* dst = out + (long)(tok0 + tk) * out_stride + (long)hd * DV;
    for (int d = 2 * lane; d < DV; d += 64)
      *reinterpret_cast<uint32_t*>(dst + d) = pack_bf16(turned_back(o_s + r * OS, d, cs, pairs, pairing),
                                                        turned_back(o_s + r * OS, d + 1, cs, pairs, pairing));
  }
}

template <int DP, int DVP>
int launch_chunk_prefill(const bf16* q, int q_stride, const bf16* kpages, const bf16* vpages, const int* block_table,
                         int max_pages, const int* kv_lens, const int* cu_seqlens, bf16* out, long out_stride,
                         int num_seqs, int num_work, int nq, int nkv, int D, int DV, int ps, float scale, int chunk,
                         int skip_single, const float* turns, int pairs, int pairing, const float* sinks,
                         cudaStream_t stream) {
  const size_t pipe = (size_t)BLOCK_M * DP * 2 + (size_t)prefill_stages<DP, DVP>() * TILE * (DP + DVP) * 2;
  const size_t rows = (size_t)BLOCK_M * (DVP + 8) * 4;
  const size_t smem = pipe > rows ? pipe : rows;
  static bool configured_on[Q3_MAX_DEVICES];
  bool& configured = configured_on[q3_current_device()];
  if (!configured) {
    if (cudaFuncSetAttribute(chunk_prefill_kernel<DP, DVP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) !=
        cudaSuccess)
      return Q3_ERR_LAUNCH;
    configured = true;
  }
  chunk_prefill_kernel<DP, DVP><<<dim3(num_work, nkv), PF_THREADS, smem, stream>>>(
      q, q_stride, kpages, vpages, block_table, max_pages, kv_lens, cu_seqlens, out, out_stride, num_seqs, nq, nkv, D, DV,
      ps, scale * 1.4426950408889634f, chunk, skip_single, turns, pairs, pairing, sinks);
  return q3_launch_status();
}

// ---- one token per sequence --------------------------------------------------------------------------
constexpr int DC_WARPS = 4;
constexpr int DC_THREADS = DC_WARPS * 32;

// What a (sequence, kv head)'s slices leave: mid_o [item][G][splits][DVP] normalised sums, mid_lse [item][G][splits]
// their log-sum-exps (base 2), item = place in the launch * nkv + kv head.  Slices are multiples of 64 keys from the
// tile of the first visible key on, as many as the sequence's visible keys need, at most `splits`.
template <int DP, int DVP>
__global__ void __launch_bounds__(DC_THREADS)
chunk_decode_kernel(const bf16* __restrict__ q, int q_stride, const bf16* __restrict__ kpages,
                    const bf16* __restrict__ vpages, const int* __restrict__ block_table, int max_pages,
                    const int* __restrict__ kv_lens, const int* __restrict__ cu_seqlens, const int* __restrict__ seq_list,
                    bf16* __restrict__ out, long out_stride, float* mid_o, float* mid_lse, int* tickets, int nq, int nkv,
                    int D, int DV, int ps, float scale_log2, int chunk, int splits, const float* __restrict__ turns,
                    int pairs, int pairing, const float* __restrict__ sinks) {
  constexpr int KCH = DP / 8, VCH = DVP / 8;
  constexpr int K_BYTES = TILE * DP * 2, V_BYTES = TILE * DVP * 2;
  extern __shared__ __align__(128) unsigned char smem[];
  unsigned char* q_s = smem;                // [16][DP]
  unsigned char* kv_s = smem + 16 * DP * 2;  // 2 x (K tile, V tile); later the warps' results
  __shared__ int last_s;
  pdl_wait();
  const int split = blockIdx.x, kvh = blockIdx.y, slot = blockIdx.z;
  const int seq = seq_list ? seq_list[slot] : slot;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int G = nq / nkv;
  const int kv_len = kv_lens[seq], tok = cu_seqlens[seq], p = kv_len - 1;
  const int lo = first_seen(p, chunk);
  const int begin0 = lo & ~(TILE - 1);
  const int tiles_all = (kv_len - begin0 + TILE - 1) / TILE;
  const int per = (tiles_all + splits - 1) / splits;       // tiles of a slice
  const int slices = (tiles_all + per - 1) / per;
  if (split >= slices) return;
  const int k_begin = begin0 + split * per * TILE;
  const int k_end = min(kv_len, k_begin + per * TILE);
  const int num_tiles = (k_end - k_begin + TILE - 1) / TILE;
  const int* bt = block_table + (long)seq * max_pages;
  const long item = (long)slot * nkv + kvh;

  for (int c = tid; c < 16 * KCH; c += DC_THREADS) {
    const int row = c / KCH, ch = c % KCH;
    uint4 v = make_uint4(0, 0, 0, 0);
    if (row < G && ch * 8 < D)
      v = *reinterpret_cast<const uint4*>(q + (long)tok * q_stride + (long)(kvh * G + row) * D + ch * 8);
    *reinterpret_cast<uint4*>(q_s + swz<DP>(row, ch)) = v;
  }
  // neighbouring threads on a key: its page is looked up once a thread and tile
  auto load_tile = [&](int tile, int stage) {
    unsigned char* k_dst = kv_s + (size_t)stage * (K_BYTES + V_BYTES);
    unsigned char* v_dst = k_dst + K_BYTES;
    const int base = k_begin + tile * TILE;
    constexpr int MCH = KCH > VCH ? KCH : VCH;
    constexpr int TPR = MCH < 16 ? MCH : 16;            // threads on a row (neighbouring chunks)
    for (int r = tid / TPR; r < TILE; r += DC_THREADS / TPR) {
      const int j = base + r;
      const bool valid = j >= lo && j < k_end;
      long row = 0;
      if (valid) row = ((long)bt[j / ps] * nkv + kvh) * ps + (j % ps);
#pragma unroll
      for (int ch = tid % TPR; ch < MCH; ch += TPR) {
        if (ch < KCH) {
          const bool in = valid && ch * 8 < D;
          cp_async16(smem_u32(k_dst + swz<DP>(r, ch)), kpages + (in ? row * D + ch * 8 : 0), in ? 16 : 0);
        }
        if (ch < VCH) {
          const bool in = valid && ch * 8 < DV;
          cp_async16(smem_u32(v_dst + swz<DVP>(r, ch)), vpages + (in ? row * DV + ch * 8 : 0), in ? 16 : 0);
        }
      }
    }
  };
  load_tile(0, 0);
  cp_async_commit();
  __syncthreads();  // q_s complete

  constexpr bool Q_REGS = DP <= 128;
  uint32_t qreg[Q_REGS ? DP / 16 : 1][4];
  if (Q_REGS) {
#pragma unroll
    for (int ks = 0; ks < DP / 16; ++ks)
      ldmatrix_x4(qreg[Q_REGS ? ks : 0], smem_u32(q_s + swz<DP>(lane & 15, 2 * ks + (lane >> 4))));
  }
  float o[DVP / 8][4];
#pragma unroll
  for (int i = 0; i < DVP / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.f, 0.f};

  for (int tile = 0; tile < num_tiles; ++tile) {
    cp_async_wait<0>();
    __syncthreads();
    if (tile + 1 < num_tiles) load_tile(tile + 1, (tile + 1) & 1);
    cp_async_commit();
    const unsigned char* k_t = kv_s + (size_t)(tile & 1) * (K_BYTES + V_BYTES);
    const unsigned char* v_t = k_t + K_BYTES;
    const int key0 = k_begin + tile * TILE + warp * 16;  // this warp's 16 keys
    if (key0 >= k_end || key0 + 15 < lo) continue;
    float s[2][4];
#pragma unroll
    for (int n = 0; n < 2; ++n) s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.f;
#pragma unroll
    for (int ks = 0; ks < DP / 16; ++ks) {
      if (ks * 16 >= D) break;
      uint32_t qa[4], kb[4];
      if (Q_REGS) {
#pragma unroll
        for (int e = 0; e < 4; ++e) qa[e] = qreg[Q_REGS ? ks : 0][e];
      } else {
        ldmatrix_x4(qa, smem_u32(q_s + swz<DP>(lane & 15, 2 * ks + (lane >> 4))));
      }
      const int row = warp * 16 + (lane & 7) + ((lane >> 4) << 3);
      ldmatrix_x4(kb, smem_u32(k_t + swz<DP>(row, 2 * ks + ((lane >> 3) & 1))));
      mma_bf16(s[0], qa, kb[0], kb[1]);
      mma_bf16(s[1], qa, kb[2], kb[3]);
    }
    float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int j = key0 + n * 8 + 2 * (lane & 3) + (e & 1);
        if (j < lo || j >= k_end) s[n][e] = -INFINITY;
        mx[e >> 1] = fmaxf(mx[e >> 1], s[n][e]);
      }
    float corr[2], m_use[2];
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
      mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
      const float m_new = fmaxf(m_run[r], mx[r]);
      m_use[r] = m_new == -INFINITY ? 0.f : m_new;
      corr[r] = exp2f((m_run[r] - m_use[r]) * scale_log2);
      m_run[r] = m_new;
      l_run[r] *= corr[r];
    }
    float pv[2][4];
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        pv[n][e] = exp2f((s[n][e] - m_use[e >> 1]) * scale_log2);
        l_run[e >> 1] += pv[n][e];
      }
    const uint32_t pa[4] = {pack_bf16(pv[0][0], pv[0][1]), pack_bf16(pv[0][2], pv[0][3]), pack_bf16(pv[1][0], pv[1][1]),
                            pack_bf16(pv[1][2], pv[1][3])};
    if (__any_sync(0xffffffffu, corr[0] != 1.f || corr[1] != 1.f)) {
#pragma unroll
      for (int i = 0; i < DVP / 8; ++i) {
        o[i][0] *= corr[0]; o[i][1] *= corr[0];
        o[i][2] *= corr[1]; o[i][3] *= corr[1];
      }
    }
#pragma unroll
    for (int i = 0; i < DVP / 16; ++i) {
      if (i * 16 >= DV) break;
      uint32_t vb[4];
      const int row = warp * 16 + (lane & 7) + (((lane >> 3) & 1) << 3);
      ldmatrix_x4_trans(vb, smem_u32(v_t + swz<DVP>(row, 2 * i + (lane >> 4))));
      mma_bf16(o[2 * i], pa, vb[0], vb[1]);
      mma_bf16(o[2 * i + 1], pa, vb[2], vb[3]);
    }
  }
  // ---- the four warps' results side by side, then merged --------------------------------------------
  pdl_launch_dependents();
  cp_async_wait<0>();
  __syncthreads();
  constexpr int OS = DVP + 8;
  float* o_s = reinterpret_cast<float*>(kv_s);  // [WARPS][16][OS]
  float* ml_s = o_s + DC_WARPS * 16 * OS;       // [WARPS][16][2]
  float* fin = ml_s + DC_WARPS * 32;            // [16][DVP]: the result's rows
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    l_run[r] += __shfl_xor_sync(0xffffffffu, l_run[r], 1);
    l_run[r] += __shfl_xor_sync(0xffffffffu, l_run[r], 2);
    const int row = warp * 16 + (lane >> 2) + r * 8;
#pragma unroll
    for (int i = 0; i < DVP / 8; ++i)
      *reinterpret_cast<float2*>(o_s + (size_t)row * OS + i * 8 + 2 * (lane & 3)) = make_float2(o[i][2 * r], o[i][2 * r + 1]);
    if ((lane & 3) == 0) {
      ml_s[row * 2] = m_run[r];
      ml_s[row * 2 + 1] = l_run[r];
    }
  }
  __syncthreads();
  for (int idx = tid; idx < G * DV; idx += DC_THREADS) {
    const int g = idx / DV, d = idx - g * DV;
    float m = -INFINITY;
#pragma unroll
    for (int w = 0; w < DC_WARPS; ++w) m = fmaxf(m, ml_s[(w * 16 + g) * 2]);
    float l = 0.f, acc = 0.f;
#pragma unroll
    for (int w = 0; w < DC_WARPS; ++w) {
      const float mw = ml_s[(w * 16 + g) * 2];
      const float f = mw == -INFINITY ? 0.f : exp2f((mw - m) * scale_log2);
      l += ml_s[(w * 16 + g) * 2 + 1] * f;
      acc += o_s[((size_t)w * 16 + g) * OS + d] * f;
    }
    if (slices == 1) {
      if (sinks) l += exp2f(sinks[kvh * G + g] * LOG2_E - m * scale_log2);
      fin[g * DVP + d] = acc / l;
    } else {
      const float val = l > 0.f ? acc / l : 0.f;
      mid_o[((item * G + g) * splits + split) * DVP + d] = val;
      if (d == 0) mid_lse[(item * G + g) * splits + split] = l > 0.f ? m * scale_log2 + log2f(l) : -INFINITY;
    }
  }
  if (slices > 1) {
    __threadfence();
    __syncthreads();
    if (tid == 0) {
      last_s = atomicAdd(tickets + item, 1) == slices - 1;
      if (last_s) tickets[item] = 0;
    }
    __syncthreads();
    if (!last_s) return;
    __threadfence();
    for (int idx = tid; idx < G * DV; idx += DC_THREADS) {
      const int g = idx / DV, d = idx - g * DV;
      const float* lse = mid_lse + (item * G + g) * splits;
      const float* src = mid_o + (item * G + g) * splits * DVP + d;
      float mx = -INFINITY;
      for (int s = 0; s < slices; ++s) mx = fmaxf(mx, __ldcg(lse + s));
      float acc = 0.f, wsum = sinks ? exp2f(sinks[kvh * G + g] * LOG2_E - mx) : 0.f;
#pragma unroll 4
      for (int s = 0; s < slices; ++s) {
        const float w = exp2f(__ldcg(lse + s) - mx);
        wsum += w;
        acc = fmaf(w, __ldcg(src + (long)s * DVP), acc);
      }
      fin[g * DVP + d] = acc / wsum;
    }
  }
  __syncthreads();
  const float* cs = turns ? turns + (long)tok * 2 * pairs : nullptr;
  bf16* dst = out + (long)tok * out_stride + (long)kvh * G * DV;
  for (int idx = 2 * tid; idx < G * DV; idx += 2 * DC_THREADS) {
    const int g = idx / DV, d = idx - g * DV;
    *reinterpret_cast<uint32_t*>(dst + idx) = pack_bf16(turned_back(fin + g * DVP, d, cs, pairs, pairing),
                                                        turned_back(fin + g * DVP, d + 1, cs, pairs, pairing));
  }
}

template <int DP, int DVP>
int launch_chunk_decode(const bf16* q, int q_stride, const bf16* kpages, const bf16* vpages, const int* block_table,
                        int max_pages, const int* kv_lens, const int* cu_seqlens, const int* seq_list, bf16* out,
                        long out_stride, float* mid_o, float* mid_lse, int* tickets, int num_seqs, int nq, int nkv, int D,
                        int DV, int ps, float scale, int chunk, int splits, const float* turns, int pairs, int pairing,
                        const float* sinks, cudaStream_t stream) {
  const size_t pipe = (size_t)2 * TILE * (DP + DVP) * 2;
  const size_t merge = ((size_t)DC_WARPS * 16 * (DVP + 8) + DC_WARPS * 32 + 16 * DVP) * 4;
  const size_t smem = 16 * DP * 2 + (pipe > merge ? pipe : merge);
  static bool configured_on[Q3_MAX_DEVICES];
  bool& configured = configured_on[q3_current_device()];
  if (!configured) {
    if (cudaFuncSetAttribute(chunk_decode_kernel<DP, DVP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) !=
        cudaSuccess)
      return Q3_ERR_LAUNCH;
    configured = true;
  }
  return launch_pdl(chunk_decode_kernel<DP, DVP>, dim3(splits, nkv, num_seqs), dim3(DC_THREADS), smem, stream, q, q_stride,
                    kpages, vpages, block_table, max_pages, kv_lens, cu_seqlens, seq_list, out, out_stride, mid_o, mid_lse,
                    tickets, nq, nkv, D, DV, ps, scale * 1.4426950408889634f, chunk, splits, turns, pairs,
                    pairing, sinks) == cudaSuccess
             ? Q3_OK
             : Q3_ERR_LAUNCH;
}

bool chunk_sizes_ok(const void* q, int q_stride, const void* kpages, const void* vpages, const void* out, long out_stride,
                    int nq, int nkv, int D, int DV) {
  return D >= 8 && DV >= 8 && D <= 256 && DV <= 256 && D % 8 == 0 && DV % 8 == 0 && q_stride % 8 == 0 &&
         out_stride % 2 == 0 && nq / nkv <= 16 && nkv <= 65535 &&
         !(((uintptr_t)q | (uintptr_t)kpages | (uintptr_t)vpages) & 15) && !((uintptr_t)out & 3);
}

}  // namespace

#define Q3_CHUNK_SIZES(CALL)                                                                    \
  if (D <= 64) { if (DV <= 64) CALL(64, 64); if (DV <= 128) CALL(64, 128); CALL(64, 256); }      \
  if (D <= 128) { if (DV <= 64) CALL(128, 64); if (DV <= 128) CALL(128, 128); CALL(128, 256); }  \
  if (DV <= 64) CALL(256, 64);                                                                  \
  if (DV <= 128) CALL(256, 128);                                                                \
  CALL(256, 256);

// Prompt portions: num_work = sum over the served sequences of ceil(q_len * (nq / nkv) / 128); with skip_single the
// sequences of one token are left out.  turns: null, or fp32 [num_tokens, 2, pairs].  sinks: null, or fp32
// [nq].  Groups of at most 16 heads.
Q3_EXPORT int q3_chunk_attention_prefill(const void* q, int q_stride, const void* kpages, const void* vpages,
                                         const int* block_table, int max_pages, const int* kv_lens,
                                         const int* cu_seqlens, void* out, long out_stride, int num_seqs, int num_work,
                                         int nq, int nkv, int D, int DV, int ps, float scale, int chunk, int skip_single,
                                         const float* turns, int pairs, int pairing, const float* sinks,
                                         cudaStream_t stream) {
  if (!q || !kpages || !vpages || !block_table || !kv_lens || !cu_seqlens || !out) return Q3_ERR_ARGUMENT;
  if (nq < 1 || nkv < 1 || nq % nkv || ps < 1 || num_seqs < 0 || num_work < 0 || chunk < 0) return Q3_ERR_ARGUMENT;
  if (turns && (pairs < 1 || 2 * pairs > DV || pairing < 0 || pairing > 1)) return Q3_ERR_ARGUMENT;
  if (!chunk_sizes_ok(q, q_stride, kpages, vpages, out, out_stride, nq, nkv, D, DV)) return Q3_ERR_UNSUPPORTED;
  if (num_work == 0) return Q3_OK;
#define Q3_CHUNK_PREFILL(dp, dvp)                                                                                     \
  return launch_chunk_prefill<dp, dvp>((const bf16*)q, q_stride, (const bf16*)kpages, (const bf16*)vpages, block_table, \
                                       max_pages, kv_lens, cu_seqlens, (bf16*)out, out_stride, num_seqs, num_work, nq, nkv, \
                                       D, DV, ps, scale, chunk, skip_single, turns, pairs, pairing, sinks, stream)
  Q3_CHUNK_SIZES(Q3_CHUNK_PREFILL)
#undef Q3_CHUNK_PREFILL
}

// One token per sequence: those of seq_list (or all, when it is null).  splits: the most slices a sequence's visible
// keys are cut into; with more than one, mid_o holds num_seqs * nq * splits * DVP floats (DVP: DV rounded up to 64, 128
// or 256), mid_lse num_seqs * nq * splits, and tickets num_seqs * nkv ints that are zero before the call and after it.
Q3_EXPORT int q3_chunk_attention_decode(const void* q, int q_stride, const void* kpages, const void* vpages,
                                        const int* block_table, int max_pages, const int* kv_lens, const int* cu_seqlens,
                                        const int* seq_list, void* out, long out_stride, float* mid_o, float* mid_lse,
                                        int* tickets, int num_seqs, int nq, int nkv, int D, int DV, int ps, float scale,
                                        int chunk, int splits, const float* turns, int pairs, int pairing,
                                        const float* sinks, cudaStream_t stream) {
  if (!q || !kpages || !vpages || !block_table || !kv_lens || !cu_seqlens || !out) return Q3_ERR_ARGUMENT;
  if (nq < 1 || nkv < 1 || nq % nkv || ps < 1 || num_seqs < 0 || splits < 1 || chunk < 0) return Q3_ERR_ARGUMENT;
  if (splits > 1 && (!mid_o || !mid_lse || !tickets)) return Q3_ERR_ARGUMENT;
  if (turns && (pairs < 1 || 2 * pairs > DV || pairing < 0 || pairing > 1)) return Q3_ERR_ARGUMENT;
  if (num_seqs > 65535 || !chunk_sizes_ok(q, q_stride, kpages, vpages, out, out_stride, nq, nkv, D, DV))
    return Q3_ERR_UNSUPPORTED;
  if (num_seqs == 0) return Q3_OK;
#define Q3_CHUNK_DECODE(dp, dvp)                                                                                      \
  return launch_chunk_decode<dp, dvp>((const bf16*)q, q_stride, (const bf16*)kpages, (const bf16*)vpages, block_table, \
                                      max_pages, kv_lens, cu_seqlens, seq_list, (bf16*)out, out_stride, mid_o, mid_lse, \
                                      tickets, num_seqs, nq, nkv, D, DV, ps, scale, chunk, splits, turns, pairs, pairing, \
                                      sinks, stream)
  Q3_CHUNK_SIZES(Q3_CHUNK_DECODE)
#undef Q3_CHUNK_DECODE
}
