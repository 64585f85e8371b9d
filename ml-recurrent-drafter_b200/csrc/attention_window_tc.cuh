// Masked attention on warp-level tensor cores (bf16; query/key size <= DQ, value size <= DV, multiples of 8).
//
//   prefill  one CTA = 128 queries of one (row, head), 16 per warp; K/V tiles of 64 keys stream through a three-stage
//            cp.async ring.  Only the tiles that hold a kept token or lie in some query's window are visited.
//   decode   few new tokens per row: the query heads of one key/value head and their tokens share a tile of 16 query
//            rows, so K and V are read once per key/value head; a cluster of CTAs shares the key tiles and merges its
//            partial results through distributed shared memory.
#pragma once
#include <cooperative_groups.h>

#include "attention_window.cuh"
#include "mma_sync.cuh"

namespace rd_win {

using namespace rd_mma;
namespace cg = cooperative_groups;

constexpr int kBN = 64;  // keys per tile
constexpr float kLog2e = 1.4426950408889634f;

template <int CH>
__device__ __forceinline__ int swz(int r, int c) {
  return r * (CH * 16) + ((c ^ (r & 7)) << 4);
}

// 64 rows [row0, row0 + 64) of a matrix with `dim` features and rows ld apart into a tile of D features, the features from
// dim - tail_dim on from a second matrix; rows >= row_end and features >= dim are zero (row row_end - 1 stands in as address)
template <int D, int THREADS>
__device__ __forceinline__ void load_tile(uint8_t* dst, const __nv_bfloat16* src_base, int64_t ld, int dim, int row0, int row_end, int tid,
                                          const __nv_bfloat16* tail = nullptr, int64_t ld_tail = 0, int tail_dim = 0) {
  constexpr int CH = D / 8;
#pragma unroll
  for (int i = 0; i < (kBN * CH) / THREADS; ++i) {
    const int idx = i * THREADS + tid;
    const int r = idx / CH, c = idx % CH;
    const bool in = row0 + r < row_end && c * 8 < dim;
    const int64_t row = in ? row0 + r : row_end - 1;
    const int d = in ? c * 8 : 0;
    const __nv_bfloat16* src = d < dim - tail_dim ? src_base + row * ld + d : tail + row * ld_tail + (d - (dim - tail_dim));
    cp_async16(dst + swz<CH>(r, c), src, in);
  }
}

// Key tiles that some query with positions p_first .. sees: the tiles of the kept tokens, then [first, n).
struct TileRange {
  int kept, first, n;
  __device__ __forceinline__ void init(int lo, int keep_first, int kv_end) {
    n = (kv_end + kBN - 1) / kBN;
    first = lo > 0 ? lo / kBN : 0;
    if (first > n) first = n;
    kept = (min(keep_first, kv_end) + kBN - 1) / kBN;
    if (kept > first) kept = first;
  }
  __device__ __forceinline__ int count() const { return kept + n - first; }
  __device__ __forceinline__ int tile(int t) const { return t < kept ? t : first + t - kept; }
};

// ------------------------------------------------------------------------------------------------ prefill
constexpr int kBM = 128;
constexpr int kPrefillThreads = 256;
constexpr int kStages = 3;

template <int DQ, int DV>
struct PrefillSmem {
  static constexpr int kQ = kBM * DQ * 2, kK = kBN * DQ * 2, kV = kBN * DV * 2;
  static constexpr int kBytes = kQ + kStages * (kK + kV);
};

template <int DQ, int DV>
__global__ void __launch_bounds__(kPrefillThreads) attention_window_prefill_kernel(const Args a) {
  using Y = PrefillSmem<DQ, DV>;
  rd::pdl_launch_dependents();
  rd::pdl_wait();
  const int b = blockIdx.z, h = blockIdx.y;
  const int rs = a.row_start[b];
  const int n_new = a.row_start[b + 1] - rs;
  const int q0 = blockIdx.x * kBM;
  if (q0 >= n_new) return;
  extern __shared__ __align__(128) uint8_t smem[];
  uint8_t* sQ = smem;
  uint8_t* sKV = smem + Y::kQ;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int g = lane >> 2, t4 = lane & 3;
  const int base = a.base_len[b];
  const bool tree = a.mode == RD_ATTN_TREE;
  const int p_first = tree ? base : base + q0;                           // smallest position of a query of this CTA
  const int p_last = tree ? base + RD_MAX_BEAM_LENGTH - 1 : base + min(n_new, q0 + kBM) - 1;
  const int kv_end = tree ? base + n_new : p_last + 1;
  TileRange tiles;
  tiles.init(first_visible(a.mask_kind, a.window, p_first), a.keep_first, kv_end);
  const int n_tiles = tiles.count();
  const int hk = h / (a.nh / a.nkv);
  RowKeys<__nv_bfloat16> keys;
  keys.init(a, b, hk);
  constexpr int CQ = DQ / 8, CV = DV / 8;
  for (int idx = tid; idx < kBM * CQ; idx += kPrefillThreads) {
    const int r = idx / CQ, c = idx % CQ;
    const bool in = q0 + r < n_new && c * 8 < a.dim;
    cp_async16(sQ + swz<CQ>(r, c),
               (const __nv_bfloat16*)a.q + (int64_t)(rs + (in ? q0 + r : 0)) * a.ldq + (int64_t)h * a.dim + (in ? c * 8 : 0), in);
  }
  auto load = [&](int t) {
    if (t < n_tiles) {
      uint8_t* dst = sKV + (t % kStages) * (Y::kK + Y::kV);
      load_tile<DQ, kPrefillThreads>(dst, keys.k, a.k_row, a.dim, tiles.tile(t) * kBN, kv_end, tid, keys.tail, a.tail_row, a.tail_dim);
      load_tile<DV, kPrefillThreads>(dst + Y::kK, keys.v, a.v_row, a.vdim, tiles.tile(t) * kBN, kv_end, tid);
    }
    cp_async_commit();  // one group per tile, empty or not
  };
  load(0);
  load(1);

  uint32_t qf[DQ / 16][4];
  float o[DV / 8][4];
#pragma unroll
  for (int i = 0; i < DV / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.f, 0.f};
  Query qu[2];  // this thread's two query rows
#pragma unroll
  for (int hh = 0; hh < 2; ++hh) qu[hh].init(a, base, rs, n_new, min(q0 + warp * 16 + g + hh * 8, n_new - 1));
  const float scale_log2 = a.scale * kLog2e;
  const int first_last = first_visible(a.mask_kind, a.window, p_last);

  for (int it = 0; it < n_tiles; ++it) {
    cp_async_wait<1>();
    __syncthreads();
    load(it + 2);
    if (it == 0) {
#pragma unroll
      for (int kd = 0; kd < DQ / 16; ++kd)
        ldmatrix_x4(qf[kd][0], qf[kd][1], qf[kd][2], qf[kd][3],
                    smem_addr(sQ + swz<CQ>(warp * 16 + (lane & 15), kd * 2 + (lane >> 4))));
    }
    const uint8_t* sK = sKV + (it % kStages) * (Y::kK + Y::kV);
    const uint8_t* sV = sK + Y::kK;
    float s[kBN / 8][4];
#pragma unroll
    for (int nb = 0; nb < kBN / 8; ++nb) s[nb][0] = s[nb][1] = s[nb][2] = s[nb][3] = 0.f;
#pragma unroll
    for (int kd = 0; kd < DQ / 16; ++kd) {
#pragma unroll
      for (int nb = 0; nb < kBN / 8; nb += 2) {
        uint32_t b0, b1, b2, b3;
        ldmatrix_x4(b0, b1, b2, b3, smem_addr(sK + swz<CQ>(nb * 8 + ((lane >> 4) << 3) + (lane & 7), kd * 2 + ((lane >> 3) & 1))));
        mma_bf16(s[nb], qf[kd], b0, b1);
        mma_bf16(s[nb + 1], qf[kd], b2, b3);
      }
    }
    const int j0 = tiles.tile(it) * kBN, j_last = j0 + kBN - 1;
    // a tile that every query of the CTA sees in full needs no mask
    const bool open = j_last <= p_first && j_last < kv_end && (!tree || j_last < base) &&
                      (j0 >= first_last || j_last < a.keep_first);
    float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
    for (int nb = 0; nb < kBN / 8; ++nb)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        float v = s[nb][e] * scale_log2;
        if (!open && !qu[e >> 1].sees(a, j0 + nb * 8 + t4 * 2 + (e & 1))) v = -INFINITY;
        s[nb][e] = v;
        mx[e >> 1] = fmaxf(mx[e >> 1], v);
      }
    float alpha[2], m_use[2];
#pragma unroll
    for (int hh = 0; hh < 2; ++hh) {
      mx[hh] = fmaxf(mx[hh], __shfl_xor_sync(0xffffffffu, mx[hh], 1));
      mx[hh] = fmaxf(mx[hh], __shfl_xor_sync(0xffffffffu, mx[hh], 2));
      const float m_new = fmaxf(m_run[hh], mx[hh]);
      m_use[hh] = m_new == -INFINITY ? 0.f : m_new;
      alpha[hh] = m_run[hh] == -INFINITY ? 0.f : exp2f(m_run[hh] - m_use[hh]);
      m_run[hh] = m_new;
    }
    float sum[2] = {0.f, 0.f};
    uint32_t pf[kBN / 16][4];
#pragma unroll
    for (int nb = 0; nb < kBN / 8; ++nb) {
      const float p0 = exp2f(s[nb][0] - m_use[0]), p1 = exp2f(s[nb][1] - m_use[0]);
      const float p2 = exp2f(s[nb][2] - m_use[1]), p3 = exp2f(s[nb][3] - m_use[1]);
      sum[0] += p0 + p1;
      sum[1] += p2 + p3;
      pf[nb >> 1][(nb & 1) * 2] = pack_bf16(p0, p1);
      pf[nb >> 1][(nb & 1) * 2 + 1] = pack_bf16(p2, p3);
    }
#pragma unroll
    for (int hh = 0; hh < 2; ++hh) l_run[hh] = l_run[hh] * alpha[hh] + sum[hh];
#pragma unroll
    for (int db = 0; db < DV / 8; ++db) {
      o[db][0] *= alpha[0];
      o[db][1] *= alpha[0];
      o[db][2] *= alpha[1];
      o[db][3] *= alpha[1];
    }
#pragma unroll
    for (int kk = 0; kk < kBN / 16; ++kk) {
#pragma unroll
      for (int db = 0; db < DV / 8; db += 2) {
        uint32_t b0, b1, b2, b3;
        ldmatrix_x4_trans(b0, b1, b2, b3, smem_addr(sV + swz<CV>(kk * 16 + (((lane >> 3) & 1) << 3) + (lane & 7), db + (lane >> 4))));
        mma_bf16(o[db], pf[kk], b0, b1);
        mma_bf16(o[db + 1], pf[kk], b2, b3);
      }
    }
  }
  cp_async_wait<0>();
#pragma unroll
  for (int hh = 0; hh < 2; ++hh) {
    l_run[hh] += __shfl_xor_sync(0xffffffffu, l_run[hh], 1);
    l_run[hh] += __shfl_xor_sync(0xffffffffu, l_run[hh], 2);
    const int i = q0 + warp * 16 + g + hh * 8;
    if (i < n_new) {
      float f = finish_softmax(m_run[hh], l_run[hh], a.sink, h);
      if (a.gate != nullptr) f *= sigmoid_exact(__bfloat162float(((const __nv_bfloat16*)a.gate)[(int64_t)(rs + i) * a.ld_gate + h]));
      __nv_bfloat16* dst = (__nv_bfloat16*)a.out + ((int64_t)(rs + i) * a.nh + h) * a.vdim;
#pragma unroll
      for (int db = 0; db < DV / 8; ++db)
        if (db * 8 < a.vdim) *reinterpret_cast<uint32_t*>(dst + db * 8 + t4 * 2) = pack_bf16(o[db][hh * 2] * f, o[db][hh * 2 + 1] * f);
    }
  }
}

// ------------------------------------------------------------------------------------------------ decode
constexpr int kDecodeThreads = 128;  // four warps: each takes 16 of a tile's 64 keys
constexpr int kDecodeStages = 3;
constexpr int kRows = 16;            // query rows (head of the group, new token) per CTA

template <int DQ, int DV>
struct DecodeSmem {
  static constexpr int kQ = kRows * DQ * 2, kK = kBN * DQ * 2, kV = kBN * DV * 2;
  static constexpr int kOld = DV + 4;                        // floats per partial output row
  static constexpr int kPart = 4 * kRows * kOld * 4;         // one partial per warp, over the K/V ring
  static constexpr int kRing = kDecodeStages * (kK + kV);
  static constexpr int kMl = 4 * kRows * 2 * 4;              // running max and sum of every warp's rows
  static constexpr int kCta = kRows * (kOld + 2) * 4;        // the CTA's merged partial
  static constexpr int kBytes = kQ + (kRing > kPart ? kRing : kPart) + kMl + kCta;
};

// grid (cluster, nkv * row tiles, B); cluster (n_split, 1, 1)
template <int DQ, int DV>
__global__ void __launch_bounds__(kDecodeThreads) attention_window_decode_kernel(const Args a) {
  using Y = DecodeSmem<DQ, DV>;
  cg::cluster_group cluster = cg::this_cluster();
  rd::pdl_launch_dependents();
  rd::pdl_wait();
  const int b = blockIdx.z;
  const int group = a.nh / a.nkv;
  const int hk = blockIdx.y % a.nkv, row_tile = blockIdx.y / a.nkv;
  const int rank = (int)cluster.block_rank(), n_ranks = (int)cluster.num_blocks();
  const int rs = a.row_start[b];
  const int n_new = a.row_start[b + 1] - rs;
  const int n_rows = group * n_new - row_tile * kRows;  // rows of this tile and after
  if (n_rows <= 0) return;                              // the same for the whole cluster
  extern __shared__ __align__(128) uint8_t smem[];
  uint8_t* sQ = smem;
  uint8_t* ring = smem + Y::kQ;
  float* part_o = reinterpret_cast<float*>(ring);  // [4][kRows][kOld], after the ring's last use
  float* part_ml = reinterpret_cast<float*>(smem + Y::kQ + (Y::kRing > Y::kPart ? Y::kRing : Y::kPart));  // [4][kRows][2]
  float* cta_o = part_ml + 4 * kRows * 2;          // [kRows][kOld]
  float* cta_ml = cta_o + kRows * Y::kOld;         // [kRows][2]
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int g = lane >> 2, t4 = lane & 3;
  const int base = a.base_len[b];
  // row r of the tile: head hk * group + (row / n_new), new token row % n_new, row = row_tile * 16 + r
  auto head_of = [&](int r) { return hk * group + (row_tile * kRows + r) / n_new; };
  auto tok_of = [&](int r) { return (row_tile * kRows + r) % n_new; };
  const int kv_end = base + n_new;
  TileRange tiles;
  tiles.init(first_visible(a.mask_kind, a.window, base), a.keep_first, kv_end);  // no query sits before position base
  const int n_all = tiles.count();
  const int per = (n_all + n_ranks - 1) / n_ranks;
  const int t_begin = min(rank * per, n_all), n_tiles = min(per, n_all - t_begin);
  RowKeys<__nv_bfloat16> keys;
  keys.init(a, b, hk);
  constexpr int CQ = DQ / 8, CV = DV / 8;
  for (int idx = tid; idx < kRows * CQ; idx += kDecodeThreads) {
    const int r = idx / CQ, c = idx % CQ;
    const bool in = r < n_rows && c * 8 < a.dim;
    const __nv_bfloat16* src = (const __nv_bfloat16*)a.q;
    if (in) src += (int64_t)(rs + tok_of(r)) * a.ldq + (int64_t)head_of(r) * a.dim + c * 8;
    cp_async16(sQ + swz<CQ>(r, c), src, in);
  }
  auto load = [&](int t) {
    if (t < n_tiles) {
      uint8_t* dst = ring + (t % kDecodeStages) * (Y::kK + Y::kV);
      const int j0 = tiles.tile(t_begin + t) * kBN;
      load_tile<DQ, kDecodeThreads>(dst, keys.k, a.k_row, a.dim, j0, kv_end, tid, keys.tail, a.tail_row, a.tail_dim);
      load_tile<DV, kDecodeThreads>(dst + Y::kK, keys.v, a.v_row, a.vdim, j0, kv_end, tid);
    }
    cp_async_commit();
  };
  load(0);
  load(1);
  float o[DV / 8][4];
#pragma unroll
  for (int i = 0; i < DV / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.f, 0.f};
  Query qu[2];
#pragma unroll
  for (int hh = 0; hh < 2; ++hh) qu[hh].init(a, base, rs, n_new, tok_of(min(g + hh * 8, n_rows - 1)));
  const float scale_log2 = a.scale * kLog2e;
  for (int it = 0; it < n_tiles; ++it) {
    cp_async_wait<1>();
    __syncthreads();
    load(it + 2);
    const uint8_t* sK = ring + (it % kDecodeStages) * (Y::kK + Y::kV);
    const uint8_t* sV = sK + Y::kK;
    const int k0 = warp * 16;  // this warp's keys of the tile
    float s[2][4] = {};
#pragma unroll
    for (int kd = 0; kd < DQ / 16; ++kd) {
      uint32_t af[4], b0, b1, b2, b3;
      ldmatrix_x4(af[0], af[1], af[2], af[3], smem_addr(sQ + swz<CQ>(lane & 15, kd * 2 + (lane >> 4))));
      ldmatrix_x4(b0, b1, b2, b3, smem_addr(sK + swz<CQ>(k0 + ((lane >> 4) << 3) + (lane & 7), kd * 2 + ((lane >> 3) & 1))));
      mma_bf16(s[0], af, b0, b1);
      mma_bf16(s[1], af, b2, b3);
    }
    const int j0 = tiles.tile(t_begin + it) * kBN + k0;
    float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
    for (int nb = 0; nb < 2; ++nb)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float v = qu[e >> 1].sees(a, j0 + nb * 8 + t4 * 2 + (e & 1)) ? s[nb][e] * scale_log2 : -INFINITY;
        s[nb][e] = v;
        mx[e >> 1] = fmaxf(mx[e >> 1], v);
      }
    float alpha[2], m_use[2];
#pragma unroll
    for (int hh = 0; hh < 2; ++hh) {
      mx[hh] = fmaxf(mx[hh], __shfl_xor_sync(0xffffffffu, mx[hh], 1));
      mx[hh] = fmaxf(mx[hh], __shfl_xor_sync(0xffffffffu, mx[hh], 2));
      const float m_new = fmaxf(m_run[hh], mx[hh]);
      m_use[hh] = m_new == -INFINITY ? 0.f : m_new;
      alpha[hh] = m_run[hh] == -INFINITY ? 0.f : exp2f(m_run[hh] - m_use[hh]);
      m_run[hh] = m_new;
    }
    float p[2][4];
#pragma unroll
    for (int nb = 0; nb < 2; ++nb)
#pragma unroll
      for (int e = 0; e < 4; ++e) p[nb][e] = exp2f(s[nb][e] - m_use[e >> 1]);
    l_run[0] = l_run[0] * alpha[0] + p[0][0] + p[0][1] + p[1][0] + p[1][1];
    l_run[1] = l_run[1] * alpha[1] + p[0][2] + p[0][3] + p[1][2] + p[1][3];
    const uint32_t pf[4] = {pack_bf16(p[0][0], p[0][1]), pack_bf16(p[0][2], p[0][3]), pack_bf16(p[1][0], p[1][1]),
                            pack_bf16(p[1][2], p[1][3])};
#pragma unroll
    for (int db = 0; db < DV / 8; db += 2) {
      uint32_t b0, b1, b2, b3;
      ldmatrix_x4_trans(b0, b1, b2, b3, smem_addr(sV + swz<CV>(k0 + (((lane >> 3) & 1) << 3) + (lane & 7), db + (lane >> 4))));
#pragma unroll
      for (int q = 0; q < 2; ++q) {
        o[db + q][0] *= alpha[0];
        o[db + q][1] *= alpha[0];
        o[db + q][2] *= alpha[1];
        o[db + q][3] *= alpha[1];
      }
      mma_bf16(o[db], pf, b0, b1);
      mma_bf16(o[db + 1], pf, b2, b3);
    }
  }
  cp_async_wait<0>();
  __syncthreads();  // the ring becomes the warps' partials
#pragma unroll
  for (int hh = 0; hh < 2; ++hh) {
    l_run[hh] += __shfl_xor_sync(0xffffffffu, l_run[hh], 1);
    l_run[hh] += __shfl_xor_sync(0xffffffffu, l_run[hh], 2);
    float* dst = part_o + (warp * kRows + g + hh * 8) * Y::kOld;
#pragma unroll
    for (int db = 0; db < DV / 8; ++db) *reinterpret_cast<float2*>(dst + db * 8 + t4 * 2) = make_float2(o[db][hh * 2], o[db][hh * 2 + 1]);
    if (t4 == 0) {
      part_ml[(warp * kRows + g + hh * 8) * 2] = m_run[hh];
      part_ml[(warp * kRows + g + hh * 8) * 2 + 1] = l_run[hh];
    }
  }
  __syncthreads();
  for (int idx = tid; idx < kRows * DV; idx += kDecodeThreads) {
    const int r = idx / DV, d = idx % DV;
    float m = -INFINITY;
#pragma unroll
    for (int w = 0; w < 4; ++w) m = fmaxf(m, part_ml[(w * kRows + r) * 2]);
    float acc = 0.f, l = 0.f;
#pragma unroll
    for (int w = 0; w < 4; ++w) {
      const float mw = part_ml[(w * kRows + r) * 2];
      const float f = mw == -INFINITY ? 0.f : exp2f(mw - m);
      acc = fmaf(f, part_o[(w * kRows + r) * Y::kOld + d], acc);
      l = fmaf(f, part_ml[(w * kRows + r) * 2 + 1], l);
    }
    cta_o[r * Y::kOld + d] = acc;
    if (d == 0) {
      cta_ml[r * 2] = m;
      cta_ml[r * 2 + 1] = l;
    }
  }
  cluster.sync();
  // the ranks share the rows of the output
  for (int idx = rank * kDecodeThreads + tid; idx < min(n_rows, kRows) * DV; idx += n_ranks * kDecodeThreads) {
    const int r = idx / DV, d = idx % DV;
    if (d >= a.vdim) continue;
    float m = -INFINITY;
    for (int k = 0; k < n_ranks; ++k) m = fmaxf(m, cluster.map_shared_rank(cta_ml, k)[r * 2]);
    float acc = 0.f, l = 0.f;
    for (int k = 0; k < n_ranks; ++k) {
      const float* ml = cluster.map_shared_rank(cta_ml, k);
      const float f = ml[r * 2] == -INFINITY ? 0.f : exp2f(ml[r * 2] - m);
      acc = fmaf(f, cluster.map_shared_rank(cta_o, k)[r * Y::kOld + d], acc);
      l = fmaf(f, ml[r * 2 + 1], l);
    }
    const int t = rs + tok_of(r), h = head_of(r);
    float f = finish_softmax(m, l, a.sink, h);
    if (a.gate != nullptr) f *= sigmoid_exact(__bfloat162float(((const __nv_bfloat16*)a.gate)[(int64_t)t * a.ld_gate + h]));
    ((__nv_bfloat16*)a.out)[((int64_t)t * a.nh + h) * a.vdim + d] = __float2bfloat16_rn(acc * f);
  }
  cluster.sync();  // peers have read this CTA's partial
}

template <int DQ, int DV>
int launch_prefill(const Args& a, cudaStream_t s) {
  auto kern = attention_window_prefill_kernel<DQ, DV>;
  constexpr int smem = PrefillSmem<DQ, DV>::kBytes;
  static bool set = false;
  if (!set) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    RD_CHECK_CHAINED(e);
    set = true;
  }
  cudaError_t err = rd::launch_chained(kern, dim3((a.max_new + kBM - 1) / kBM, a.nh, a.B), dim3(kPrefillThreads), smem, s, 1, a);
  RD_CHECK_CHAINED(err);
  return RD_OK;
}

template <int DQ, int DV>
int launch_decode(const Args& a, cudaStream_t s) {
  auto kern = attention_window_decode_kernel<DQ, DV>;
  constexpr int smem = DecodeSmem<DQ, DV>::kBytes;
  static bool set = false;
  if (!set) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    RD_CHECK_CHAINED(e);
    set = true;
  }
  const int row_tiles = ((a.nh / a.nkv) * a.max_new + kRows - 1) / kRows;
  // a cluster's CTAs share the key tiles of a row: enough of them to fill the GPU twice, at least two tiles each
  const int64_t visible = (int64_t)a.window + a.max_new + a.keep_first + 2 * kBN;
  const int tiles = (int)((visible < a.max_kv ? visible : a.max_kv) + kBN - 1) / kBN;
  int ranks = 1;
  while (ranks < 8 && (int64_t)a.B * a.nkv * row_tiles * ranks < 2 * 148 && tiles / (ranks * 2) >= 2) ranks *= 2;
  cudaError_t err = rd::launch_chained(kern, dim3(ranks, a.nkv * row_tiles, a.B), dim3(kDecodeThreads), smem, s, ranks, a);
  RD_CHECK_CHAINED(err);
  return RD_OK;
}

}  // namespace rd_win
