// Masked attention where all heads share one key and the values are the first part of that key (latent attention with the
// up-projections of keys and values moved to the queries and the output), bf16, warp-level tensor cores fed by TMA.
//
// One CTA serves 16 * MT query rows (token, head) of one batch row; a key tile of 64 is read once for scores and values and
// for all of them.  One thread requests queries and key tiles (boxes of 64 features, 128-byte swizzle) ahead of their use;
// eight warps each take a share of the tile's keys for the scores, then their own eighth of the value columns for all rows
// (row maxima and the weights travel through shared memory).  A cluster of CTAs shares the key tiles and merges its
// partial results through distributed shared memory.  Barrier waits are bounded: on give-up the CTA records a code in
// *status, lets its copies land and leaves through the same cluster barriers.
#include "attention_window_tc.cuh"
#include "umma.cuh"

namespace {

using namespace rd_win;
using rd_umma::mbar_expect_tx;
using rd_umma::mbar_init;
using rd_umma::mbar_wait;
using rd_umma::tma_load_2d;

constexpr int kLatThreads = 256;
constexpr int kLatWarps = kLatThreads / 32;
constexpr int kMaxRanks = 8;

struct LatentPlan {
  CUtensorMap map_q;  // [query rows, dim] box 64 x 16
  CUtensorMap map_k;  // [cache rows, dim] box 64 x 64
  int dim;
};

// 16 bytes of feature chunk c (eight features) of row r in a column of boxes of `rows` rows
template <int rows>
__device__ __forceinline__ int boxed(int r, int c) {
  return (c >> 3) * (rows * 128) + r * 128 + (((c & 7) ^ (r & 7)) << 4);
}

template <int DK, int DV, int MT>
struct LatentSmem {
  static constexpr int kR = 16 * MT;                   // query rows per CTA
  static constexpr int kKG = kLatWarps / MT;           // groups of keys of a tile
  static constexpr int kStages = DK > 320 ? 2 : 3;
  static constexpr int kQ = kR * DK * 2, kK = kBN * DK * 2;
  static constexpr int kRing = kStages * kK;
  static constexpr int kOld = DV + 4;                  // floats per partial output row, over the key ring
  static constexpr int kP = kR * kBN * 2;
  static constexpr int kRed = 2 * kKG * kR * 4;        // row maxima and sums of every key group
  static constexpr int kMl = kR * 2 * 4;
  static constexpr int kWeights = kMaxRanks * kR * 4;  // what every rank's partial counts in the result
  static constexpr int kBytes = kQ + kRing + kP + kRed + kMl + kWeights + 64;  // and the barriers
  static_assert(kR * kOld * 4 <= kRing, "the partial output lies over the key ring");
};

// grid (cluster, row tiles, B); cluster (n_split, 1, 1)
template <int DK, int DV, int MT>
__global__ void __launch_bounds__(kLatThreads)
    attention_latent_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k, const Args a, int32_t* status) {
  using Y = LatentSmem<DK, DV, MT>;
  constexpr int R = Y::kR, KG = Y::kKG, ST = Y::kStages;
  constexpr int NB = DV / (8 * kLatWarps);  // 8-column blocks of values per warp
  cg::cluster_group cluster = cg::this_cluster();
  rd::pdl_launch_dependents();
  extern __shared__ __align__(1024) uint8_t smem[];  // the swizzled boxes start at multiples of 1024
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + Y::kBytes - 64);
  uint64_t* q_full = bars;
  uint64_t* k_full = bars + 1;  // [ST]
  if (threadIdx.x == 0) {
    asm volatile("prefetch.tensormap [%0];" ::"l"(&map_q) : "memory");
    asm volatile("prefetch.tensormap [%0];" ::"l"(&map_k) : "memory");
    for (int i = 0; i < 1 + ST; ++i) mbar_init(&bars[i], 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  rd::pdl_wait();
  const int b = blockIdx.z, row_first = blockIdx.y * R;
  const int rank = (int)cluster.block_rank(), n_ranks = (int)cluster.num_blocks();
  const int rs = a.row_start[b];
  const int n_new = a.row_start[b + 1] - rs;
  const int n_rows = min(R, a.nh * n_new - row_first);
  if (n_rows <= 0) return;  // the same for the whole cluster
  uint8_t* sQ = smem;
  uint8_t* ring = smem + Y::kQ;
  float* cta_o = reinterpret_cast<float*>(ring);  // [R][kOld], after the ring's last use
  uint8_t* sP = ring + Y::kRing;
  float* red_m = reinterpret_cast<float*>(sP + Y::kP);  // [KG][R]
  float* red_l = red_m + KG * R;                        // [KG][R]
  float* cta_ml = red_l + KG * R;                       // [R][2]
  float* weight = cta_ml + R * 2;                       // [kMaxRanks][R]
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int g = lane >> 2, t4 = lane & 3;
  const int mt_s = warp % MT, kg = warp / MT, k0 = kg * 8 * MT;  // this warp's rows and keys of a score tile
  const int base = a.base_len[b];
  const int tok_first = row_first / a.nh, tok_last = (row_first + n_rows - 1) / a.nh;
  const bool tree = a.mode == RD_ATTN_TREE;
  const int kv_end = tree ? base + n_new : base + tok_last + 1;
  TileRange tiles;
  tiles.init(first_visible(a.mask_kind, a.window, tree ? base : base + tok_first), a.keep_first, kv_end);
  const int n_all = tiles.count();
  const int per = (n_all + n_ranks - 1) / n_ranks;
  const int t_begin = min(rank * per, n_all), n_tiles = min(per, n_all - t_begin);
  const int key_row0 = b * (int)(a.k_batch / a.k_row) + a.kv_begin[b];  // matrix row of key 0
  // by thread 0; a tile's rows past kv_end hold other keys of the cache, which the mask hides
  auto load = [&](int t) {
    if (t < n_tiles) {
      mbar_expect_tx(&k_full[t % ST], Y::kK);
      const int row = key_row0 + tiles.tile(t_begin + t) * kBN;
#pragma unroll
      for (int i = 0; i < DK / 64; ++i) tma_load_2d(ring + (t % ST) * Y::kK + i * (kBN * 128), &map_k, &k_full[t % ST], i * 64, row);
    }
  };
  if (tid == 0) {
    if (n_tiles > 0) {
      mbar_expect_tx(q_full, Y::kQ);
#pragma unroll
      for (int i = 0; i < DK / 64; ++i)
#pragma unroll
        for (int mt = 0; mt < MT; ++mt)
          tma_load_2d(sQ + i * (R * 128) + mt * 2048, &map_q, q_full, i * 64, rs * a.nh + row_first + mt * 16);
    }
    for (int t = 0; t < ST - 1; ++t) load(t);
  }
  __syncthreads();  // the barriers exist
  float o[MT][NB][4];
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int i = 0; i < NB; ++i) o[mt][i][0] = o[mt][i][1] = o[mt][i][2] = o[mt][i][3] = 0.f;
  float m_run[MT][2], l_run[2] = {0.f, 0.f};
#pragma unroll
  for (int mt = 0; mt < MT; ++mt) m_run[mt][0] = m_run[mt][1] = -INFINITY;
  Query qu[2];  // this thread's two rows of the score tile
#pragma unroll
  for (int hh = 0; hh < 2; ++hh) qu[hh].init(a, base, rs, n_new, (row_first + min(mt_s * 16 + g + hh * 8, n_rows - 1)) / a.nh);
  const float scale_log2 = a.scale * kLog2e;
  const int p_first = tree ? base : base + tok_first;                      // positions of the rows lie in
  const int p_last = tree ? base + RD_MAX_BEAM_LENGTH - 1 : base + tok_last;  // [p_first, p_last]
  const int first_last = first_visible(a.mask_kind, a.window, p_last);
  // this thread's places in a box: row and swizzle of the Q rows and of the keys it loads
  const int q_row = mt_s * 16 + (lane & 15);
  const int k_row = MT == 1 ? k0 + (lane & 7) : k0 + ((lane >> 4) << 3) + (lane & 7);
  const uint32_t q_addr = smem_addr(sQ) + q_row * 128;
  bool ok = n_tiles == 0 || mbar_wait(q_full, 0);
  for (int it = 0; it < n_tiles; ++it) {
    ok = ok && mbar_wait(&k_full[it % ST], (it / ST) & 1);
    if (__syncthreads_or(!ok)) {  // every warp is done with the stage that is requested next
      ok = false;
      break;
    }
    if (tid == 0) load(it + ST - 1);
    const uint8_t* sK = ring + (it % ST) * Y::kK;
    const uint32_t k_addr = smem_addr(sK) + k_row * 128;
    float s2[2][MT][4] = {};  // even and odd steps along the features
#pragma unroll 6
    for (int kd = 0; kd < DK / 16; kd += 2) {
      const uint32_t qb = q_addr + (kd >> 2) * (R * 128), kb = k_addr + (kd >> 2) * (kBN * 128);
      const int c0 = (kd & 3) * 2;
      uint32_t a0[4], a1[4];
      ldmatrix_x4(a0[0], a0[1], a0[2], a0[3], qb + (((c0 + (lane >> 4)) ^ (q_row & 7)) << 4));
      ldmatrix_x4(a1[0], a1[1], a1[2], a1[3], qb + (((c0 + 2 + (lane >> 4)) ^ (q_row & 7)) << 4));
      uint32_t b0, b1, b2, b3;
      if constexpr (MT == 1) {
        ldmatrix_x4(b0, b1, b2, b3, kb + (((c0 + (lane >> 3)) ^ (k_row & 7)) << 4));
        mma_bf16(s2[0][0], a0, b0, b1);
        mma_bf16(s2[1][0], a1, b2, b3);
      } else {
        ldmatrix_x4(b0, b1, b2, b3, kb + (((c0 + ((lane >> 3) & 1)) ^ (k_row & 7)) << 4));
        mma_bf16(s2[0][0], a0, b0, b1);
        mma_bf16(s2[0][MT - 1], a0, b2, b3);
        ldmatrix_x4(b0, b1, b2, b3, kb + (((c0 + 2 + ((lane >> 3) & 1)) ^ (k_row & 7)) << 4));
        mma_bf16(s2[1][0], a1, b0, b1);
        mma_bf16(s2[1][MT - 1], a1, b2, b3);
      }
    }
    const int j0 = tiles.tile(t_begin + it) * kBN + k0;
    // a tile that every row sees in full needs no mask
    const int tile0 = j0 - k0, tile_last = tile0 + kBN - 1;
    const bool open = tile_last <= p_first && tile_last < kv_end && (!tree || tile_last < base) &&
                      (tile0 >= first_last || tile_last < a.keep_first);
    float s[MT][4], mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
    for (int nb = 0; nb < MT; ++nb)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float v = open || qu[e >> 1].sees(a, j0 + nb * 8 + t4 * 2 + (e & 1)) ? (s2[0][nb][e] + s2[1][nb][e]) * scale_log2 : -INFINITY;
        s[nb][e] = v;
        mx[e >> 1] = fmaxf(mx[e >> 1], v);
      }
#pragma unroll
    for (int hh = 0; hh < 2; ++hh) {
      mx[hh] = fmaxf(mx[hh], __shfl_xor_sync(0xffffffffu, mx[hh], 1));
      mx[hh] = fmaxf(mx[hh], __shfl_xor_sync(0xffffffffu, mx[hh], 2));
      if (t4 == 0) red_m[kg * R + mt_s * 16 + g + hh * 8] = mx[hh];
    }
    __syncthreads();
    float alpha[MT][2], m_use[MT][2];
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int hh = 0; hh < 2; ++hh) {
        float m_new = m_run[mt][hh];
#pragma unroll
        for (int k = 0; k < KG; ++k) m_new = fmaxf(m_new, red_m[k * R + mt * 16 + g + hh * 8]);
        m_use[mt][hh] = m_new == -INFINITY ? 0.f : m_new;
        alpha[mt][hh] = m_run[mt][hh] == -INFINITY ? 0.f : exp2f(m_run[mt][hh] - m_use[mt][hh]);
        m_run[mt][hh] = m_new;
      }
    const float mu[2] = {MT == 1 || mt_s == 0 ? m_use[0][0] : m_use[MT - 1][0], MT == 1 || mt_s == 0 ? m_use[0][1] : m_use[MT - 1][1]};
    const float al[2] = {MT == 1 || mt_s == 0 ? alpha[0][0] : alpha[MT - 1][0], MT == 1 || mt_s == 0 ? alpha[0][1] : alpha[MT - 1][1]};
    l_run[0] *= al[0];
    l_run[1] *= al[1];
#pragma unroll
    for (int nb = 0; nb < MT; ++nb) {
      const float p0 = exp2f(s[nb][0] - mu[0]), p1 = exp2f(s[nb][1] - mu[0]);
      const float p2 = exp2f(s[nb][2] - mu[1]), p3 = exp2f(s[nb][3] - mu[1]);
      l_run[0] += p0 + p1;
      l_run[1] += p2 + p3;
      const int chunk = (k0 >> 3) + nb;
      *reinterpret_cast<uint32_t*>(sP + swz<8>(mt_s * 16 + g, chunk) + t4 * 4) = pack_bf16(p0, p1);
      *reinterpret_cast<uint32_t*>(sP + swz<8>(mt_s * 16 + g + 8, chunk) + t4 * 4) = pack_bf16(p2, p3);
    }
    __syncthreads();
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int db = 0; db < NB; ++db) {
        o[mt][db][0] *= alpha[mt][0];
        o[mt][db][1] *= alpha[mt][0];
        o[mt][db][2] *= alpha[mt][1];
        o[mt][db][3] *= alpha[mt][1];
      }
#pragma unroll
    for (int kk = 0; kk < kBN / 16; ++kk) {
      uint32_t pf[MT][4];
#pragma unroll
      for (int mt = 0; mt < MT; ++mt)
        ldmatrix_x4(pf[mt][0], pf[mt][1], pf[mt][2], pf[mt][3], smem_addr(sP + swz<8>(mt * 16 + (lane & 15), kk * 2 + (lane >> 4))));
#pragma unroll
      for (int db = 0; db < NB; db += 2) {
        uint32_t b0, b1, b2, b3;
        ldmatrix_x4_trans(b0, b1, b2, b3,
                          smem_addr(sK + boxed<kBN>(kk * 16 + (((lane >> 3) & 1) << 3) + (lane & 7), warp * NB + db + (lane >> 4))));
#pragma unroll
        for (int mt = 0; mt < MT; ++mt) {
          mma_bf16(o[mt][db], pf[mt], b0, b1);
          mma_bf16(o[mt][db + 1], pf[mt], b2, b3);
        }
      }
    }
  }
  if (!ok) {
    if (tid == 0) {
      if (status) atomicExch(status, 41);
      for (int i = 0; i < 2000; ++i) __nanosleep(1000);  // let copies in flight land
    }
  }
  __syncthreads();  // the ring becomes the CTA's partial
#pragma unroll
  for (int hh = 0; hh < 2; ++hh) {
    l_run[hh] += __shfl_xor_sync(0xffffffffu, l_run[hh], 1);
    l_run[hh] += __shfl_xor_sync(0xffffffffu, l_run[hh], 2);
    if (t4 == 0) red_l[kg * R + mt_s * 16 + g + hh * 8] = l_run[hh];
#pragma unroll
    for (int mt = 0; mt < MT; ++mt) {
      float* dst = cta_o + (mt * 16 + g + hh * 8) * Y::kOld + warp * NB * 8 + t4 * 2;
#pragma unroll
      for (int db = 0; db < NB; ++db) *reinterpret_cast<float2*>(dst + db * 8) = make_float2(o[mt][db][hh * 2], o[mt][db][hh * 2 + 1]);
      if (warp == 0 && t4 == 0) cta_ml[(mt * 16 + g + hh * 8) * 2] = m_run[mt][hh];
    }
  }
  __syncthreads();
  if (tid < R) {
    float l = 0.f;
#pragma unroll
    for (int k = 0; k < KG; ++k) l += red_l[k * R + tid];
    cta_ml[tid * 2 + 1] = l;
  }
  cluster.sync();
  // what each rank's partial counts in each row, the softmax's sum and the gate included
  if (tid < n_rows) {
    float mk[kMaxRanks], lk[kMaxRanks], m = -INFINITY, l = 0.f;
#pragma unroll
    for (int k = 0; k < kMaxRanks; ++k) {
      const float2 ml = k < n_ranks ? *reinterpret_cast<const float2*>(cluster.map_shared_rank(cta_ml, k) + tid * 2) : make_float2(-INFINITY, 0.f);
      mk[k] = ml.x, lk[k] = ml.y;
      m = fmaxf(m, ml.x);
    }
#pragma unroll
    for (int k = 0; k < kMaxRanks; ++k) {
      mk[k] = mk[k] == -INFINITY ? 0.f : exp2f(mk[k] - m);
      l = fmaf(mk[k], lk[k], l);
    }
    const int t = rs + (row_first + tid) / a.nh, h = (row_first + tid) % a.nh;
    float f = finish_softmax(m, l, a.sink, h);
    if (a.gate != nullptr) f *= sigmoid_exact(__bfloat162float(((const __nv_bfloat16*)a.gate)[(int64_t)t * a.ld_gate + h]));
#pragma unroll
    for (int k = 0; k < kMaxRanks; ++k) weight[k * R + tid] = mk[k] * f;
  }
  __syncthreads();
  // the ranks share the rows of the output, four values per thread
  for (int idx = rank * kLatThreads + tid; idx < n_rows * (DV / 4); idx += n_ranks * kLatThreads) {
    const int r = idx / (DV / 4), d = idx % (DV / 4) * 4;
    if (d >= a.vdim) continue;
    float4 part[kMaxRanks];
#pragma unroll
    for (int k = 0; k < kMaxRanks; ++k)
      if (k < n_ranks) part[k] = *reinterpret_cast<const float4*>(cluster.map_shared_rank(cta_o, k) + r * Y::kOld + d);
    float acc[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int k = 0; k < kMaxRanks; ++k)
      if (k < n_ranks) {
        const float w = weight[k * R + r];
        acc[0] = fmaf(w, part[k].x, acc[0]);
        acc[1] = fmaf(w, part[k].y, acc[1]);
        acc[2] = fmaf(w, part[k].z, acc[2]);
        acc[3] = fmaf(w, part[k].w, acc[3]);
      }
    __nv_bfloat16* dst = (__nv_bfloat16*)a.out + ((int64_t)(rs + (row_first + r) / a.nh) * a.nh + (row_first + r) % a.nh) * a.vdim + d;
    if (a.vdim % 4 == 0 && (reinterpret_cast<uintptr_t>(a.out) & 7) == 0) {
      *reinterpret_cast<uint2*>(dst) = make_uint2(pack_bf16(acc[0], acc[1]), pack_bf16(acc[2], acc[3]));
    } else {
#pragma unroll
      for (int e = 0; e < 4; ++e)
        if (d + e < a.vdim) dst[e] = __float2bfloat16_rn(acc[e]);
    }
  }
  cluster.sync();  // peers have read this CTA's partial
}

// How many clusters of 1, 2, 4, 8 CTAs (one CTA per SM) run at the same time.
struct ActiveClusters {
  int n[4] = {0, 0, 0, 0};
};

template <int DK, int DV, int MT>
int prepare(ActiveClusters& act) {
  static ActiveClusters known;
  if (known.n[0] == 0) {
    auto kern = attention_latent_kernel<DK, DV, MT>;
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, LatentSmem<DK, DV, MT>::kBytes);
    RD_CHECK_CHAINED(e);
    ActiveClusters found;
    for (int i = 0; i < 4; ++i) {
      cudaLaunchConfig_t cfg = {};
      cfg.gridDim = dim3(1 << i);
      cfg.blockDim = dim3(kLatThreads);
      cfg.dynamicSmemBytes = LatentSmem<DK, DV, MT>::kBytes;
      cudaLaunchAttribute attr;
      attr.id = cudaLaunchAttributeClusterDimension;
      attr.val.clusterDim.x = 1 << i;
      attr.val.clusterDim.y = attr.val.clusterDim.z = 1;
      cfg.attrs = &attr;
      cfg.numAttrs = 1;
      e = cudaOccupancyMaxActiveClusters(&found.n[i], kern, &cfg);
      RD_CHECK_CHAINED(e);
      if (found.n[i] < 1) found.n[i] = 1;
    }
    known = found;
  }
  act = known;
  return RD_OK;
}

template <int DK, int DV, int MT>
int launch(const LatentPlan* p, const Args& a, int32_t* status, const ActiveClusters& act, cudaStream_t s) {
  using Y = LatentSmem<DK, DV, MT>;
  const int64_t row_tiles = ((int64_t)a.nh * a.max_new + Y::kR - 1) / Y::kR;
  RD_REQUIRE(row_tiles <= 65535, RD_ERR_SIZE);
  // a cluster's CTAs share the key tiles of a row: the largest cluster of which all run at the same time, at least two
  // tiles per CTA
  const int64_t visible = (int64_t)a.window + a.max_new + a.keep_first + 2 * kBN;
  const int tiles = (int)((visible < a.max_kv ? visible : a.max_kv) + kBN - 1) / kBN;
  int i = 0;
  while (i < 3 && a.B * row_tiles <= act.n[i + 1] && (tiles >> (i + 1)) >= 2) ++i;
  const int ranks = 1 << i;
  cudaError_t err = rd::launch_chained(attention_latent_kernel<DK, DV, MT>, dim3(ranks, (int)row_tiles, a.B), dim3(kLatThreads), Y::kBytes, s,
                                       ranks, p->map_q, p->map_k, a, status);
  RD_CHECK_CHAINED(err);
  return RD_OK;
}

template <int DK, int DV>
int launch_rows(const LatentPlan* p, const Args& a, int32_t* status, cudaStream_t s) {
  // 16 rows per CTA while that leaves room for clusters of eight: the keys are read more often, from L2, but a CTA's chain
  // is shorter
  ActiveClusters act;
  int rc = prepare<DK, DV, 1>(act);
  if (rc != RD_OK) return rc;
  const int64_t small_tiles = ((int64_t)a.nh * a.max_new + 15) / 16;
  if (small_tiles == 1 || small_tiles * a.B <= act.n[3]) return launch<DK, DV, 1>(p, a, status, act, s);
  rc = prepare<DK, DV, 2>(act);
  return rc != RD_OK ? rc : launch<DK, DV, 2>(p, a, status, act, s);
}

}  // namespace

extern "C" void* rd_attention_latent_plan_create(const void* q, int64_t q_rows, const void* cache, int64_t cache_rows, int dim) {
  if (!q || !cache || q_rows < 1 || cache_rows < 1 || q_rows > INT32_MAX || cache_rows > INT32_MAX || dim < 8 || dim % 8 || dim > 576) return nullptr;
  if (((uintptr_t)q | (uintptr_t)cache) & 15) return nullptr;
  LatentPlan* p = new LatentPlan();
  p->dim = dim;
  if (!rd_umma::make_map(&p->map_q, q, q_rows, dim, dim, 16) || !rd_umma::make_map(&p->map_k, cache, cache_rows, dim, dim, kBN)) {
    delete p;
    return nullptr;
  }
  return p;
}

extern "C" void rd_attention_latent_plan_destroy(void* plan) { delete static_cast<LatentPlan*>(plan); }

extern "C" int rd_attention_latent(const void* plan, const rd_attention_desc* desc, int32_t* status, void* stream) {
  RD_REQUIRE(plan && desc, RD_ERR_ARG);
  const LatentPlan* p = static_cast<const LatentPlan*>(plan);
  const Args& a = *desc;
  RD_REQUIRE(a.out && a.row_start && a.kv_begin && a.base_len, RD_ERR_ARG);
  RD_REQUIRE(a.mode == RD_ATTN_CAUSAL || (a.mode == RD_ATTN_TREE && a.tree_mask && a.tok_pos && a.mask_words >= 1), RD_ERR_ARG);
  RD_REQUIRE(a.dtype == RD_BF16, RD_ERR_DTYPE);
  RD_REQUIRE(a.mask_kind == RD_MASK_WINDOW || a.mask_kind == RD_MASK_CHUNK, RD_ERR_ARG);
  RD_REQUIRE(a.B >= 1 && a.B <= 65535 && a.nh >= 1 && a.nkv == 1 && a.dim == p->dim && a.vdim >= 1 && a.vdim <= a.dim && a.vdim <= 512 &&
                 a.tail_dim == 0 && a.ldq == (int64_t)a.nh * a.dim && a.k_row == a.dim && a.k_batch % a.k_row == 0 && a.max_new >= 1 &&
                 a.window >= 1 && a.keep_first >= 0,
             RD_ERR_SIZE);
  cudaStream_t s = (cudaStream_t)stream;
  if (a.dim <= 128) return launch_rows<128, 128>(p, a, status, s);
  if (a.dim <= 320 && a.vdim <= 256) return launch_rows<320, 256>(p, a, status, s);
  return launch_rows<576, 512>(p, a, status, s);
}
