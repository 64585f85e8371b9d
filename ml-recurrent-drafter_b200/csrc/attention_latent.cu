// Masked attention where all heads share one key and the values are the first part of that key (latent attention with the
// up-projections of keys and values moved to the queries and the output), bf16, warp-level tensor cores.
//
// One CTA serves 16 * MT query rows (token, head) of one batch row; a key tile of 64 is read once for scores and values and
// for all of them.  Eight warps: each takes a share of the tile's keys for the scores, then its own eighth of the value
// columns for all rows (row maxima and the weights travel through shared memory).  A cluster of CTAs shares the key tiles
// and merges its partial results through distributed shared memory.
#include "attention_window_tc.cuh"

namespace {

using namespace rd_win;

constexpr int kLatThreads = 256;
constexpr int kLatWarps = kLatThreads / 32;
constexpr int kMaxRanks = 8;

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
  static constexpr int kBytes = kQ + kRing + kP + kRed + kMl + kWeights;
  static_assert(kR * kOld * 4 <= kRing, "the partial output lies over the key ring");
};

// grid (cluster, row tiles, B); cluster (n_split, 1, 1)
template <int DK, int DV, int MT>
__global__ void __launch_bounds__(kLatThreads) attention_latent_kernel(const Args a) {
  using Y = LatentSmem<DK, DV, MT>;
  constexpr int R = Y::kR, KG = Y::kKG, ST = Y::kStages, CK = DK / 8;
  constexpr int NB = DV / (8 * kLatWarps);  // 8-column blocks of values per warp
  cg::cluster_group cluster = cg::this_cluster();
  rd::pdl_launch_dependents();
  rd::pdl_wait();
  const int b = blockIdx.z, row_first = blockIdx.y * R;
  const int rank = (int)cluster.block_rank(), n_ranks = (int)cluster.num_blocks();
  const int rs = a.row_start[b];
  const int n_new = a.row_start[b + 1] - rs;
  const int n_rows = min(R, a.nh * n_new - row_first);
  if (n_rows <= 0) return;  // the same for the whole cluster
  extern __shared__ __align__(128) uint8_t smem[];
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
  RowKeys<__nv_bfloat16> keys;
  keys.init(a, b, 0);
  for (int idx = tid; idx < R * CK; idx += kLatThreads) {
    const int r = idx / CK, c = idx % CK;
    const bool in = r < n_rows && c * 8 < a.dim;
    const __nv_bfloat16* src = (const __nv_bfloat16*)a.q;
    if (in) src += (int64_t)(rs + (row_first + r) / a.nh) * a.ldq + (int64_t)((row_first + r) % a.nh) * a.dim + c * 8;
    cp_async16(sQ + swz<CK>(r, c), src, in);
  }
  auto load = [&](int t) {
    if (t < n_tiles)
      load_tile<DK, kLatThreads>(ring + (t % ST) * Y::kK, keys.k, a.k_row, a.dim, tiles.tile(t_begin + t) * kBN, kv_end, tid);
    cp_async_commit();
  };
  for (int t = 0; t < ST - 1; ++t) load(t);
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
  for (int it = 0; it < n_tiles; ++it) {
    cp_async_wait<ST - 2>();
    __syncthreads();
    load(it + ST - 1);
    const uint8_t* sK = ring + (it % ST) * Y::kK;
    float s2[2][MT][4] = {};  // even and odd steps along the features
#pragma unroll 4
    for (int kd = 0; kd < DK / 16; kd += 2) {
      uint32_t a0[4], a1[4];
      ldmatrix_x4(a0[0], a0[1], a0[2], a0[3], smem_addr(sQ + swz<CK>(mt_s * 16 + (lane & 15), kd * 2 + (lane >> 4))));
      ldmatrix_x4(a1[0], a1[1], a1[2], a1[3], smem_addr(sQ + swz<CK>(mt_s * 16 + (lane & 15), kd * 2 + 2 + (lane >> 4))));
      uint32_t b0, b1, b2, b3;
      if constexpr (MT == 1) {
        ldmatrix_x4(b0, b1, b2, b3, smem_addr(sK + swz<CK>(k0 + (lane & 7), kd * 2 + (lane >> 3))));
        mma_bf16(s2[0][0], a0, b0, b1);
        mma_bf16(s2[1][0], a1, b2, b3);
      } else {
        const int row = k0 + ((lane >> 4) << 3) + (lane & 7);
        ldmatrix_x4(b0, b1, b2, b3, smem_addr(sK + swz<CK>(row, kd * 2 + ((lane >> 3) & 1))));
        mma_bf16(s2[0][0], a0, b0, b1);
        mma_bf16(s2[0][MT - 1], a0, b2, b3);
        ldmatrix_x4(b0, b1, b2, b3, smem_addr(sK + swz<CK>(row, kd * 2 + 2 + ((lane >> 3) & 1))));
        mma_bf16(s2[1][0], a1, b0, b1);
        mma_bf16(s2[1][MT - 1], a1, b2, b3);
      }
    }
    const int j0 = tiles.tile(t_begin + it) * kBN + k0;
    float s[MT][4], mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
    for (int nb = 0; nb < MT; ++nb)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float v = qu[e >> 1].sees(a, j0 + nb * 8 + t4 * 2 + (e & 1)) ? (s2[0][nb][e] + s2[1][nb][e]) * scale_log2 : -INFINITY;
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
                          smem_addr(sK + swz<CK>(kk * 16 + (((lane >> 3) & 1) << 3) + (lane & 7), warp * NB + db + (lane >> 4))));
#pragma unroll
        for (int mt = 0; mt < MT; ++mt) {
          mma_bf16(o[mt][db], pf[mt], b0, b1);
          mma_bf16(o[mt][db + 1], pf[mt], b2, b3);
        }
      }
    }
  }
  cp_async_wait<0>();
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

template <int DK, int DV, int MT>
int launch(const Args& a, cudaStream_t s) {
  auto kern = attention_latent_kernel<DK, DV, MT>;
  using Y = LatentSmem<DK, DV, MT>;
  static bool set = false;
  if (!set) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, Y::kBytes);
    RD_CHECK_CHAINED(e);
    set = true;
  }
  const int64_t row_tiles = ((int64_t)a.nh * a.max_new + Y::kR - 1) / Y::kR;
  RD_REQUIRE(row_tiles <= 65535, RD_ERR_SIZE);
  // a cluster's CTAs share the key tiles of a row: enough of them to fill the GPU, at least two tiles each
  const int64_t visible = (int64_t)a.window + a.max_new + a.keep_first + 2 * kBN;
  const int tiles = (int)((visible < a.max_kv ? visible : a.max_kv) + kBN - 1) / kBN;
  int ranks = 1;
  while (ranks < kMaxRanks && a.B * row_tiles * ranks < 148 && tiles / (ranks * 2) >= 2) ranks *= 2;
  cudaError_t err = rd::launch_chained(kern, dim3(ranks, (int)row_tiles, a.B), dim3(kLatThreads), Y::kBytes, s, ranks, a);
  RD_CHECK_CHAINED(err);
  return RD_OK;
}

template <int DK, int DV>
int launch_rows(const Args& a, cudaStream_t s) {
  return (int64_t)a.nh * a.max_new <= 16 ? launch<DK, DV, 1>(a, s) : launch<DK, DV, 2>(a, s);
}

}  // namespace

bool rd_attention_latent_ok(const Args& a) {
  const uintptr_t bits = (uintptr_t)a.q | (uintptr_t)a.k;
  const int64_t strides = a.ldq | a.k_batch | a.k_row;
  return a.dtype == RD_BF16 && a.v == a.k && a.nkv == 1 && a.v_row == a.k_row && a.v_batch == a.k_batch && a.tail_dim == 0 &&
         a.vdim <= a.dim && a.dim % 8 == 0 && strides % 8 == 0 && bits % 16 == 0 && a.dim <= 576 && a.vdim <= 512;
}

int rd_attention_latent_launch(const Args& a, cudaStream_t s) {
  if (a.dim <= 128) return launch_rows<128, 128>(a, s);
  if (a.dim <= 320 && a.vdim <= 256) return launch_rows<320, 256>(a, s);
  return launch_rows<576, 512>(a, s);
}
