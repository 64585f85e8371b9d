// The matrix-memory recurrence of mlstm.cu for prompts: chunks of 64 tokens on the tensor cores (bf16 operands, fp32
// accumulators), the state carried in fp32 registers from chunk to chunk.
//
// Within a chunk, with F_t the running sum of the log forget gates and m_t the running maximum of the recurrence,
//   m_t   = F_t + max(m_in, max_{j <= t} (i_j - F_j))
//   P_tj  = (q_t . k_j) e^(F_t - F_j + i_j - m_t)                       j <= t
//   num_t = sum_j P_tj v_j + e^(F_t + m_in - m_t) S_in^T q_t,   den_t = sum_j P_tj + e^(F_t + m_in - m_t) n_in . q_t
//   S_out = e^(F_L + m_in - m_L) S_in + sum_j e^(F_L - F_j + i_j - m_L) k_j v_j^T      (n likewise with k alone)
// so every exponent is <= 0, and the result is the token-by-token recurrence up to rounding.
//
// A CTA owns VS value columns of one (row, head) and walks the row's chunks.  It keeps S^T [VS x dim] as mma
// accumulators: warp (mt, ks) holds value columns 16 mt .. +16 and the dim range of share ks.  As accumulators turn
// directly into A operands, S^T Q^T needs no exchange; the shares' partial outputs meet in shared memory.  The fp32
// operands of the products - P, S and what enters the state, e^(...) v_j - are each split into two bf16 parts (their
// rounding error is then about 2^-17).
#include "mlstm_common.cuh"
#include "mma_sync.cuh"

namespace {

using namespace rd_mma;
using namespace rd_mlstm;

constexpr int L = 64;         // tokens per chunk
constexpr int kThreads = 256;
constexpr int kRedLd = 66;    // floats per value column in the reduction buffer

struct ChunkArgs {
  const __nv_bfloat16* proj;  // [m, ld]: q | k | v | g
  int64_t ld;
  const float* gates;         // [m, ld_gates]: zi | zf
  int64_t ld_gates;
  const float* bias_i;
  const float* bias_f;
  float cap;
  float* o;                   // [m, nh * vdim] fp32
  float* S;
  const float* n;
  const float* m;
  float* nm_out;              // [B, nh, dim + 1]: n and m after the row's tokens (committed by the norm kernel)
  const int32_t* row_start;
  const int32_t* base_len;
  int nh, dim, vdim;
};

// 16-byte chunk c of row r in a tile of CH chunks per row, spread so that 8 consecutive rows hit 8 different bank groups
template <int CH>
__device__ __forceinline__ int swz(int r, int c) {
  if constexpr (CH >= 8)
    return r * (CH * 16) + ((c ^ (r & 7)) << 4);
  else
    return r * (CH * 16) + ((c ^ ((r >> 1) & 3)) << 4);  // 4 chunks: two rows per 128 bytes
}

// x as hi + lo, both bf16
__device__ __forceinline__ void split2(float x0, float x1, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x0, x1);
  const float2 f = __bfloat1622float2(h);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = pack_bf16(x0 - f.x, x1 - f.y);
}
__device__ __forceinline__ void split_store(uint8_t* hi, uint8_t* lo, int off, float x0, float x1) {
  split2(x0, x1, *reinterpret_cast<uint32_t*>(hi + off), *reinterpret_cast<uint32_t*>(lo + off));
}

template <int DP, int VS>
struct Layout {
  static constexpr int kQ = L * DP * 2, kV = L * VS * 2, kP = L * L * 2;
  static constexpr int kStage = 2 * kQ + kV;  // q, k, v
  static constexpr int kRed = 8 * 16 * kRedLd * 4;
  static constexpr int kMisc = (9 * L + DP + 8) * 4;
  static constexpr int kBytes = 2 * kStage + 2 * kP + 2 * kV + kRed + kMisc;
};

template <int DP, int VS>
__global__ void __launch_bounds__(kThreads, 1) mlstm_chunk_kernel(const ChunkArgs a) {
  using Y = Layout<DP, VS>;
  constexpr int MT = VS / 16, KS = 8 / MT;    // value tiles, dim shares
  constexpr int DS = DP / KS;                 // dims per share
  constexpr int NT = DS / 8;                  // accumulator tiles of S^T per warp
  constexpr int CQ = DP / 8, CV = VS / 8;     // 16-byte chunks per row
  extern __shared__ __align__(128) uint8_t smem[];
  rd::pdl_launch_dependents();
  rd::pdl_wait();
  const int b = blockIdx.z, h = blockIdx.y, c0 = blockIdx.x * VS;
  const int rs = a.row_start[b];
  const int n_tok = a.row_start[b + 1] - rs;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int g = lane >> 2, t4 = lane & 3;
  float* nm_out = a.nm_out + ((int64_t)b * a.nh + h) * (a.dim + 1);
  const bool fresh = a.base_len[b] == 0;
  if (n_tok <= 0) return;

  uint8_t* sP = smem + 2 * Y::kStage;
  uint8_t* sPlo = sP + Y::kP;
  uint8_t* sWhi = sPlo + Y::kP;
  uint8_t* sWlo = sWhi + Y::kV;
  float* red = reinterpret_cast<float*>(sWlo + Y::kV);  // [8 warps][16][kRedLd]
  float* misc = red + 8 * 16 * kRedLd;
  float* s_Fm = misc;            // [L] F_t - m_t
  float* s_iF = misc + L;        // [L] i_j - F_j  (-inf past the end)
  float* s_e = misc + 2 * L;     // [L] dim^(-1/2) e^(F_t + m_in - m_t)
  float* s_w = misc + 3 * L;     // [L] e^(F_L - F_j + i_j - m_L)
  float* s_floor = misc + 4 * L; // [L] e^(-m_t)
  float* s_rs = misc + 5 * L;    // [2][L] row sums of P
  float* s_nq = misc + 7 * L;    // [L] n_in . q_t
  float* s_n = misc + 9 * L;     // [DP]
  float* s_sc = s_n + DP;        // [0] e^(F_L + m_in - m_L), [1] m_L

  const int mt = warp % MT, ks = warp / MT;
  const float qs = rsqrtf((float)a.dim);
  const float bi = a.bias_i[h], bf = a.bias_f[h];

  // state
  float S[NT][4];
  float* S_g = a.S + ((int64_t)b * a.nh + h) * a.dim * a.vdim;
  auto each_state = [&](auto&& fn) {
#pragma unroll
    for (int nt = 0; nt < NT; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int d = ks * DS + nt * 8 + t4 * 2 + (e & 1), v = c0 + mt * 16 + g + (e >> 1) * 8;
        fn(S[nt][e], d < a.dim && v < a.vdim, (int64_t)d * a.vdim + v);
      }
  };
  each_state([&](float& s, bool in, int64_t off) { s = (in && !fresh) ? S_g[off] : 0.f; });
  for (int d = tid; d < DP; d += kThreads) s_n[d] = (d < a.dim && !fresh) ? a.n[((int64_t)b * a.nh + h) * a.dim + d] : 0.f;
  float m_in = fresh ? 0.f : a.m[(int64_t)b * a.nh + h];  // tracked by warp 0

  auto load_chunk = [&](int c) {
    uint8_t* st = smem + (c & 1) * Y::kStage;
    const int t0 = c * L;
    for (int idx = tid; idx < L * CQ; idx += kThreads) {
      const int r = idx / CQ, ch = idx % CQ;
      const bool in = t0 + r < n_tok && ch * 8 < a.dim;
      const __nv_bfloat16* src = a.proj + (int64_t)(rs + (in ? t0 + r : 0)) * a.ld + h * a.dim + (in ? ch * 8 : 0);
      cp_async16(st + swz<CQ>(r, ch), src, in);
      cp_async16(st + Y::kQ + swz<CQ>(r, ch), src + a.nh * a.dim, in);
    }
    for (int idx = tid; idx < L * CV; idx += kThreads) {
      const int r = idx / CV, ch = idx % CV;
      const bool in = t0 + r < n_tok && c0 + ch * 8 < a.vdim;
      const __nv_bfloat16* src =
          a.proj + (int64_t)(rs + (in ? t0 + r : 0)) * a.ld + 2 * a.nh * a.dim + h * a.vdim + (in ? c0 + ch * 8 : 0);
      cp_async16(st + 2 * Y::kQ + swz<CV>(r, ch), src, in);
    }
    cp_async_commit();
  };
  // the two gate pre-activations of this lane's tokens of a chunk (warp 0)
  float gi[2], gf[2];
  auto load_gates = [&](int c) {
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int t = c * L + lane * 2 + e;
      const float* p = a.gates + (int64_t)(rs + min(t, n_tok - 1)) * a.ld_gates + h;
      gi[e] = p[0];
      gf[e] = p[a.nh];
    }
  };

  const int n_chunks = (n_tok + L - 1) / L;
  load_chunk(0);
  if (warp == 0) load_gates(0);

  for (int c = 0; c < n_chunks; ++c) {
    const int live = min(L, n_tok - c * L);
    const uint8_t* sQ = smem + (c & 1) * Y::kStage;
    const uint8_t* sK = sQ + Y::kQ;
    const uint8_t* sV = sQ + 2 * Y::kQ;
    if (warp == 0) {
      // gates: lane owns tokens 2 lane and 2 lane + 1
      float f[2], x[2], F[2], M[2];
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const bool in = lane * 2 + e < live;
        f[e] = in ? log_sigmoid(soft_cap(gf[e] + bf, a.cap)) : 0.f;
        x[e] = in ? soft_cap(gi[e] + bi, a.cap) : -INFINITY;
      }
      float run = f[0] + f[1];
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float up = __shfl_up_sync(0xffffffffu, run, o);
        if (lane >= o) run += up;
      }
      F[1] = run;
      F[0] = run - f[1];
      x[0] -= F[0];  // i_j - F_j
      x[1] -= F[1];
      float mx = fmaxf(x[0], x[1]);
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float up = __shfl_up_sync(0xffffffffu, mx, o);
        if (lane >= o) mx = fmaxf(mx, up);
      }
      const float before = __shfl_up_sync(0xffffffffu, mx, 1);
      M[0] = fmaxf(lane ? before : -INFINITY, x[0]);
      M[1] = mx;
      float mm[2];
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        mm[e] = F[e] + fmaxf(m_in, M[e]);
        const int t = lane * 2 + e;
        s_Fm[t] = F[e] - mm[e];
        s_iF[t] = x[e];
        s_e[t] = qs * expf(F[e] + m_in - mm[e]);
        s_floor[t] = expf(-mm[e]);
      }
      // tokens past the end repeat the last live one's F and m (f = 0, i = -inf), so lane 31 holds the chunk's
      const float FL = __shfl_sync(0xffffffffu, F[1], 31), mL = __shfl_sync(0xffffffffu, mm[1], 31);
#pragma unroll
      for (int e = 0; e < 2; ++e) s_w[lane * 2 + e] = expf(FL - mL + x[e]);
      if (lane == 0) {
        s_sc[0] = expf(FL + m_in - mL);
        s_sc[1] = mL;
      }
      m_in = mL;
      if (c + 1 < n_chunks) load_gates(c + 1);
    }
    cp_async_wait<0>();
    __syncthreads();  // chunk c and its gates are visible; everyone has left chunk c - 1
    if (c + 1 < n_chunks) load_chunk(c + 1);

    // ---- P = (Q K^T) o weights: warp -> 16 tokens x 32 keys
    {
      const int t0 = (warp & 3) * 16, j0 = (warp >> 2) * 32;
      float s[4][4];
#pragma unroll
      for (int nt = 0; nt < 4; ++nt) s[nt][0] = s[nt][1] = s[nt][2] = s[nt][3] = 0.f;
      if (j0 <= t0 + 15) {
#pragma unroll 4
        for (int kd = 0; kd < DP / 16; ++kd) {
          uint32_t af[4];
          ldmatrix_x4(af[0], af[1], af[2], af[3], smem_addr(sQ + swz<CQ>(t0 + (lane & 15), kd * 2 + (lane >> 4))));
#pragma unroll
          for (int nb = 0; nb < 4; nb += 2) {
            uint32_t b0, b1, b2, b3;
            ldmatrix_x4(b0, b1, b2, b3,
                        smem_addr(sK + swz<CQ>(j0 + nb * 8 + ((lane >> 4) << 3) + (lane & 7), kd * 2 + ((lane >> 3) & 1))));
            mma_bf16(s[nb], af, b0, b1);
            mma_bf16(s[nb + 1], af, b2, b3);
          }
        }
      }
      float sum[2] = {0.f, 0.f};
#pragma unroll
      for (int hh = 0; hh < 2; ++hh) {
        const int t = t0 + g + hh * 8;
        const float Fm = s_Fm[t];
#pragma unroll
        for (int nt = 0; nt < 4; ++nt) {
          const int j = j0 + nt * 8 + t4 * 2;
          const float p0 = j <= t ? s[nt][hh * 2] * qs * expf(Fm + s_iF[j]) : 0.f;
          const float p1 = j + 1 <= t ? s[nt][hh * 2 + 1] * qs * expf(Fm + s_iF[j + 1]) : 0.f;
          sum[hh] += p0 + p1;
          split_store(sP, sPlo, swz<8>(t, j >> 3) + (j & 7) * 2, p0, p1);
        }
        sum[hh] += __shfl_xor_sync(0xffffffffu, sum[hh], 1);
        sum[hh] += __shfl_xor_sync(0xffffffffu, sum[hh], 2);
        if (t4 == 0) s_rs[(warp >> 2) * L + t] = sum[hh];
      }
    }
    // ---- w_j v_j as hi + lo
    for (int idx = tid; idx < L * VS / 2; idx += kThreads) {
      const int r = idx / (VS / 2), cc = (idx % (VS / 2)) * 2;
      const int off = swz<CV>(r, cc >> 3) + (cc & 7) * 2;
      const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(sV + off));
      const float w = s_w[r];
      const float x0 = v.x * w, x1 = v.y * w;
      split_store(sWhi, sWlo, off, x0, x1);
    }
    // ---- n_in . q_t: four threads per token
    {
      const int t = tid >> 2, part = tid & 3;
      float acc = 0.f;
#pragma unroll 4
      for (int ch = part; ch < CQ; ch += 4) {
        const uint4 u = *reinterpret_cast<const uint4*>(sQ + swz<CQ>(t, ch));
        const __nv_bfloat162* q2 = reinterpret_cast<const __nv_bfloat162*>(&u);
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float2 f = __bfloat1622float2(q2[e]);
          acc = fmaf(f.x, s_n[ch * 8 + 2 * e], acc);
          acc = fmaf(f.y, s_n[ch * 8 + 2 * e + 1], acc);
        }
      }
      acc += __shfl_xor_sync(0xffffffffu, acc, 1);
      acc += __shfl_xor_sync(0xffffffffu, acc, 2);
      if (part == 0) s_nq[t] = acc;
    }
    __syncthreads();

    // ---- O^T (this warp's share) = e_t S^T Q^T + V^T P^T
    {
      float o[8][4];
#pragma unroll
      for (int nt = 0; nt < 8; ++nt) o[nt][0] = o[nt][1] = o[nt][2] = o[nt][3] = 0.f;
#pragma unroll
      for (int kd = 0; kd < DS / 16; ++kd) {
        uint32_t hi[4], lo[4];
        split2(S[2 * kd][0], S[2 * kd][1], hi[0], lo[0]);
        split2(S[2 * kd][2], S[2 * kd][3], hi[1], lo[1]);
        split2(S[2 * kd + 1][0], S[2 * kd + 1][1], hi[2], lo[2]);
        split2(S[2 * kd + 1][2], S[2 * kd + 1][3], hi[3], lo[3]);
#pragma unroll
        for (int nb = 0; nb < 8; nb += 2) {
          uint32_t b0, b1, b2, b3;
          ldmatrix_x4(b0, b1, b2, b3,
                      smem_addr(sQ + swz<CQ>(nb * 8 + ((lane >> 4) << 3) + (lane & 7), (ks * DS) / 8 + kd * 2 + ((lane >> 3) & 1))));
          mma_bf16(o[nb], hi, b0, b1);
          mma_bf16(o[nb + 1], hi, b2, b3);
          mma_bf16(o[nb], lo, b0, b1);
          mma_bf16(o[nb + 1], lo, b2, b3);
        }
      }
#pragma unroll
      for (int nt = 0; nt < 8; ++nt) {
        const float e0 = s_e[nt * 8 + t4 * 2], e1 = s_e[nt * 8 + t4 * 2 + 1];
        o[nt][0] *= e0;
        o[nt][1] *= e1;
        o[nt][2] *= e0;
        o[nt][3] *= e1;
      }
      // this share's tokens j: 64 / KS of them
#pragma unroll
      for (int kj = 0; kj < L / KS / 16; ++kj) {
        const int j0 = ks * (L / KS) + kj * 16;
        uint32_t af[4];
        ldmatrix_x4_trans(af[0], af[1], af[2], af[3],
                          smem_addr(sV + swz<CV>(j0 + ((lane >> 4) << 3) + (lane & 7), mt * 2 + ((lane >> 3) & 1))));
#pragma unroll
        for (int nb = 0; nb < 8; nb += 2) {
          const int off = swz<8>(nb * 8 + ((lane >> 4) << 3) + (lane & 7), (j0 >> 3) + ((lane >> 3) & 1));
          uint32_t b0, b1, b2, b3;
          ldmatrix_x4(b0, b1, b2, b3, smem_addr(sP + off));
          mma_bf16(o[nb], af, b0, b1);
          mma_bf16(o[nb + 1], af, b2, b3);
          ldmatrix_x4(b0, b1, b2, b3, smem_addr(sPlo + off));
          mma_bf16(o[nb], af, b0, b1);
          mma_bf16(o[nb + 1], af, b2, b3);
        }
      }
      float* dst = red + (ks * MT + mt) * 16 * kRedLd;
#pragma unroll
      for (int nt = 0; nt < 8; ++nt) {
        *reinterpret_cast<float2*>(dst + g * kRedLd + nt * 8 + t4 * 2) = make_float2(o[nt][0], o[nt][1]);
        *reinterpret_cast<float2*>(dst + (g + 8) * kRedLd + nt * 8 + t4 * 2) = make_float2(o[nt][2], o[nt][3]);
      }
    }
    // ---- S^T = A S^T + (w V)^T K
    {
      const float A = s_sc[0];
#pragma unroll
      for (int nt = 0; nt < NT; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) S[nt][e] *= A;
#pragma unroll
      for (int kj = 0; kj < L / 16; ++kj) {
        const int row = kj * 16 + ((lane >> 4) << 3) + (lane & 7), ch = mt * 2 + ((lane >> 3) & 1);
        uint32_t hi[4], lo[4];
        ldmatrix_x4_trans(hi[0], hi[1], hi[2], hi[3], smem_addr(sWhi + swz<CV>(row, ch)));
        ldmatrix_x4_trans(lo[0], lo[1], lo[2], lo[3], smem_addr(sWlo + swz<CV>(row, ch)));
#pragma unroll
        for (int nt = 0; nt < NT; nt += 2) {
          uint32_t b0, b1, b2, b3;
          ldmatrix_x4_trans(b0, b1, b2, b3,
                            smem_addr(sK + swz<CQ>(kj * 16 + (((lane >> 3) & 1) << 3) + (lane & 7), (ks * DS) / 8 + nt + (lane >> 4))));
          mma_bf16(S[nt], hi, b0, b1);
          mma_bf16(S[nt + 1], hi, b2, b3);
          mma_bf16(S[nt], lo, b0, b1);
          mma_bf16(S[nt + 1], lo, b2, b3);
        }
      }
      for (int d = tid; d < DP; d += kThreads) {
        float nn = s_n[d] * A;
#pragma unroll 8
        for (int j = 0; j < L; ++j)
          nn = fmaf(s_w[j], __bfloat162float(*reinterpret_cast<const __nv_bfloat16*>(sK + swz<CQ>(j, d >> 3) + (d & 7) * 2)), nn);
        s_n[d] = nn;  // only this thread reads or writes it until the next barrier
      }
    }
    __syncthreads();
    // ---- outputs: sum of the shares over the denominator
    for (int idx = tid; idx < live * VS; idx += kThreads) {
      const int t = idx / VS, v = idx % VS;
      if (c0 + v < a.vdim) {
        const float* src = red + ((v >> 4) * 16 + (v & 15)) * kRedLd + t;
        float num = 0.f;
#pragma unroll
        for (int k = 0; k < KS; ++k) num += src[k * MT * 16 * kRedLd];
        const float den = s_rs[t] + s_rs[L + t] + s_e[t] * s_nq[t];
        a.o[((int64_t)(rs + c * L + t) * a.nh + h) * a.vdim + c0 + v] = num / (fmaxf(fabsf(den), s_floor[t]) + kDenEps);
      }
    }
    __syncthreads();  // the gate arrays are rewritten by warp 0 for the next chunk
  }
  each_state([&](float& s, bool in, int64_t off) {
    if (in) S_g[off] = s;
  });
  if (blockIdx.x == 0) {
    for (int d = tid; d < a.dim; d += kThreads) nm_out[d] = s_n[d];
    if (tid == 0) nm_out[a.dim] = s_sc[1];
  }
}

template <int DP, int VS>
int launch_chunk(const ChunkArgs& a, int B, cudaStream_t s) {
  using Y = Layout<DP, VS>;
  auto kern = mlstm_chunk_kernel<DP, VS>;
  static bool smem_set = false;
  if (!smem_set) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, Y::kBytes);
    RD_CHECK_CHAINED(e);
    smem_set = true;
  }
  cudaError_t err = rd::launch_chained(kern, dim3((a.vdim + VS - 1) / VS, a.nh, B), dim3(kThreads), Y::kBytes, s, 1, a);
  RD_CHECK_CHAINED(err);
  return RD_OK;
}

}  // namespace

extern "C" int64_t rd_mlstm_chunk_workspace_bytes(int m_max, int B, int nh, int dim, int vdim) {
  return ((int64_t)m_max * nh * vdim + (int64_t)B * nh * (dim + 1)) * (int64_t)sizeof(float);
}

extern "C" int rd_mlstm_chunk(const void* proj, int64_t ld, const float* gates, int64_t ld_gates, const float* bias_i,
                              const float* bias_f, float gate_cap, const void* norm_weight, float eps, void* out, float* S,
                              float* n, float* m, const int32_t* row_start, const int32_t* base_len, int B, int nh, int dim,
                              int vdim, int m_max, void* workspace, int64_t workspace_bytes, void* stream) {
  RD_REQUIRE(proj && gates && bias_i && bias_f && norm_weight && out && S && n && m && row_start && base_len && workspace, RD_ERR_ARG);
  RD_REQUIRE(B >= 1 && B <= 65535 && nh >= 1 && nh <= 65535 && dim >= 8 && dim <= 256 && dim % 8 == 0 && vdim >= 8 && vdim % 8 == 0 &&
                 m_max >= 1 && gate_cap > 0.f && ld >= 2 * (int64_t)nh * (dim + vdim) && ld_gates >= 2 * nh,
             RD_ERR_SIZE);
  RD_REQUIRE((((uintptr_t)proj | (uintptr_t)norm_weight | (uintptr_t)out | (uintptr_t)workspace) & 15) == 0 && ld % 8 == 0, RD_ERR_ALIGN);
  RD_REQUIRE(workspace_bytes >= rd_mlstm_chunk_workspace_bytes(m_max, B, nh, dim, vdim), RD_ERR_CAPACITY);
  float* o = (float*)workspace;
  float* nm = o + (int64_t)m_max * nh * vdim;
  ChunkArgs a{(const __nv_bfloat16*)proj, ld, gates, ld_gates, bias_i, bias_f, gate_cap, o, S, n, m, nm, row_start, base_len, nh, dim, vdim};
  cudaStream_t s = (cudaStream_t)stream;
  // narrow slices until every SM has a CTA: half the columns per CTA repeat the chunk's Q K^T, but the row's chunks, which
  // follow one another, take about 0.6 of the time
  const bool wide = (int64_t)B * nh * ((vdim + 63) / 64) >= 148;
  int rc;
  if (dim <= 64)
    rc = wide ? launch_chunk<64, 64>(a, B, s) : launch_chunk<64, 32>(a, B, s);
  else if (dim <= 128)
    rc = wide ? launch_chunk<128, 64>(a, B, s) : launch_chunk<128, 32>(a, B, s);
  else
    rc = wide ? launch_chunk<256, 64>(a, B, s) : launch_chunk<256, 32>(a, B, s);
  if (rc != RD_OK) return rc;
  const __nv_bfloat16* gp = (const __nv_bfloat16*)proj + (int64_t)2 * nh * dim + (int64_t)nh * vdim;
  return launch_norm_gate<__nv_bfloat16>(o, gp, ld, norm_weight, out, eps, m_max, row_start, B, nh, dim, vdim, nm, n, m, s);
}
