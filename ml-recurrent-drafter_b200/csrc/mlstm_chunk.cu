// The matrix-memory recurrence of mlstm.cu for prompts: chunks of 128 tokens on the tensor cores (bf16 operands, fp32
// accumulators).
//
// Within a chunk, with F_t the running sum of the log forget gates and m_t the running maximum of the recurrence,
//   m_t   = F_t + max(m_in, max_{j <= t} (i_j - F_j))
//   P_tj  = (q_t . k_j) e^(F_t - F_j + i_j - m_t)                       j <= t
//   num_t = sum_j P_tj v_j + e^(F_t + m_in - m_t) S_in^T q_t,   den_t = sum_j P_tj + e^(F_t + m_in - m_t) n_in . q_t
//   S_out = e^(F_L + m_in - m_L) S_in + sum_j e^(F_L - F_j + i_j - m_L) k_j v_j^T      (n likewise with k alone)
// so every exponent is <= 0, and the result is the token-by-token recurrence up to rounding.  Three kernels:
//   gates    one CTA per (head, row): the scalars above for every token; only the chunks' maxima follow one another
//   states   one CTA per 64 x 64 tile of S: walks the chunks, the tile in fp32 accumulators, and leaves S and n at the
//            start of every chunk in the workspace
//   outputs  one CTA per 64 tokens of a head: scores, both products, the head's RMS norm, the norm weight and the output
//            gate, independent of all other chunks
// The fp32 operands of the products - P, S and what enters the state, e^(...) v_j - are each split into two bf16 parts
// (their rounding error is then about 2^-17).
#include "mlstm_common.cuh"
#include "mma_sync.cuh"

namespace {

using namespace rd_mma;
using namespace rd_mlstm;

constexpr int L = 128;  // tokens per chunk
constexpr int kThreads = 256;

struct ChunkArgs {
  const __nv_bfloat16* proj;  // [m, ld]: q | k | v | g
  int64_t ld;
  const float* gates;         // [m, ld_gates]: zi | zf
  int64_t ld_gates;
  const float* bias_i;
  const float* bias_f;
  float cap;
  const __nv_bfloat16* norm_w;
  float eps;
  __nv_bfloat16* out;         // [m, nh * vdim]
  float* S;
  float* n;
  float* m;
  const int32_t* row_start;
  const int32_t* base_len;
  int nh, dim, vdim, dpad, vpad, m_max;
  // workspace.  Per head and token [nh][m_max]:
  float* Fm;     // F_t - m_t
  float* iF;     // i_j - F_j
  float* e;      // dim^(-1/2) e^(F_t + m_in - m_t)
  float* w;      // e^(F_L - F_j + i_j - m_L)
  float* floor;  // e^(-m_t)
  // per chunk slot and head; row b's chunk c has slot row_start[b] / L + b + c
  float* decay;  // e^(F_L + m_in - m_L)
  float* nc;     // [dpad] n at the chunk's start
  __nv_bfloat16* Shi;  // [dpad][vpad] S at the chunk's start
  __nv_bfloat16* Slo;
};

__device__ __forceinline__ int chunk_slot(int rs, int b, int c) { return rs / L + b + c; }

// 16-byte chunk c of row r in a tile of CH >= 8 chunks per row, spread so that 8 consecutive rows hit 8 different bank groups
template <int CH>
__device__ __forceinline__ int swz(int r, int c) {
  return r * (CH * 16) + ((c ^ (r & 7)) << 4);
}

// x as hi + lo, both bf16
__device__ __forceinline__ void split2(float x0, float x1, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x0, x1);
  const float2 f = __bfloat1622float2(h);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = pack_bf16(x0 - f.x, x1 - f.y);
}

// ------------------------------------------------------------------------------------------------ gates
__global__ void __launch_bounds__(kThreads) mlstm_gates_kernel(const ChunkArgs a) {
  extern __shared__ __align__(128) uint8_t smem[];
  rd::pdl_launch_dependents();
  rd::pdl_wait();
  const int h = blockIdx.x, b = blockIdx.y;
  const int rs = a.row_start[b], n_tok = a.row_start[b + 1] - rs;
  if (n_tok <= 0) return;
  const int n_chunks = (n_tok + L - 1) / L;
  float* c_F = reinterpret_cast<float*>(smem);  // F_L of every chunk
  float* c_M = c_F + n_chunks;                  // max_j (i_j - F_j)
  float* c_m = c_M + n_chunks;                  // m_in
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const float bi = a.bias_i[h], bf = a.bias_f[h];
  const int64_t at = (int64_t)h * a.m_max + rs;
  for (int c = warp; c < n_chunks; c += kThreads / 32) {
    // lane owns four consecutive tokens
    float f[4], x[4], F = 0.f, mx = -INFINITY;
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int t = c * L + lane * 4 + e;
      const float* p = a.gates + (int64_t)(rs + min(t, n_tok - 1)) * a.ld_gates + h;
      f[e] = t < n_tok ? log_sigmoid(soft_cap(p[a.nh] + bf, a.cap)) : 0.f;
      x[e] = t < n_tok ? soft_cap(p[0] + bi, a.cap) : -INFINITY;
      F += f[e];
    }
    float run = F;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float up = __shfl_up_sync(0xffffffffu, run, o);
      if (lane >= o) run += up;
    }
    F = run - F;  // sum before this lane's tokens
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      F += f[e];
      f[e] = F;
      x[e] -= F;
      mx = fmaxf(mx, x[e]);
    }
    float up_to = mx;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float up = __shfl_up_sync(0xffffffffu, up_to, o);
      if (lane >= o) up_to = fmaxf(up_to, up);
    }
    float M = __shfl_up_sync(0xffffffffu, up_to, 1);
    if (lane == 0) M = -INFINITY;
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int t = c * L + lane * 4 + e;
      M = fmaxf(M, x[e]);
      if (t < n_tok) {
        // for the second pass: F_t, i_t - F_t, running maximum
        a.Fm[at + t] = f[e];
        a.iF[at + t] = x[e];
        a.floor[at + t] = M;
      }
    }
    if (lane == 31) {
      c_F[c] = f[3];
      c_M[c] = up_to;
    }
  }
  __syncthreads();
  if (threadIdx.x == 0) {
    float m = a.base_len[b] == 0 ? 0.f : a.m[(int64_t)b * a.nh + h];
    for (int c = 0; c < n_chunks; ++c) {
      c_m[c] = m;
      m = c_F[c] + fmaxf(m, c_M[c]);
    }
    a.m[(int64_t)b * a.nh + h] = m;
  }
  __syncthreads();
  const float qs = rsqrtf((float)a.dim);
  for (int c = warp; c < n_chunks; c += kThreads / 32) {
    const float m_in = c_m[c], FL = c_F[c], mL = FL + fmaxf(m_in, c_M[c]);
    if (lane == 0) a.decay[(int64_t)chunk_slot(rs, b, c) * a.nh + h] = expf(FL + m_in - mL);
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int t = c * L + lane * 4 + e;
      if (t < n_tok) {
        const float F = a.Fm[at + t], x = a.iF[at + t], m = F + fmaxf(m_in, a.floor[at + t]);
        a.Fm[at + t] = F - m;
        a.e[at + t] = qs * expf(F + m_in - m);
        a.w[at + t] = expf(FL - mL + x);
        a.floor[at + t] = expf(-m);
      }
    }
  }
}

// ------------------------------------------------------------------------------------------------ states
struct StateSmem {
  static constexpr int kTile = L * 64 * 2;  // [L tokens][64 features]
  static constexpr int kBytes = 4 * kTile + 2 * kTile + (2 * L + 64) * 4;  // two stages of K and V, wV hi and lo, w, n
};

// grid (dim tiles * value tiles, nh, B).  Warp: 16 dims x 32 value columns.
__global__ void __launch_bounds__(kThreads, 2) mlstm_states_kernel(const ChunkArgs a) {
  extern __shared__ __align__(128) uint8_t smem[];
  rd::pdl_launch_dependents();
  rd::pdl_wait();
  const int b = blockIdx.z, h = blockIdx.y;
  const int v_tiles = a.vpad / 64;
  const int d0 = (blockIdx.x / v_tiles) * 64, v0 = (blockIdx.x % v_tiles) * 64;
  const int rs = a.row_start[b], n_tok = a.row_start[b + 1] - rs;
  if (n_tok <= 0) return;
  const int n_chunks = (n_tok + L - 1) / L;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  const int dm = (warp >> 1) * 16, vn = (warp & 1) * 32;
  constexpr int T = StateSmem::kTile;
  uint8_t* sHi = smem + 4 * T;
  uint8_t* sLo = sHi + T;
  float* s_w = reinterpret_cast<float*>(sLo + T);  // [2][L]
  float* s_n = s_w + 2 * L;                         // [64]
  const bool fresh = a.base_len[b] == 0, owns_n = v0 == 0;
  const int64_t at = (int64_t)h * a.m_max + rs;
  float* S_g = a.S + ((int64_t)b * a.nh + h) * a.dim * a.vdim;
  float* n_g = a.n + ((int64_t)b * a.nh + h) * a.dim;

  float acc[4][4];
  auto each_state = [&](auto&& fn) {
#pragma unroll
    for (int nt = 0; nt < 4; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int d = d0 + dm + g + (e >> 1) * 8, v = v0 + vn + nt * 8 + t4 * 2 + (e & 1);
        fn(acc[nt][e], d < a.dim && v < a.vdim, (int64_t)d * a.vdim + v);
      }
  };
  each_state([&](float& s, bool in, int64_t off) { s = (in && !fresh) ? S_g[off] : 0.f; });
  if (tid < 64) s_n[tid] = (d0 + tid < a.dim && !fresh) ? n_g[d0 + tid] : 0.f;

  auto load = [&](int c) {
    uint8_t* sK = smem + (c & 1) * 2 * T;
#pragma unroll
    for (int i = 0; i < L * 8 / kThreads; ++i) {
      const int idx = i * kThreads + tid, r = idx >> 3, ch = idx & 7;
      const bool live = c * L + r < n_tok;
      const bool in_k = live && d0 + ch * 8 < a.dim, in_v = live && v0 + ch * 8 < a.vdim;
      const __nv_bfloat16* row = a.proj + (int64_t)(rs + (live ? c * L + r : 0)) * a.ld;
      cp_async16(sK + swz<8>(r, ch), row + (a.nh + h) * a.dim + (in_k ? d0 + ch * 8 : 0), in_k);
      cp_async16(sK + T + swz<8>(r, ch), row + 2 * a.nh * a.dim + h * a.vdim + (in_v ? v0 + ch * 8 : 0), in_v);
    }
    cp_async_commit();
    if (tid < L) s_w[(c & 1) * L + tid] = c * L + tid < n_tok ? a.w[at + c * L + tid] : 0.f;
  };
  load(0);
  for (int c = 0; c < n_chunks; ++c) {
    const int64_t slot = (int64_t)chunk_slot(rs, b, c) * a.nh + h;
    const float A = a.decay[slot];
    // the state at the chunk's start
    {
      uint32_t* hi = reinterpret_cast<uint32_t*>(a.Shi + slot * a.dpad * a.vpad);
      uint32_t* lo = reinterpret_cast<uint32_t*>(a.Slo + slot * a.dpad * a.vpad);
#pragma unroll
      for (int nt = 0; nt < 4; ++nt)
#pragma unroll
        for (int hh = 0; hh < 2; ++hh) {
          const int64_t off = ((int64_t)(d0 + dm + g + hh * 8) * a.vpad + v0 + vn + nt * 8 + t4 * 2) >> 1;
          uint32_t x, y;
          split2(acc[nt][hh * 2], acc[nt][hh * 2 + 1], x, y);
          hi[off] = x;
          lo[off] = y;
        }
    }
    cp_async_wait<0>();
    __syncthreads();  // chunk c is here; everyone has left chunk c - 1
    if (c + 1 < n_chunks) load(c + 1);
    const uint8_t* sK = smem + (c & 1) * 2 * T;
    const uint8_t* sV = sK + T;
    const float* w = s_w + (c & 1) * L;
#pragma unroll 4
    for (int i = 0; i < L * 32 / kThreads; ++i) {
      const int idx = i * kThreads + tid, r = idx >> 5, cc = (idx & 31) * 2;
      const int off = swz<8>(r, cc >> 3) + (cc & 7) * 2;
      const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(sV + off));
      split2(v.x * w[r], v.y * w[r], *reinterpret_cast<uint32_t*>(sHi + off), *reinterpret_cast<uint32_t*>(sLo + off));
    }
    if (owns_n) {
      // four threads per dim, 32 tokens each
      const int d = tid >> 2, part = tid & 3;
      float sum = 0.f;
#pragma unroll 8
      for (int j = part; j < L; j += 4)
        sum = fmaf(w[j], __bfloat162float(*reinterpret_cast<const __nv_bfloat16*>(sK + swz<8>(j, d >> 3) + (d & 7) * 2)), sum);
      sum += __shfl_xor_sync(0xffffffffu, sum, 1);
      sum += __shfl_xor_sync(0xffffffffu, sum, 2);
      if (part == 0) {
        a.nc[slot * a.dpad + d0 + d] = s_n[d];
        s_n[d] = fmaf(A, s_n[d], sum);  // this thread's alone
      }
    }
    __syncthreads();
#pragma unroll
    for (int nt = 0; nt < 4; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[nt][e] *= A;
#pragma unroll
    for (int kj = 0; kj < L / 16; ++kj) {
      uint32_t af[4];
      ldmatrix_x4_trans(af[0], af[1], af[2], af[3],
                        smem_addr(sK + swz<8>(kj * 16 + ((lane >> 4) << 3) + (lane & 7), (dm >> 3) + ((lane >> 3) & 1))));
#pragma unroll
      for (int nt = 0; nt < 4; nt += 2) {
        const int off = swz<8>(kj * 16 + (((lane >> 3) & 1) << 3) + (lane & 7), (vn >> 3) + nt + (lane >> 4));
        uint32_t b0, b1, b2, b3;
        ldmatrix_x4_trans(b0, b1, b2, b3, smem_addr(sHi + off));
        mma_bf16(acc[nt], af, b0, b1);
        mma_bf16(acc[nt + 1], af, b2, b3);
        ldmatrix_x4_trans(b0, b1, b2, b3, smem_addr(sLo + off));
        mma_bf16(acc[nt], af, b0, b1);
        mma_bf16(acc[nt + 1], af, b2, b3);
      }
    }
  }
  each_state([&](float& s, bool in, int64_t off) {
    if (in) S_g[off] = s;
  });
  if (owns_n && (tid & 3) == 0 && d0 + (tid >> 2) < a.dim) n_g[d0 + (tid >> 2)] = s_n[tid >> 2];
}

// ------------------------------------------------------------------------------------------------ outputs
constexpr int BT = 64;  // query tokens per CTA
constexpr int BK = 32;  // dims or tokens per streamed block

template <int DP, int WN>
struct OutSmem {
  static constexpr int kCols = WN * 64;
  static constexpr int kQ = BT * DP * 2, kK = L * DP * 2, kP = BT * L * 2;
  static constexpr int kBlock = BK * kCols * 2;    // one streamed block of one operand
  static constexpr int kStage = 2 * kBlock;        // hi and lo
  static constexpr int kRing = 2 * kStage > kK ? 2 * kStage : kK;  // K is dead once the scores are formed
  static constexpr int kMisc = (5 * BT + L + DP + 2 * BT + WN * BT) * 4;
  static constexpr int kBytes = kQ + 2 * kP + kRing + kMisc;
};

// grid (64-token tiles, nh, B).  WN warps along the value columns (64 each), 8 / WN along the tokens.
template <int DP, int WN>
__global__ void __launch_bounds__(kThreads, 1) mlstm_outputs_kernel(const ChunkArgs a) {
  using Y = OutSmem<DP, WN>;
  constexpr int WM = 8 / WN < 4 ? 8 / WN : 4;  // warps along the tokens
  constexpr int MT = 4 / WM;                   // 16-token tiles per warp
  constexpr int CQ = DP / 8, CP = L / 8, CB = Y::kCols / 8;
  extern __shared__ __align__(128) uint8_t smem[];
  rd::pdl_launch_dependents();
  rd::pdl_wait();
  const int b = blockIdx.z, h = blockIdx.y;
  const int rs = a.row_start[b], n_tok = a.row_start[b + 1] - rs;
  const int t0 = blockIdx.x * BT;  // first token of the tile within the row
  if (t0 >= n_tok) return;
  const int c = t0 / L, j0 = c * L, n_keys = t0 - j0 + BT;  // keys j0 .. j0 + n_keys - 1 (64 or 128)
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  const int64_t slot = (int64_t)chunk_slot(rs, b, c) * a.nh + h, at = (int64_t)h * a.m_max + rs;
  uint8_t* sQ = smem;
  uint8_t* sPh = sQ + Y::kQ;
  uint8_t* sPl = sPh + Y::kP;
  uint8_t* ring = sPl + Y::kP;
  uint8_t* sK = ring;
  float* s_Fm = reinterpret_cast<float*>(ring + Y::kRing);
  float* s_e = s_Fm + BT;
  float* s_floor = s_e + BT;
  float* s_nq = s_floor + BT;
  float* s_inv = s_nq + BT;
  float* s_iF = s_inv + BT;   // [L]
  float* s_n = s_iF + L;      // [DP]
  float* s_rs = s_n + DP;     // [2][BT]
  float* s_ss = s_rs + 2 * BT;  // [WN][BT]
  const float qs = rsqrtf((float)a.dim);

  for (int idx = tid; idx < BT * CQ; idx += kThreads) {
    const int r = idx / CQ, ch = idx % CQ;
    const bool in = t0 + r < n_tok && ch * 8 < a.dim;
    cp_async16(sQ + swz<CQ>(r, ch), a.proj + (int64_t)(rs + (in ? t0 + r : 0)) * a.ld + h * a.dim + (in ? ch * 8 : 0), in);
  }
  for (int idx = tid; idx < n_keys * CQ; idx += kThreads) {
    const int r = idx / CQ, ch = idx % CQ;
    const bool in = j0 + r < n_tok && ch * 8 < a.dim;
    cp_async16(sK + swz<CQ>(r, ch), a.proj + (int64_t)(rs + (in ? j0 + r : 0)) * a.ld + (a.nh + h) * a.dim + (in ? ch * 8 : 0), in);
  }
  cp_async_commit();
  if (tid < BT) {
    const bool in = t0 + tid < n_tok;
    s_Fm[tid] = in ? a.Fm[at + t0 + tid] : 0.f;
    s_e[tid] = in ? a.e[at + t0 + tid] : 0.f;
    s_floor[tid] = in ? a.floor[at + t0 + tid] : 1.f;
  }
  if (tid < L) s_iF[tid] = (tid < n_keys && j0 + tid < n_tok) ? a.iF[at + j0 + tid] : -INFINITY;
  for (int d = tid; d < DP; d += kThreads) s_n[d] = d < a.dpad ? a.nc[slot * a.dpad + d] : 0.f;
  cp_async_wait<0>();
  __syncthreads();

  // ---- P = (Q K^T) o weights: warp -> 16 tokens x half of the keys
  {
    const int tw = (warp & 3) * 16, half = n_keys / 2, jw = (warp >> 2) * half;
    const bool first_half = n_keys == BT;  // the chunk's first 64 tokens: keys and queries coincide
    float s[8][4];
#pragma unroll
    for (int nt = 0; nt < 8; ++nt) s[nt][0] = s[nt][1] = s[nt][2] = s[nt][3] = 0.f;
    const int n_nt = half / 8;  // 4 or 8
    const int q_off = first_half ? 0 : BT;
    if (jw <= tw + 15 + q_off) {
#pragma unroll 2
      for (int kd = 0; kd < DP / 16; ++kd) {
        uint32_t af[4];
        ldmatrix_x4(af[0], af[1], af[2], af[3], smem_addr(sQ + swz<CQ>(tw + (lane & 15), kd * 2 + (lane >> 4))));
#pragma unroll
        for (int nb = 0; nb < 8; nb += 2) {
          if (nb < n_nt) {
            uint32_t b0, b1, b2, b3;
            ldmatrix_x4(b0, b1, b2, b3, smem_addr(sK + swz<CQ>(jw + nb * 8 + ((lane >> 4) << 3) + (lane & 7), kd * 2 + ((lane >> 3) & 1))));
            mma_bf16(s[nb], af, b0, b1);
            mma_bf16(s[nb + 1], af, b2, b3);
          }
        }
      }
    }
#pragma unroll
    for (int hh = 0; hh < 2; ++hh) {
      const int t = tw + g + hh * 8, tk = t + q_off;  // tk: the query's place among the keys
      const float Fm = s_Fm[t];
      float sum = 0.f;
#pragma unroll
      for (int nt = 0; nt < 8; ++nt)
        if (nt < n_nt) {
          const int j = jw + nt * 8 + t4 * 2;
          const float p0 = j <= tk ? s[nt][hh * 2] * qs * expf(Fm + s_iF[j]) : 0.f;
          const float p1 = j + 1 <= tk ? s[nt][hh * 2 + 1] * qs * expf(Fm + s_iF[j + 1]) : 0.f;
          sum += p0 + p1;
          const int off = swz<CP>(t, j >> 3) + (j & 7) * 2;
          split2(p0, p1, *reinterpret_cast<uint32_t*>(sPh + off), *reinterpret_cast<uint32_t*>(sPl + off));
        }
      sum += __shfl_xor_sync(0xffffffffu, sum, 1);
      sum += __shfl_xor_sync(0xffffffffu, sum, 2);
      if (t4 == 0) s_rs[(warp >> 2) * BT + t] = sum;
    }
  }
  // ---- n_in . q_t: four threads per token
  {
    const int t = tid >> 2, part = tid & 3;
    float acc = 0.f;
#pragma unroll 2
    for (int ch = part; ch < CQ; ch += 4) {
      const uint4 u = *reinterpret_cast<const uint4*>(sQ + swz<CQ>(t, ch));
      const __nv_bfloat162* q2 = reinterpret_cast<const __nv_bfloat162*>(&u);
      const float4 n0 = *reinterpret_cast<const float4*>(s_n + ch * 8), n1 = *reinterpret_cast<const float4*>(s_n + ch * 8 + 4);
      const float2 f0 = __bfloat1622float2(q2[0]), f1 = __bfloat1622float2(q2[1]);
      const float2 f2 = __bfloat1622float2(q2[2]), f3 = __bfloat1622float2(q2[3]);
      acc = fmaf(f0.x, n0.x, fmaf(f0.y, n0.y, fmaf(f1.x, n0.z, fmaf(f1.y, n0.w, acc))));
      acc = fmaf(f2.x, n1.x, fmaf(f2.y, n1.y, fmaf(f3.x, n1.z, fmaf(f3.y, n1.w, acc))));
    }
    acc += __shfl_xor_sync(0xffffffffu, acc, 1);
    acc += __shfl_xor_sync(0xffffffffu, acc, 2);
    if (part == 0) s_nq[t] = acc;
  }
  __syncthreads();  // P is complete, K is dead
  if (tid < BT) {
    const float den = s_rs[tid] + s_rs[BT + tid] + s_e[tid] * s_nq[tid];
    s_inv[tid] = 1.0f / (fmaxf(fabsf(den), s_floor[tid]) + kDenEps);
  }

  // ---- O = e_t Q S + P V, the second operands streamed in blocks of 32 rows
  const int n_dim = (a.dpad < DP ? a.dpad : DP) / BK, n_blocks = n_dim + n_keys / BK;
  auto load = [&](int blk) {
    if (blk < n_blocks) {
      uint8_t* dst = ring + (blk & 1) * Y::kStage;
      if (blk < n_dim) {
        const __nv_bfloat16* hi = a.Shi + (slot * a.dpad + blk * BK) * a.vpad;
        const __nv_bfloat16* lo = a.Slo + (slot * a.dpad + blk * BK) * a.vpad;
#pragma unroll
        for (int i = 0; i < BK * CB / kThreads; ++i) {
          const int idx = i * kThreads + tid, r = idx / CB, ch = idx % CB;
          const bool in = ch * 8 < a.vpad;
          const int64_t off = (int64_t)r * a.vpad + (in ? ch * 8 : 0);
          cp_async16(dst + swz<CB>(r, ch), hi + off, in);
          cp_async16(dst + Y::kBlock + swz<CB>(r, ch), lo + off, in);
        }
      } else {
        const int jb = j0 + (blk - n_dim) * BK;
#pragma unroll
        for (int i = 0; i < BK * CB / kThreads; ++i) {
          const int idx = i * kThreads + tid, r = idx / CB, ch = idx % CB;
          const bool in = jb + r < n_tok && ch * 8 < a.vdim;
          cp_async16(dst + swz<CB>(r, ch),
                     a.proj + (int64_t)(rs + (in ? jb + r : 0)) * a.ld + 2 * a.nh * a.dim + h * a.vdim + (in ? ch * 8 : 0), in);
        }
      }
    }
    cp_async_commit();
  };
  const int wn = warp % WN, wm = warp / WN;
  const bool works = wm < WM;  // WN == 1 would leave warps idle; WN >= 2 uses all eight
  float o[MT][8][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int nt = 0; nt < 8; ++nt) o[m][nt][0] = o[m][nt][1] = o[m][nt][2] = o[m][nt][3] = 0.f;
  load(0);
  for (int blk = 0; blk < n_blocks; ++blk) {
    cp_async_wait<0>();
    __syncthreads();  // block blk is here; everyone has left block blk - 1
    load(blk + 1);
    if (!works) continue;
    const uint8_t* sB = ring + (blk & 1) * Y::kStage;
    if (blk == n_dim) {
      // the state's part is complete: scale it before the scores' part is added
#pragma unroll
      for (int m = 0; m < MT; ++m) {
        const float e0 = s_e[(wm * MT + m) * 16 + g], e1 = s_e[(wm * MT + m) * 16 + g + 8];
#pragma unroll
        for (int nt = 0; nt < 8; ++nt) {
          o[m][nt][0] *= e0;
          o[m][nt][1] *= e0;
          o[m][nt][2] *= e1;
          o[m][nt][3] *= e1;
        }
      }
    }
    const bool state = blk < n_dim;
#pragma unroll
    for (int k16 = 0; k16 < BK / 16; ++k16) {
      const int row = k16 * 16 + (((lane >> 3) & 1) << 3) + (lane & 7);
      if (state) {
        uint32_t af[MT][4];
#pragma unroll
        for (int m = 0; m < MT; ++m)
          ldmatrix_x4(af[m][0], af[m][1], af[m][2], af[m][3],
                      smem_addr(sQ + swz<CQ>((wm * MT + m) * 16 + (lane & 15), blk * (BK / 8) + k16 * 2 + (lane >> 4))));
#pragma unroll
        for (int nt = 0; nt < 8; nt += 2) {
          const int off = swz<CB>(row, wn * 8 + nt + (lane >> 4));
          uint32_t b0, b1, b2, b3;
          ldmatrix_x4_trans(b0, b1, b2, b3, smem_addr(sB + off));
#pragma unroll
          for (int m = 0; m < MT; ++m) {
            mma_bf16(o[m][nt], af[m], b0, b1);
            mma_bf16(o[m][nt + 1], af[m], b2, b3);
          }
          ldmatrix_x4_trans(b0, b1, b2, b3, smem_addr(sB + Y::kBlock + off));
#pragma unroll
          for (int m = 0; m < MT; ++m) {
            mma_bf16(o[m][nt], af[m], b0, b1);
            mma_bf16(o[m][nt + 1], af[m], b2, b3);
          }
        }
      } else {
#pragma unroll
        for (int part = 0; part < 2; ++part) {
          const uint8_t* sP = part ? sPl : sPh;
          uint32_t af[MT][4];
#pragma unroll
          for (int m = 0; m < MT; ++m)
            ldmatrix_x4(af[m][0], af[m][1], af[m][2], af[m][3],
                        smem_addr(sP + swz<CP>((wm * MT + m) * 16 + (lane & 15), (blk - n_dim) * (BK / 8) + k16 * 2 + (lane >> 4))));
#pragma unroll
          for (int nt = 0; nt < 8; nt += 2) {
            uint32_t b0, b1, b2, b3;
            ldmatrix_x4_trans(b0, b1, b2, b3, smem_addr(sB + swz<CB>(row, wn * 8 + nt + (lane >> 4))));
#pragma unroll
            for (int m = 0; m < MT; ++m) {
              mma_bf16(o[m][nt], af[m], b0, b1);
              mma_bf16(o[m][nt + 1], af[m], b2, b3);
            }
          }
        }
      }
    }
  }
  cp_async_wait<0>();

  // ---- o / denominator, RMS over the head, norm weight, output gate
  if (works) {
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int hh = 0; hh < 2; ++hh) {
        const int t = (wm * MT + m) * 16 + g + hh * 8;
        const float inv = s_inv[t];
        float ss = 0.f;
#pragma unroll
        for (int nt = 0; nt < 8; ++nt) {
          o[m][nt][hh * 2] *= inv;
          o[m][nt][hh * 2 + 1] *= inv;
          ss = fmaf(o[m][nt][hh * 2], o[m][nt][hh * 2], ss);
          ss = fmaf(o[m][nt][hh * 2 + 1], o[m][nt][hh * 2 + 1], ss);
        }
        ss += __shfl_xor_sync(0xffffffffu, ss, 1);
        ss += __shfl_xor_sync(0xffffffffu, ss, 2);
        if (t4 == 0) s_ss[wn * BT + t] = ss;
      }
  }
  __syncthreads();
  if (!works) return;
  const __nv_bfloat16* w_h = a.norm_w + (int64_t)h * a.vdim;
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int hh = 0; hh < 2; ++hh) {
      const int t = (wm * MT + m) * 16 + g + hh * 8;
      if (t0 + t >= n_tok) continue;
      float ss = 0.f;
#pragma unroll
      for (int k = 0; k < WN; ++k) ss += s_ss[k * BT + t];
      const float r = 1.0f / sqrtf(ss / (float)a.vdim + a.eps);
      const int64_t tok = rs + t0 + t;
      const __nv_bfloat16* gp = a.proj + tok * a.ld + 2 * a.nh * a.dim + (a.nh + h) * a.vdim;
      __nv_bfloat16* dst = a.out + (tok * a.nh + h) * a.vdim;
#pragma unroll
      for (int nt = 0; nt < 8; ++nt) {
        const int v = wn * 64 + nt * 8 + t4 * 2;
        if (v < a.vdim) {
          const float2 gg = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(gp + v));
          const float2 ww = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(w_h + v));
          *reinterpret_cast<uint32_t*>(dst + v) = pack_bf16(o[m][nt][hh * 2] * r * ww.x / (1.f + __expf(-gg.x)),
                                                            o[m][nt][hh * 2 + 1] * r * ww.y / (1.f + __expf(-gg.y)));
        }
      }
    }
}

template <int DP, int WN>
int launch_outputs(const ChunkArgs& a, int B, int max_new, cudaStream_t s) {
  auto kern = mlstm_outputs_kernel<DP, WN>;
  constexpr int smem = OutSmem<DP, WN>::kBytes;
  static bool set = false;
  if (!set) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    RD_CHECK_CHAINED(e);
    set = true;
  }
  cudaError_t err = rd::launch_chained(kern, dim3((max_new + BT - 1) / BT, a.nh, B), dim3(kThreads), smem, s, 1, a);
  RD_CHECK_CHAINED(err);
  return RD_OK;
}

template <int DP>
int launch_outputs_dim(const ChunkArgs& a, int B, int max_new, cudaStream_t s) {
  if (a.vdim <= 128) return launch_outputs<DP, 2>(a, B, max_new, s);
  if (a.vdim <= 256) return launch_outputs<DP, 4>(a, B, max_new, s);
  return launch_outputs<DP, 8>(a, B, max_new, s);
}

inline int64_t pad64(int64_t n) { return (n + 63) / 64 * 64; }
inline int64_t slots_of(int64_t m_max, int64_t B) { return m_max / L + B; }

}  // namespace

extern "C" int64_t rd_mlstm_chunk_workspace_bytes(int m_max, int B, int nh, int dim, int vdim) {
  const int64_t slots = slots_of(m_max, B) * nh;
  return slots * pad64(dim) * pad64(vdim) * 4 + (5 * (int64_t)nh * m_max + slots * (1 + pad64(dim)) + 64) * (int64_t)sizeof(float);
}

extern "C" int rd_mlstm_chunk(const void* proj, int64_t ld, const float* gates, int64_t ld_gates, const float* bias_i,
                              const float* bias_f, float gate_cap, const void* norm_weight, float eps, void* out, float* S,
                              float* n, float* m, const int32_t* row_start, const int32_t* base_len, int B, int nh, int dim,
                              int vdim, int m_max, int max_new, void* workspace, int64_t workspace_bytes, void* stream) {
  RD_REQUIRE(proj && gates && bias_i && bias_f && norm_weight && out && S && n && m && row_start && base_len && workspace, RD_ERR_ARG);
  RD_REQUIRE(B >= 1 && B <= 65535 && nh >= 1 && nh <= 65535 && dim >= 8 && dim <= 256 && dim % 8 == 0 && vdim >= 8 && vdim <= 512 &&
                 vdim % 8 == 0 && m_max >= 1 && max_new >= 1 && max_new <= m_max && gate_cap > 0.f &&
                 ld >= 2 * (int64_t)nh * (dim + vdim) && ld_gates >= 2 * nh,
             RD_ERR_SIZE);
  RD_REQUIRE((((uintptr_t)proj | (uintptr_t)norm_weight | (uintptr_t)out | (uintptr_t)workspace) & 15) == 0 && ld % 8 == 0, RD_ERR_ALIGN);
  RD_REQUIRE(workspace_bytes >= rd_mlstm_chunk_workspace_bytes(m_max, B, nh, dim, vdim), RD_ERR_CAPACITY);
  ChunkArgs a{};
  a.proj = (const __nv_bfloat16*)proj;
  a.ld = ld;
  a.gates = gates;
  a.ld_gates = ld_gates;
  a.bias_i = bias_i;
  a.bias_f = bias_f;
  a.cap = gate_cap;
  a.norm_w = (const __nv_bfloat16*)norm_weight;
  a.eps = eps;
  a.out = (__nv_bfloat16*)out;
  a.S = S;
  a.n = n;
  a.m = m;
  a.row_start = row_start;
  a.base_len = base_len;
  a.nh = nh;
  a.dim = dim;
  a.vdim = vdim;
  a.dpad = (int)pad64(dim);
  a.vpad = (int)pad64(vdim);
  a.m_max = m_max;
  const int64_t slots = slots_of(m_max, B) * nh, tile = (int64_t)a.dpad * a.vpad;
  a.Shi = (__nv_bfloat16*)workspace;
  a.Slo = a.Shi + slots * tile;
  float* f = (float*)(a.Slo + slots * tile);
  a.nc = f;
  a.decay = a.nc + slots * a.dpad;
  f = a.decay + slots;
  for (float** p : {&a.Fm, &a.iF, &a.e, &a.w, &a.floor}) {
    *p = f;
    f += (int64_t)nh * m_max;
  }
  cudaStream_t s = (cudaStream_t)stream;
  const size_t gates_smem = (size_t)3 * ((max_new + L - 1) / L) * sizeof(float);
  RD_REQUIRE(gates_smem <= 48 * 1024, RD_ERR_SIZE);
  cudaError_t err = rd::launch_chained(mlstm_gates_kernel, dim3(nh, B), dim3(kThreads), gates_smem, s, 1, a);
  RD_CHECK_CHAINED(err);
  static bool set = false;
  if (!set) {
    err = cudaFuncSetAttribute(mlstm_states_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, StateSmem::kBytes);
    RD_CHECK_CHAINED(err);
    set = true;
  }
  err = rd::launch_chained(mlstm_states_kernel, dim3((a.dpad / 64) * (a.vpad / 64), nh, B), dim3(kThreads), StateSmem::kBytes, s, 1, a);
  RD_CHECK_CHAINED(err);
  if (dim <= 64) return launch_outputs_dim<64>(a, B, max_new, s);
  if (dim <= 128) return launch_outputs_dim<128>(a, B, max_new, s);
  return launch_outputs_dim<256>(a, B, max_new, s);
}
