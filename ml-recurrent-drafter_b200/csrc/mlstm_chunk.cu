// The matrix-memory recurrence of mlstm.cu for prompts: chunks of 128 tokens on the tensor cores (tcgen05, bf16 operands,
// fp32 accumulators in TMEM; operands staged by TMA, or by cp.async where a tile's edge must be zero).  Waits are bounded: on give-up a
// kernel writes a code to *status, frees its TMEM and returns.
//
// Within a chunk, with F_t the running sum of the log forget gates and m_t the running maximum of the recurrence,
//   m_t   = F_t + max(m_in, max_{j <= t} (i_j - F_j))
//   P_tj  = (q_t . k_j) e^(F_t - F_j + i_j - m_t)                       j <= t
//   num_t = sum_j P_tj v_j + e^(F_t + m_in - m_t) S_in^T q_t,   den_t = sum_j P_tj + e^(F_t + m_in - m_t) n_in . q_t
//   S_out = e^(F_L + m_in - m_L) S_in + sum_j e^(F_L - F_j + i_j - m_L) k_j v_j^T      (n likewise with k alone)
// so every exponent is <= 0, and the result is the token-by-token recurrence up to rounding.  Three kernels:
//   gates    one CTA per (head, row): the scalars above for every token; only the chunks' maxima follow one another
//   states   one CTA per 128 value columns x 64 dims of S: walks the chunks, the tile in TMEM (fp32), and leaves S and n
//            at the start of every chunk in the workspace
//   outputs  one CTA per chunk of a head: scores, both products (accumulated in TMEM), the head's RMS norm, the norm
//            weight and the output gate, independent of all other chunks
// The fp32 operands of the products - P, S and what enters the state, e^(...) v_j - are each split into two bf16 parts
// (their rounding error is then about 2^-17).
#include "mlstm_common.cuh"
#include "mma_sync.cuh"
#include "umma.cuh"

namespace {

using namespace rd_mma;
using namespace rd_mlstm;

constexpr int L = 128;  // tokens per chunk

// Bounded wait by whole warps; the answer is the same for all lanes.
__device__ __forceinline__ bool wait_warp(uint64_t* bar, uint32_t parity) {
  return __all_sync(0xffffffffu, rd_umma::mbar_wait(bar, parity));
}
constexpr int kThreads = 512;
constexpr int kGateThreads = 1024;

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
  int32_t* status;
  // workspace.  Per head and token [nh][m_max]:
  float* Fm;     // F_t - m_t
  float* iF;     // i_j - F_j
  float* e;      // dim^(-1/2) e^(F_t + m_in - m_t)
  float* w;      // e^(F_L - F_j + i_j - m_L)
  float* floor;  // e^(-m_t)
  // per chunk slot and head; row b's chunk c has slot row_start[b] / L + b + c
  float* decay;  // e^(F_L + m_in - m_L)
  float* nc;     // [dpad] n at the chunk's start
  __nv_bfloat16* Shi;  // [vpad][dpad] S^T at the chunk's start
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
__global__ void __launch_bounds__(kGateThreads) mlstm_gates_kernel(const ChunkArgs a) {
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
  for (int c = warp; c < n_chunks; c += kGateThreads / 32) {
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
  for (int c = warp; c < n_chunks; c += kGateThreads / 32) {
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
// Rows of a [128 x 64] box are 128 bytes, 16-byte chunks permuted by the row: the tensor core's 128-byte swizzle.
constexpr int kBox = 128 * 128;  // bytes

constexpr int DN = 64;  // dims per CTA of the states kernel

struct StateSmem {
  static constexpr int kK = kBox, kV = 2 * kBox;  // [128 tokens] x 64 dims, x 128 value columns
  static constexpr int kStage = kK + kV;
  static constexpr int kMisc = (2 * L + DN + 8) * 4 + 64;  // w, n, barriers
  static constexpr int kBytes = 2 * kStage + 2 * kV + 2 * kBox + kMisc + 1024;  // two stages, w V and S^T as hi and lo, alignment
};

// grid (value tiles of 128 * dim tiles of DN, nh, B).  S^T tile [128 value columns = TMEM lanes][DN dims = TMEM columns].
// Per chunk: the tile is read out, stored to the workspace (TMA), scaled and put back, then (w V)^T K is added by tcgen05.mma
// (both operands MN-major: value columns and dims contiguous, tokens along K).
__global__ void __launch_bounds__(kThreads, 1) mlstm_states_kernel(const __grid_constant__ CUtensorMap map_proj,
                                                                   const __grid_constant__ CUtensorMap map_hi,
                                                                   const __grid_constant__ CUtensorMap map_lo, const ChunkArgs a) {
  using Y = StateSmem;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  rd::pdl_launch_dependents();
  rd::pdl_wait();
  const int b = blockIdx.z, h = blockIdx.y;
  const int d_tiles = a.dpad / DN;
  const int v0 = (blockIdx.x / d_tiles) * 128, d0 = (blockIdx.x % d_tiles) * DN;
  const int rs = a.row_start[b], n_tok = a.row_start[b + 1] - rs;
  if (n_tok <= 0) return;
  const int n_chunks = (n_tok + L - 1) / L;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  uint8_t* sHi = smem + 2 * Y::kStage;
  uint8_t* sLo = sHi + Y::kV;
  uint8_t* sShi = sLo + Y::kV;  // the tile on its way to the workspace
  uint8_t* sSlo = sShi + kBox;
  float* s_w = reinterpret_cast<float*>(sSlo + kBox);  // [2][L]
  float* s_n = s_w + 2 * L;                             // [DN]
  uint64_t* bar = reinterpret_cast<uint64_t*>(s_n + DN);  // a chunk's products are done
  uint64_t* full = bar + 1;                               // [2] a stage's K and V have landed
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bar + 3);
  if (tid == 0) {
    for (int i = 0; i < 3; ++i) rd_umma::mbar_init(&bar[i], 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 0) rd_umma::tmem_alloc(tmem_slot, DN);
  const bool fresh = a.base_len[b] == 0, owns_n = v0 == 0;
  const int64_t at = (int64_t)h * a.m_max + rs;
  float* S_g = a.S + ((int64_t)b * a.nh + h) * a.dim * a.vdim;
  float* n_g = a.n + ((int64_t)b * a.nh + h) * a.dim;
  if (tid < DN) s_n[tid] = (d0 + tid < a.dim && !fresh) ? n_g[d0 + tid] : 0.f;

  // One thread: K and V of chunk c by TMA.  Boxes may reach into the next row's tokens (their w is 0 and they are finite),
  // into the next head's dims (never read from the state: q is zero there) or columns (never stored).
  auto load = [&](int c) {
    uint8_t* sK = smem + (c & 1) * Y::kStage;
    rd_umma::mbar_expect_tx(&full[c & 1], Y::kStage);
    const int row = rs + c * L, k0 = (a.nh + h) * a.dim + d0, w0 = 2 * a.nh * a.dim + h * a.vdim + v0;
    rd_umma::tma_load_2d(sK, &map_proj, &full[c & 1], k0, row);
#pragma unroll
    for (int i = 0; i < 2; ++i) rd_umma::tma_load_2d(sK + Y::kK + i * kBox, &map_proj, &full[c & 1], w0 + i * 64, row);
  };
  auto w_of = [&](int c) { return (tid < L && c * L + tid < n_tok) ? a.w[at + c * L + tid] : 0.f; };
  auto decay_of = [&](int c) { return a.decay[(int64_t)chunk_slot(rs, b, c) * a.nh + h]; };
  if (tid < L) s_w[tid] = w_of(0);
  float A = decay_of(0);
  rd_umma::fence_before();
  __syncthreads();
  rd_umma::fence_after();
  if (tid == 0) load(0);  // the barriers are initialised
  const uint32_t tmem = *tmem_slot;
  const int quarter = warp & 3, cg = warp >> 2;
  const int v = v0 + quarter * 32 + lane, dq = d0 + cg * 32;  // this thread's value column and its 32 dims
  const bool has_tile = cg * 32 < DN;                         // half of the warps
  const uint32_t t_row = tmem + ((uint32_t)(quarter * 32) << 16) + cg * 32;
  bool ok = true;

  for (int c = 0; c < n_chunks; ++c) {
    // the products of chunk c - 1 are in the tile, and its operands' shared memory is free
    if (c > 0) ok = wait_warp(bar, (c - 1) & 1);
    if (tid == 0) rd_umma::tma_store_wait_read();
    if (!__syncthreads_and(ok)) break;
    if (tid == 0 && c + 1 < n_chunks) load(c + 1);
    ok = wait_warp(&full[c & 1], (c >> 1) & 1);
    rd_umma::fence_after();
    const float w_next = c + 1 < n_chunks ? w_of(c + 1) : 0.f, A_next = c + 1 < n_chunks ? decay_of(c + 1) : 0.f;
    const uint8_t* sK = smem + (c & 1) * Y::kStage;
    const uint8_t* sV = sK + Y::kK;
    const float* w = s_w + (c & 1) * L;
    const int64_t slot = (int64_t)chunk_slot(rs, b, c) * a.nh + h;
    // the state at the chunk's start goes to the workspace; scaled, it becomes the accumulator of this chunk's products
    if (has_tile) {
      float s[32];
      if (c == 0) {
#pragma unroll
        for (int i = 0; i < 32; ++i) s[i] = (!fresh && v < a.vdim && dq + i < a.dim) ? S_g[(int64_t)(dq + i) * a.vdim + v] : 0.f;
      } else {
        rd_umma::tmem_ld32(t_row, s);
      }
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        uint4 hi, lo;
        split2(s[8 * i], s[8 * i + 1], hi.x, lo.x);
        split2(s[8 * i + 2], s[8 * i + 3], hi.y, lo.y);
        split2(s[8 * i + 4], s[8 * i + 5], hi.z, lo.z);
        split2(s[8 * i + 6], s[8 * i + 7], hi.w, lo.w);
        const int off = swz<8>(quarter * 32 + lane, cg * 4 + i);
        *reinterpret_cast<uint4*>(sShi + off) = hi;
        *reinterpret_cast<uint4*>(sSlo + off) = lo;
      }
#pragma unroll
      for (int i = 0; i < 32; ++i) s[i] *= A;
      rd_umma::tmem_st32(t_row, s);
    }
    // w_j v_j as hi + lo, in the same swizzled boxes
#pragma unroll 4
    for (int i = tid; i < L * 16; i += kThreads) {
      const int r = i >> 4, ch = i & 15;
      const int off = (ch >> 3) * kBox + swz<8>(r, ch & 7);
      const float wr = w[r];
      const uint4 u = *reinterpret_cast<const uint4*>(sV + off);
      const __nv_bfloat162* x2 = reinterpret_cast<const __nv_bfloat162*>(&u);
      uint4 hi, lo;
      uint32_t* hp = reinterpret_cast<uint32_t*>(&hi);
      uint32_t* lp = reinterpret_cast<uint32_t*>(&lo);
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float2 f = __bfloat1622float2(x2[e]);
        split2(f.x * wr, f.y * wr, hp[e], lp[e]);
      }
      *reinterpret_cast<uint4*>(sHi + off) = hi;
      *reinterpret_cast<uint4*>(sLo + off) = lo;
    }
    rd_umma::fence_async_proxy();
    rd_umma::fence_before();
    if (!__syncthreads_and(ok)) {
      ok = false;
      break;
    }
    if (tid == 0) {
      rd_umma::fence_after();
      const uint32_t idesc = rd_umma::idesc_f16(DN, true, true);
#pragma unroll
      for (int k = 0; k < L / 16; ++k) {
        const uint64_t dk = rd_umma::desc_mn_major(rd_umma::smem_u32(sK + k * 2048), kBox);
        rd_umma::mma_ss(tmem, rd_umma::desc_mn_major(rd_umma::smem_u32(sHi + k * 2048), kBox), dk, idesc, 1);
        rd_umma::mma_ss(tmem, rd_umma::desc_mn_major(rd_umma::smem_u32(sLo + k * 2048), kBox), dk, idesc, 1);
      }
      rd_umma::commit(bar);
      rd_umma::tma_store_2d(&map_hi, sShi, d0, (int)(slot * a.vpad) + v0);
      rd_umma::tma_store_2d(&map_lo, sSlo, d0, (int)(slot * a.vpad) + v0);
      rd_umma::tma_store_commit();
    }
    if (owns_n) {
      // n of this tile's dims: kThreads / DN threads per dim
      constexpr int PER = kThreads / DN;
      const int d = tid / PER, part = tid % PER;
      float sum = 0.f;
#pragma unroll 8
      for (int j = part; j < L; j += PER)
        sum = fmaf(w[j], __bfloat162float(*reinterpret_cast<const __nv_bfloat16*>(sK + swz<8>(j, d >> 3) + (d & 7) * 2)), sum);
#pragma unroll
      for (int o = 1; o < PER; o <<= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
      if (part == 0) {
        a.nc[slot * a.dpad + d0 + d] = s_n[d];
        s_n[d] = fmaf(A, s_n[d], sum);  // this thread's alone
      }
    }
    if (tid < L) s_w[((c + 1) & 1) * L + tid] = w_next;
    A = A_next;
  }
  if (tid == 0) rd_umma::tma_store_wait();
  if (ok) ok = wait_warp(bar, (n_chunks - 1) & 1);
  ok = __syncthreads_and(ok);
  if (ok) {
    rd_umma::fence_after();
    if (has_tile) {
      float s[32];
      rd_umma::tmem_ld32(t_row, s);
#pragma unroll
      for (int i = 0; i < 32; ++i)
        if (v < a.vdim && dq + i < a.dim) S_g[(int64_t)(dq + i) * a.vdim + v] = s[i];
    }
    constexpr int PER = kThreads / DN;
    if (owns_n && tid % PER == 0 && d0 + tid / PER < a.dim) n_g[d0 + tid / PER] = s_n[tid / PER];
  } else if (tid == 0) {
    if (a.status) atomicExch(a.status, 31);
    for (int i = 0; i < 2000; ++i) __nanosleep(1000);  // copies in flight land before the shared memory goes away
  }
  rd_umma::fence_before();
  __syncthreads();
  if (warp == 0) {
    rd_umma::fence_after();
    rd_umma::tmem_dealloc(tmem, DN);
  }
}

// ------------------------------------------------------------------------------------------------ outputs
constexpr int kOutStages = 4;
constexpr int kItem = kBox;  // bytes of one streamed operand tile: [128 value columns x 64 dims] or [64 tokens x 128 value columns]

template <int DP>
struct OutSmem {
  static constexpr int kQ = (DP / 64) * kBox;
  static constexpr int kRing = kOutStages * kItem > kQ ? kOutStages * kItem : kQ;  // K first, then the ring
  static constexpr int kP = 2 * kBox;
  static constexpr int kMisc = (5 * L + DP + 8 * L) * 4 + 160;  // per-token scalars, n, barriers
  static constexpr int kBytes = kQ + kRing + 2 * kP + kMisc + 1024;
};

// grid (chunks, nh, B).  O [128 tokens = TMEM lanes][value columns = TMEM columns]:
//   scores Q K^T (in O's columns, before O exists) -> P hi / lo in shared memory -> O = Q S (hi, lo) -> O *= e_t ->
//   O += P V (hi, lo) -> / denominator, RMS, norm weight, output gate.
template <int DP>
__global__ void __launch_bounds__(kThreads, 1) mlstm_outputs_kernel(const __grid_constant__ CUtensorMap map_v,
                                                                    const __grid_constant__ CUtensorMap map_hi,
                                                                    const __grid_constant__ CUtensorMap map_lo, const ChunkArgs a) {
  using Y = OutSmem<DP>;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  rd::pdl_launch_dependents();
  rd::pdl_wait();
  const int b = blockIdx.z, h = blockIdx.y, c = blockIdx.x;
  const int rs = a.row_start[b], n_tok = a.row_start[b + 1] - rs;
  const int t0 = c * L;
  if (t0 >= n_tok) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int64_t slot = (int64_t)chunk_slot(rs, b, c) * a.nh + h, at = (int64_t)h * a.m_max + rs;
  uint8_t* sQ = smem;
  uint8_t* ring = sQ + Y::kQ;
  uint8_t* sPh = ring + Y::kRing;
  uint8_t* sPl = sPh + Y::kP;
  float* s_Fm = reinterpret_cast<float*>(sPl + Y::kP);
  float* s_iF = s_Fm + L;
  float* s_e = s_iF + L;
  float* s_floor = s_e + L;
  float* s_nq = s_floor + L;
  float* s_n = s_nq + L;       // [DP]
  float* s_rs = s_n + DP;      // [4][L]
  float* s_ss = s_rs + 4 * L;  // [4][L]
  uint64_t* bars = reinterpret_cast<uint64_t*>(s_ss + 4 * L);  // [kOutStages] an item's products are done
  uint64_t* full = bars + kOutStages;                           // [kOutStages] an item has landed
  uint64_t* scores_done = full + kOutStages;
  uint64_t* state_done = scores_done + 1;
  uint64_t* all_done = scores_done + 2;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(scores_done + 3);
  const uint32_t n_cols = a.vpad <= 128 ? 128 : (a.vpad <= 256 ? 256 : 512);
  if (tid == 0) {
    for (int i = 0; i < 2 * kOutStages + 3; ++i) rd_umma::mbar_init(&bars[i], 1);
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 0) rd_umma::tmem_alloc(tmem_slot, n_cols);
  const float qs = rsqrtf((float)a.dim);

  for (int i = tid; i < L * (DP / 8); i += kThreads) {
    const int r = i / (DP / 8), ch = i % (DP / 8);
    const bool in = t0 + r < n_tok && ch * 8 < a.dim;
    const __nv_bfloat16* src = a.proj + (int64_t)(rs + (in ? t0 + r : 0)) * a.ld + h * a.dim + (in ? ch * 8 : 0);
    const int off = (ch >> 3) * kBox + swz<8>(r, ch & 7);
    cp_async16(sQ + off, src, in);
    cp_async16(ring + off, src + a.nh * a.dim, in);
  }
  cp_async_commit();
  if (tid < L) {
    const bool in = t0 + tid < n_tok;
    s_Fm[tid] = in ? a.Fm[at + t0 + tid] : 0.f;
    s_iF[tid] = in ? a.iF[at + t0 + tid] : -INFINITY;
    s_e[tid] = in ? a.e[at + t0 + tid] : 0.f;
    s_floor[tid] = in ? a.floor[at + t0 + tid] : 1.f;
  }
  for (int d = tid; d < DP; d += kThreads) s_n[d] = d < a.dpad ? a.nc[slot * a.dpad + d] : 0.f;
  cp_async_wait<0>();
  rd_umma::fence_async_proxy();
  rd_umma::fence_before();
  __syncthreads();
  rd_umma::fence_after();
  const uint32_t tmem = *tmem_slot;
  if (tid == 0) {
    const uint32_t idesc = rd_umma::idesc_f16(128, false, false);
#pragma unroll
    for (int k = 0; k < DP / 16; ++k) {
      const int off = (k >> 2) * kBox + (k & 3) * 32;
      rd_umma::mma_ss(tmem, rd_umma::desc_k_major(rd_umma::smem_u32(sQ + off)), rd_umma::desc_k_major(rd_umma::smem_u32(ring + off)), idesc, k != 0);
    }
    rd_umma::commit(scores_done);
  }
  // n_in . q_t meanwhile: four threads per token
  {
    const int t = tid >> 2, part = tid & 3;
    float acc = 0.f;
#pragma unroll 2
    for (int ch = part; ch < DP / 8; ch += 4) {
      const uint4 u = *reinterpret_cast<const uint4*>(sQ + (ch >> 3) * kBox + swz<8>(t, ch & 7));
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
  const int quarter = warp & 3, cg = warp >> 2;  // cg: this warp's quarter of the TMEM columns
  const int t = quarter * 32 + lane;  // this thread's token of the chunk
  const uint32_t t_row = tmem + ((uint32_t)(quarter * 32) << 16);
  bool ok = wait_warp(scores_done, 0);
  rd_umma::fence_after();
  // The streamed second operands, one thread: S tiles (dim block, value tile, hi / lo), then V tiles (64 tokens, value tile).
  // V boxes may reach past the row's tokens (P is 0 there) and past the head's columns (never used).
  const int v_tiles = a.vpad / 128, d_blocks = a.dpad / 64;
  const int n_state = d_blocks * v_tiles * 2, n_items = n_state + ((t0 + 64 < n_tok) ? 2 : 1) * v_tiles;
  auto load = [&](int i) {
    uint8_t* dst = ring + (i % kOutStages) * kItem;
    uint64_t* bar = &full[i % kOutStages];
    rd_umma::mbar_expect_tx(bar, kItem);
    if (i < n_state) {
      const int vt = (i >> 1) % v_tiles, db = (i >> 1) / v_tiles;
      rd_umma::tma_load_2d(dst, (i & 1) ? &map_lo : &map_hi, bar, db * 64, (int)(slot * a.vpad) + vt * 128);
    } else {
      const int vt = (i - n_state) % v_tiles, jb = (i - n_state) / v_tiles;
      const int col = 2 * a.nh * a.dim + h * a.vdim + vt * 128;
      rd_umma::tma_load_2d(dst, &map_v, bar, col, rs + t0 + jb * 64);
      rd_umma::tma_load_2d(dst + kItem / 2, &map_v, bar, col + 64, rs + t0 + jb * 64);
    }
  };
  // items [i0, i1): products of each as it lands; its stage is refilled once the products of the item before are done
  auto run_items = [&](int i0, int i1) {
    for (int i = i0; i < i1; ++i) {
      if (!rd_umma::mbar_wait(&full[i % kOutStages], (i / kOutStages) & 1)) return false;
      rd_umma::fence_after();
      const uint8_t* sB = ring + (i % kOutStages) * kItem;
      if (i < n_state) {
        const int vt = (i >> 1) % v_tiles, db = (i >> 1) / v_tiles;
        const uint32_t idesc = rd_umma::idesc_f16(128, false, false);
#pragma unroll
        for (int k = 0; k < 4; ++k)
          rd_umma::mma_ss(tmem + vt * 128, rd_umma::desc_k_major(rd_umma::smem_u32(sQ + db * kBox + k * 32)),
                          rd_umma::desc_k_major(rd_umma::smem_u32(sB + k * 32)), idesc, (db | (i & 1) | k) != 0);
      } else {
        const int vt = (i - n_state) % v_tiles, jb = (i - n_state) / v_tiles;
        const uint32_t idesc = rd_umma::idesc_f16(128, false, true);
#pragma unroll
        for (int k = 0; k < 4; ++k) {
          const uint64_t dv = rd_umma::desc_mn_major(rd_umma::smem_u32(sB + k * 2048), kItem / 2);
          rd_umma::mma_ss(tmem + vt * 128, rd_umma::desc_k_major(rd_umma::smem_u32(sPh + jb * kBox + k * 32)), dv, idesc, 1);
          rd_umma::mma_ss(tmem + vt * 128, rd_umma::desc_k_major(rd_umma::smem_u32(sPl + jb * kBox + k * 32)), dv, idesc, 1);
        }
      }
      rd_umma::commit(&bars[i % kOutStages]);
      if (i > 0 && i + kOutStages - 1 < n_items) {
        if (!rd_umma::mbar_wait(&bars[(i - 1) % kOutStages], ((i - 1) / kOutStages) & 1)) return false;
        load(i + kOutStages - 1);
      }
    }
    return true;
  };
  if (ok && tid == 0)
    for (int i = 0; i < kOutStages && i < n_items; ++i) load(i);  // K has been read: its place is the ring
  __syncwarp();
  // P of this thread's token and a quarter of the keys
  if (ok) {
    const float Fm = s_Fm[t];
    const int j0 = cg * 32;
    float sum = 0.f, s[32];
    rd_umma::tmem_ld32(t_row + j0, s);
#pragma unroll
    for (int i = 0; i < 32; ++i) {
      s[i] = j0 + i <= t ? s[i] * qs * __expf(Fm + s_iF[j0 + i]) : 0.f;
      sum += s[i];
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      uint4 hi, lo;
      split2(s[8 * i], s[8 * i + 1], hi.x, lo.x);
      split2(s[8 * i + 2], s[8 * i + 3], hi.y, lo.y);
      split2(s[8 * i + 4], s[8 * i + 5], hi.z, lo.z);
      split2(s[8 * i + 6], s[8 * i + 7], hi.w, lo.w);
      const int off = (cg >> 1) * kBox + swz<8>(t, (cg & 1) * 4 + i);
      *reinterpret_cast<uint4*>(sPh + off) = hi;
      *reinterpret_cast<uint4*>(sPl + off) = lo;
    }
    s_rs[cg * L + t] = sum;
  }
  rd_umma::fence_async_proxy();
  rd_umma::fence_before();
  ok = __syncthreads_and(ok);  // P is complete, the scores have been read


  // ---- O = Q S, then O = e_t O + P V
  if (ok) {
    if (tid == 0) {
      rd_umma::fence_after();
      ok = run_items(0, n_state);
      if (ok) rd_umma::commit(state_done);
    }
    __syncwarp();
    ok = wait_warp(state_done, 0) && ok;
    rd_umma::fence_after();
    const float e = s_e[t];
    if (__all_sync(0xffffffffu, ok)) {
      for (int q = cg * v_tiles; q < (cg + 1) * v_tiles; ++q) {
        float o[32];
        rd_umma::tmem_ld32(t_row + q * 32, o);
#pragma unroll
        for (int k = 0; k < 32; ++k) o[k] *= e;
        rd_umma::tmem_st32(t_row + q * 32, o);
      }
    }
    rd_umma::fence_before();
  }
  ok = __syncthreads_and(ok);
  if (ok) {
    if (tid == 0) {
      rd_umma::fence_after();
      ok = run_items(n_state, n_items);
      if (ok) rd_umma::commit(all_done);
    }
    __syncwarp();
    ok = wait_warp(all_done, 0) && ok;
  }
  ok = __syncthreads_and(ok);
  if (ok) {
    rd_umma::fence_after();
    const float den = (s_rs[t] + s_rs[L + t]) + (s_rs[2 * L + t] + s_rs[3 * L + t]) + s_e[t] * s_nq[t];
    const float inv = 1.0f / (fmaxf(fabsf(den), s_floor[t]) + kDenEps);
    const int q_lo = cg * v_tiles, q_hi = q_lo + v_tiles;  // this warp's 32-column blocks
    float ss = 0.f;
    for (int q = q_lo; q < q_hi; ++q) {
      float o[32];
      rd_umma::tmem_ld32(t_row + q * 32, o);
#pragma unroll
      for (int k = 0; k < 32; ++k)
        if (q * 32 + k < a.vdim) ss = fmaf(o[k] * inv, o[k] * inv, ss);
    }
    s_ss[cg * L + t] = ss;
    __syncthreads();
    const float r = inv / sqrtf(((s_ss[t] + s_ss[L + t]) + (s_ss[2 * L + t] + s_ss[3 * L + t])) / (float)a.vdim + a.eps);
    // Blocks of 32 tokens x 32 columns go through shared memory, so that four lanes share a token's 64 bytes in the reads of
    // the gate and in the stores.
    constexpr int kLd = 36;  // floats per row: 16-byte accesses without conflicts
    float* scr = reinterpret_cast<float*>(ring) + warp * 32 * kLd;  // the ring and P are dead
    const int sub = lane & 3, row0 = lane >> 2;
    for (int q = q_lo; q < q_hi; ++q) {
      const int col = q * 32 + sub * 8;
      const bool in = col < a.vdim;
      uint4 gu[4];
#pragma unroll
      for (int p = 0; p < 4; ++p) {
        const int tt = t0 + quarter * 32 + p * 8 + row0;
        if (in && tt < n_tok)
          gu[p] = *reinterpret_cast<const uint4*>(a.proj + (int64_t)(rs + tt) * a.ld + 2 * a.nh * a.dim + (a.nh + h) * a.vdim + col);
      }
      float o[32];
      rd_umma::tmem_ld32(t_row + q * 32, o);
#pragma unroll
      for (int k = 0; k < 8; ++k)
        *reinterpret_cast<float4*>(scr + lane * kLd + 4 * k) = make_float4(o[4 * k] * r, o[4 * k + 1] * r, o[4 * k + 2] * r, o[4 * k + 3] * r);
      __syncwarp();
      if (in) {
        const uint4 wu = *reinterpret_cast<const uint4*>(a.norm_w + (int64_t)h * a.vdim + col);
        const __nv_bfloat162* w2 = reinterpret_cast<const __nv_bfloat162*>(&wu);
#pragma unroll
        for (int p = 0; p < 4; ++p) {
          const int tt = t0 + quarter * 32 + p * 8 + row0;
          if (tt < n_tok) {
            float y[8];
            *reinterpret_cast<float4*>(y) = *reinterpret_cast<const float4*>(scr + (p * 8 + row0) * kLd + sub * 8);
            *reinterpret_cast<float4*>(y + 4) = *reinterpret_cast<const float4*>(scr + (p * 8 + row0) * kLd + sub * 8 + 4);
            const __nv_bfloat162* g2 = reinterpret_cast<const __nv_bfloat162*>(&gu[p]);
            uint4 pk;
            uint32_t* pp = reinterpret_cast<uint32_t*>(&pk);
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              const float2 gg = __bfloat1622float2(g2[e]), ww = __bfloat1622float2(w2[e]);
              pp[e] = pack_bf16(__fdividef(y[2 * e] * ww.x, 1.f + __expf(-gg.x)), __fdividef(y[2 * e + 1] * ww.y, 1.f + __expf(-gg.y)));
            }
            *reinterpret_cast<uint4*>(a.out + ((int64_t)(rs + tt) * a.nh + h) * a.vdim + col) = pk;
          }
        }
      }
      __syncwarp();  // the scratch is reused by the next block
    }
  } else if (tid == 0) {
    if (a.status) atomicExch(a.status, 32);
    for (int i = 0; i < 2000; ++i) __nanosleep(1000);
  }
  rd_umma::fence_before();
  __syncthreads();
  if (warp == 0) {
    rd_umma::fence_after();
    rd_umma::tmem_dealloc(tmem, n_cols);
  }
}

template <typename Kern, typename... Maps>
int launch_big(Kern kern, bool& set, dim3 grid, int smem, cudaStream_t s, const Maps&... args) {
  cudaError_t err = cudaSuccess;
  if (!set) {
    err = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    RD_CHECK_CHAINED(err);
    set = true;
  }
  err = rd::launch_chained(kern, grid, dim3(kThreads), smem, s, 1, args...);
  RD_CHECK_CHAINED(err);
  return RD_OK;
}
struct Maps {
  CUtensorMap proj, v, hi, lo;  // proj in boxes of 128 and of 64 rows; the two halves of S^T
};
inline int launch_states(const Maps& m, const ChunkArgs& a, int B, cudaStream_t s) {
  static bool set = false;
  return launch_big(mlstm_states_kernel, set, dim3((a.vpad / 128) * (a.dpad / DN), a.nh, B), StateSmem::kBytes, s, m.proj, m.hi, m.lo, a);
}
template <int DP>
int launch_outputs(const Maps& m, const ChunkArgs& a, int B, int max_new, cudaStream_t s) {
  static bool set = false;
  return launch_big(mlstm_outputs_kernel<DP>, set, dim3((max_new + L - 1) / L, a.nh, B), OutSmem<DP>::kBytes, s, m.v, m.hi, m.lo, a);
}

inline int64_t pad_dim(int64_t n) { return (n + DN - 1) / DN * DN; }
inline int64_t pad_v(int64_t n) { return (n + 127) / 128 * 128; }
inline int64_t slots_of(int64_t m_max, int64_t B) { return m_max / L + B; }

}  // namespace

extern "C" int64_t rd_mlstm_chunk_workspace_bytes(int m_max, int B, int nh, int dim, int vdim) {
  const int64_t slots = slots_of(m_max, B) * nh;
  return slots * pad_dim(dim) * pad_v(vdim) * 4 + (5 * (int64_t)nh * m_max + slots * (1 + pad_dim(dim)) + 64) * (int64_t)sizeof(float);
}

extern "C" int rd_mlstm_chunk(const void* proj, int64_t ld, const float* gates, int64_t ld_gates, const float* bias_i,
                              const float* bias_f, float gate_cap, const void* norm_weight, float eps, void* out, float* S,
                              float* n, float* m, const int32_t* row_start, const int32_t* base_len, int B, int nh, int dim,
                              int vdim, int m_max, int max_new, void* workspace, int64_t workspace_bytes, int32_t* status,
                              void* stream) {
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
  a.dpad = (int)pad_dim(dim);
  a.vpad = (int)pad_v(vdim);
  a.m_max = m_max;
  a.status = status;
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
  cudaError_t err = rd::launch_chained(mlstm_gates_kernel, dim3(nh, B), dim3(kGateThreads), gates_smem, s, 1, a);
  RD_CHECK_CHAINED(err);
  Maps maps;
  const int64_t width = (int64_t)2 * nh * (dim + vdim), s_rows = slots * a.vpad;
  if (!rd_umma::make_map(&maps.proj, proj, m_max, width, ld, 128) || !rd_umma::make_map(&maps.v, proj, m_max, width, ld, 64) ||
      !rd_umma::make_map(&maps.hi, a.Shi, s_rows, a.dpad, a.dpad, 128) || !rd_umma::make_map(&maps.lo, a.Slo, s_rows, a.dpad, a.dpad, 128))
    return RD_ERR_ARG;
  int rc = launch_states(maps, a, B, s);
  if (rc != RD_OK) return rc;
  if (dim <= 64) return launch_outputs<64>(maps, a, B, max_new, s);
  if (dim <= 128) return launch_outputs<128>(maps, a, B, max_new, s);
  return launch_outputs<256>(maps, a, B, max_new, s);
}
