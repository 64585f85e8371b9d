// One small product per attention head, C[t, h, :] = W[h] A[t, h, :]: the up-projections of latent attention applied to the
// queries and to the outputs of a few tokens, where the weights are the traffic.
//
//   head_gemm_mma_kernel   bf16, warp-level tensor cores: 32 tokens x 64 outputs of one head per CTA, four-stage cp.async ring
//   head_gemm_simt_kernel  any dtype and size, fp32 sums on CUDA cores
#include "mma_sync.cuh"

namespace {

using namespace rd_mma;

struct Args {
  const void* A;
  int64_t lda, a_head;
  const void* W;  // [heads, N, K]
  void* C;
  int64_t ldc, c_head;
  int m_max;
  const int32_t* m_dev;
  int N, K;
};

// ------------------------------------------------------------------------------------------------ tensor cores
constexpr int kTM = 32, kTN = 64, kTK = 64, kRingStages = 4, kMmaThreads = 128;
constexpr int kStageBytes = (kTM + kTN) * kTK * 2;

// rows of 64 features = 8 chunks of 16 bytes
__device__ __forceinline__ int swz(int r, int c) { return r * 128 + ((c ^ (r & 7)) << 4); }

// grid (N tiles, M tiles, heads)
__global__ void __launch_bounds__(kMmaThreads) head_gemm_mma_kernel(const Args a) {
  extern __shared__ __align__(128) uint8_t smem[];
  rd::pdl_launch_dependents();
  rd::pdl_wait();
  const int M = rd::live_rows(a.m_dev, a.m_max);
  const int m0 = blockIdx.y * kTM, n0 = blockIdx.x * kTN, h = blockIdx.z;
  if (m0 >= M) return;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const __nv_bfloat16* A = (const __nv_bfloat16*)a.A + (int64_t)h * a.a_head;
  const __nv_bfloat16* W = (const __nv_bfloat16*)a.W + (int64_t)h * a.N * a.K;
  const int n_k = (a.K + kTK - 1) / kTK;
  auto load = [&](int t) {
    if (t < n_k) {
      uint8_t* dst = smem + (t % kRingStages) * kStageBytes;
#pragma unroll
      for (int i = 0; i < (kTM + kTN) * 8 / kMmaThreads; ++i) {
        const int idx = i * kMmaThreads + tid, r = idx >> 3, c = idx & 7;
        const int k = t * kTK + c * 8;
        const bool is_a = r < kTM;
        const int row = is_a ? m0 + r : n0 + r - kTM;
        const bool in = k < a.K && row < (is_a ? M : a.N);
        const __nv_bfloat16* src = is_a ? A : W;
        if (in) src += (int64_t)row * (is_a ? a.lda : a.K) + k;
        cp_async16(dst + (is_a ? 0 : kTM * 128) + swz(is_a ? r : r - kTM, c), src, in);
      }
    }
    cp_async_commit();
  };
  for (int t = 0; t < kRingStages - 1; ++t) load(t);
  float acc[2][2][4] = {};  // two 16-token tiles x two 8-output blocks: this warp's 16 outputs
  for (int t = 0; t < n_k; ++t) {
    cp_async_wait<kRingStages - 2>();
    __syncthreads();
    load(t + kRingStages - 1);
    const uint8_t* sA = smem + (t % kRingStages) * kStageBytes;
    const uint8_t* sW = sA + kTM * 128;
#pragma unroll
    for (int kd = 0; kd < kTK / 16; ++kd) {
      uint32_t a0[4], a1[4], b0, b1, b2, b3;
      ldmatrix_x4(a0[0], a0[1], a0[2], a0[3], smem_addr(sA + swz(lane & 15, kd * 2 + (lane >> 4))));
      ldmatrix_x4(a1[0], a1[1], a1[2], a1[3], smem_addr(sA + swz(16 + (lane & 15), kd * 2 + (lane >> 4))));
      ldmatrix_x4(b0, b1, b2, b3, smem_addr(sW + swz(warp * 16 + ((lane >> 4) << 3) + (lane & 7), kd * 2 + ((lane >> 3) & 1))));
      mma_bf16(acc[0][0], a0, b0, b1);
      mma_bf16(acc[0][1], a0, b2, b3);
      mma_bf16(acc[1][0], a1, b0, b1);
      mma_bf16(acc[1][1], a1, b2, b3);
    }
  }
  cp_async_wait<0>();
  const int g = lane >> 2, t4 = lane & 3;
  __nv_bfloat16* C = (__nv_bfloat16*)a.C + (int64_t)h * a.c_head;
#pragma unroll
  for (int mt = 0; mt < 2; ++mt)
#pragma unroll
    for (int hh = 0; hh < 2; ++hh) {
      const int m = m0 + mt * 16 + g + hh * 8;
      if (m >= M) continue;
#pragma unroll
      for (int nb = 0; nb < 2; ++nb) {
        const int n = n0 + warp * 16 + nb * 8 + t4 * 2;
        if (n < a.N) *reinterpret_cast<uint32_t*>(C + (int64_t)m * a.ldc + n) = pack_bf16(acc[mt][nb][hh * 2], acc[mt][nb][hh * 2 + 1]);
      }
    }
}

// ------------------------------------------------------------------------------------------------ CUDA cores
constexpr int kB = 32, kBK = 16;  // 32 x 32 outputs per CTA, 256 threads with 2 x 2 each

template <typename T>
__global__ void __launch_bounds__(256) head_gemm_simt_kernel(const Args a) {
  rd::pdl_launch_dependents();
  rd::pdl_wait();
  const int M = rd::live_rows(a.m_dev, a.m_max);
  const int m0 = blockIdx.y * kB, n0 = blockIdx.x * kB, h = blockIdx.z;
  if (m0 >= M) return;
  __shared__ float As[kBK][kB + 1], Ws[kBK][kB + 1];
  const T* A = (const T*)a.A + (int64_t)h * a.a_head;
  const T* W = (const T*)a.W + (int64_t)h * a.N * a.K;
  const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
  float acc[2][2] = {};
  for (int k0 = 0; k0 < a.K; k0 += kBK) {
    for (int i = tid; i < kB * kBK; i += 256) {
      const int r = i / kBK, k = i % kBK;
      As[k][r] = (m0 + r < M && k0 + k < a.K) ? rd::Num<T>::to_f(A[(int64_t)(m0 + r) * a.lda + k0 + k]) : 0.f;
      Ws[k][r] = (n0 + r < a.N && k0 + k < a.K) ? rd::Num<T>::to_f(W[(int64_t)(n0 + r) * a.K + k0 + k]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kBK; ++k)
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int j = 0; j < 2; ++j) acc[i][j] = fmaf(As[k][ty * 2 + i], Ws[k][tx * 2 + j], acc[i][j]);
    __syncthreads();
  }
  T* C = (T*)a.C + (int64_t)h * a.c_head;
#pragma unroll
  for (int i = 0; i < 2; ++i)
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int m = m0 + ty * 2 + i, n = n0 + tx * 2 + j;
      if (m < M && n < a.N) C[(int64_t)m * a.ldc + n] = rd::Num<T>::from_f(acc[i][j]);
    }
}

}  // namespace

extern "C" int rd_head_gemm(int dtype, const void* A, int64_t lda, int64_t a_head, const void* W, void* C, int64_t ldc, int64_t c_head,
                            int m_max, const int32_t* m_dev, int heads, int N, int K, void* stream) {
  RD_REQUIRE(A && W && C, RD_ERR_ARG);
  RD_REQUIRE(dtype == RD_F32 || dtype == RD_BF16, RD_ERR_DTYPE);
  RD_REQUIRE(m_max >= 1 && heads >= 1 && heads <= 65535 && N >= 1 && K >= 1 && (m_max + kTM - 1) / kTM <= 65535, RD_ERR_SIZE);
  const Args a{A, lda, a_head, W, C, ldc, c_head, m_max, m_dev, N, K};
  cudaStream_t s = (cudaStream_t)stream;
  cudaError_t err;
  const uintptr_t bits = (uintptr_t)A | (uintptr_t)W | (uintptr_t)C;
  if (dtype == RD_BF16 && K % 8 == 0 && N % 8 == 0 && (lda | a_head | ldc | c_head) % 8 == 0 && bits % 16 == 0) {
    err = rd::launch_chained(head_gemm_mma_kernel, dim3((N + kTN - 1) / kTN, (m_max + kTM - 1) / kTM, heads), dim3(kMmaThreads),
                             (size_t)kRingStages * kStageBytes, s, 1, a);
  } else {
    auto kern = dtype == RD_F32 ? head_gemm_simt_kernel<float> : head_gemm_simt_kernel<__nv_bfloat16>;
    err = rd::launch_chained(kern, dim3((N + kB - 1) / kB, (m_max + kB - 1) / kB, heads), dim3(256), 0, s, 1, a);
  }
  RD_CHECK_CHAINED(err);
  return RD_OK;
}
