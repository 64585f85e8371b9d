// What the matrix-memory kernels share: the gates, and the norm + output gate that follows the recurrence.
#pragma once
#include "rd_common.cuh"

namespace rd_mlstm {

constexpr float kDenEps = 1e-6f;

__device__ __forceinline__ float soft_cap(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }

// Per token and head: o / rms(o) * norm weight * sigmoid(g), one warp per head.
constexpr int kNormThreads = 256;

template <typename T, int VEC>
__global__ void __launch_bounds__(kNormThreads) norm_gate_kernel(
    const float* o, const T* g, int64_t ld, const T* w, T* out, float eps,
    const int32_t* row_start, int B, int nh, int vdim) {
  rd::pdl_launch_dependents();
  rd::pdl_wait();
  const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (t >= row_start[B]) return;
  for (int h = warp; h < nh; h += kNormThreads / 32) {
    const int64_t base = ((int64_t)t * nh + h) * vdim;
    const float* src = o + base;
    const T* gp = g + (int64_t)t * ld + (int64_t)h * vdim;
    const T* wp = w + (int64_t)h * vdim;
    float ss = 0.f;
    for (int u = lane * VEC; u < vdim; u += 32 * VEC) {
      float f[VEC];
      if constexpr (VEC == 4)
        *reinterpret_cast<float4*>(f) = *reinterpret_cast<const float4*>(src + u);
      else
        f[0] = src[u];
#pragma unroll
      for (int e = 0; e < VEC; ++e) ss = fmaf(f[e], f[e], ss);
    }
    ss = rd::warp_sum(ss);
    const float r = 1.0f / sqrtf(ss / (float)vdim + eps);
    for (int u = lane * VEC; u < vdim; u += 32 * VEC) {
      float f[VEC];
      T gg[VEC], ww[VEC], y[VEC];
      if constexpr (VEC == 4) {
        *reinterpret_cast<float4*>(f) = *reinterpret_cast<const float4*>(src + u);
        *reinterpret_cast<uint2*>(gg) = *reinterpret_cast<const uint2*>(gp + u);
        *reinterpret_cast<uint2*>(ww) = *reinterpret_cast<const uint2*>(wp + u);
      } else {
        f[0] = src[u];
        gg[0] = gp[u];
        ww[0] = wp[u];
      }
#pragma unroll
      for (int e = 0; e < VEC; ++e) {
        const float z = rd::Num<T>::to_f(gg[e]);
        const float sg = 1.0f / (1.0f + (sizeof(T) == 2 ? __expf(-z) : expf(-z)));
        y[e] = rd::Num<T>::from_f(f[e] * r * rd::Num<T>::to_f(ww[e]) * sg);
      }
      if constexpr (VEC == 4)
        *reinterpret_cast<uint2*>(out + base + u) = *reinterpret_cast<const uint2*>(y);
      else
        out[base + u] = y[0];
    }
  }
}

// rows: upper bound of the packed tokens
template <typename T>
int launch_norm_gate(const float* o, const void* g, int64_t ld, const void* w, void* out, float eps, int rows, const int32_t* row_start,
                     int B, int nh, int vdim, cudaStream_t s) {
  const bool vec = sizeof(T) == 2 && vdim % 4 == 0 && ld % 4 == 0 && (((uintptr_t)o | (uintptr_t)out) & 15) == 0 &&
                   (((uintptr_t)g | (uintptr_t)w) & 7) == 0;
  const dim3 grid(rows);
  cudaError_t err;
  if constexpr (sizeof(T) == 2) {
    err = rd::launch_chained(vec ? norm_gate_kernel<T, 4> : norm_gate_kernel<T, 1>, grid, dim3(kNormThreads), 0, s, 1, o, (const T*)g, ld,
                             (const T*)w, (T*)out, eps, row_start, B, nh, vdim);
  } else {
    err = rd::launch_chained(norm_gate_kernel<T, 1>, grid, dim3(kNormThreads), 0, s, 1, o, (const T*)g, ld, (const T*)w, (T*)out, eps,
                             row_start, B, nh, vdim);
  }
  RD_CHECK_CHAINED(err);
  return RD_OK;
}

}  // namespace rd_mlstm
