// Shared device/host helpers for the ReDrafter B200 kernels.
#pragma once

#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include "../../include/redrafter_b200.h"

#define RD_LOG_0 (-50000.0f)

// Launch-time check: returns a negative code for an invalid argument found on the host.
#define RD_REQUIRE(cond, code) \
  do {                         \
    if (!(cond)) return (code); \
  } while (0)

// Returns RD_ERR_LAUNCH when the launch itself was rejected (bad configuration).
#define RD_CHECK_LAUNCH()                                   \
  do {                                                      \
    cudaError_t e__ = cudaPeekAtLastError();                \
    if (e__ != cudaSuccess) {                               \
      rd_set_last_cuda_error((int)e__);                     \
      return RD_ERR_LAUNCH;                                 \
    }                                                       \
  } while (0)

// The same for a cudaError_t already in hand (rd::launch_chained() returns one).
#define RD_CHECK_CHAINED(err)                               \
  do {                                                      \
    if ((err) != cudaSuccess) {                             \
      rd_set_last_cuda_error((int)(err));                   \
      return RD_ERR_LAUNCH;                                 \
    }                                                       \
  } while (0)

void rd_set_last_cuda_error(int e);
// 1 unless the environment variable RD_PDL is "0" (read once): launch the kernels of the decode
// chain with programmatic stream serialisation so that a kernel's launch and prologue overlap the
// tail of its predecessor.
int rd_pdl_enabled();

namespace rd {

template <typename T>
struct Num;
template <>
struct Num<float> {
  static __device__ __forceinline__ float to_f(float v) { return v; }
  static __device__ __forceinline__ float from_f(float v) { return v; }
};
template <>
struct Num<__nv_bfloat16> {
  static __device__ __forceinline__ float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
  static __device__ __forceinline__ __nv_bfloat16 from_f(float v) { return __float2bfloat16_rn(v); }
};

// fast form for rounded (bf16) outputs: approximate exp and division, ~2 ulp
__device__ __forceinline__ float silu_f(float x) { return __fdividef(x, 1.0f + __expf(-x)); }
// expf with full fp32 accuracy (used where parity with a CPU fp32 path matters)
__device__ __forceinline__ float silu_exact(float x) { return x / (1.0f + expf(-x)); }

// xIELU: pos z^2 + z/2 above zero, neg (e^z - 1 - z) + z/2 elsewhere.  Each part vanishes on the other's side, so neither
// needs a branch.
__device__ __forceinline__ float xielu_exact(float z, float pos, float neg) {
  const float p = fmaxf(z, 0.f), m = fminf(z, 0.f);
  return fmaf(pos * p, p, neg * (expm1f(m) - m)) + 0.5f * z;
}
// form for rounded (bf16) outputs: e^z - 1 carries an absolute error of about 1e-7 near zero
__device__ __forceinline__ float xielu_f(float z, float pos, float neg) {
  const float p = fmaxf(z, 0.f), m = fminf(z, 0.f);
  return fmaf(pos * p, p, fmaf(neg, __expf(m) - 1.0f - m, 0.5f * z));
}

// Gated unit with cut inputs: g sigmoid(alpha g) (u + 1), g = min(gate, limit), u = up cut to [-limit, limit].
__device__ __forceinline__ float clamped_glu_exact(float gate, float up, float limit, float alpha) {
  const float g = fminf(gate, limit), u = fminf(fmaxf(up, -limit), limit);
  return g / (1.0f + expf(-alpha * g)) * (u + 1.0f);
}
// form for rounded (bf16) outputs
__device__ __forceinline__ float clamped_glu_f(float gate, float up, float limit, float alpha) {
  const float g = fminf(gate, limit), u = fminf(fmaxf(up, -limit), limit);
  return __fdividef(g, 1.0f + __expf(-alpha * g)) * (u + 1.0f);
}

__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
  return v;
}
__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
__device__ __forceinline__ int warp_sum_i(int v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}

// Order-preserving map float -> uint32 (larger float <=> larger key).
__device__ __forceinline__ uint32_t float_key(float f) {
  uint32_t u = __float_as_uint(f);
  return (u & 0x80000000u) ? ~u : (u | 0x80000000u);
}

// Effective row count: min(*m_dev, m_max) when a device-side count is given.
__device__ __forceinline__ int live_rows(const int* m_dev, int m_max) {
  if (m_dev == nullptr) return m_max;
  int m = *m_dev;
  return m < m_max ? (m < 0 ? 0 : m) : m_max;
}

// Programmatic dependent launch.  A kernel launched with rd::launch_chained() may begin before the
// previous kernel of the stream has finished: it must execute pdl_wait() before its first access to
// global memory (reads of the predecessor's results and writes to anything the predecessor may still
// read), and it lets its own successor start early with pdl_launch_dependents().  Both are no-ops
// in a kernel that was launched the ordinary way.  Data of an earlier kernel must not be read through a const
// __restrict__ pointer in straight-line code after the wait: the compiler may treat such loads as invariant and
// hoist them above it (a commit kernel read the previous step's acceptance that way once its launch overlapped).
__device__ __forceinline__ void pdl_launch_dependents() { asm volatile("griddepcontrol.launch_dependents;" ::: "memory"); }
__device__ __forceinline__ void pdl_wait() { asm volatile("griddepcontrol.wait;" ::: "memory"); }

template <typename... KArgs, typename... Args>
inline cudaError_t launch_chained(void (*kern)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t s, int cluster_x,
                                  Args&&... args) {
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = grid;
  cfg.blockDim = block;
  cfg.dynamicSmemBytes = smem;
  cfg.stream = s;
  cudaLaunchAttribute attr[2];
  int n = 0;
  if (cluster_x > 1) {
    attr[n].id = cudaLaunchAttributeClusterDimension;
    attr[n].val.clusterDim.x = cluster_x;
    attr[n].val.clusterDim.y = 1;
    attr[n].val.clusterDim.z = 1;
    ++n;
  }
  if (rd_pdl_enabled()) {
    attr[n].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[n].val.programmaticStreamSerializationAllowed = 1;
    ++n;
  }
  cfg.attrs = attr;
  cfg.numAttrs = n;
  return cudaLaunchKernelEx(&cfg, kern, static_cast<KArgs>(args)...);
}

}  // namespace rd
