// Element-wise and reduction kernels of decoders with a 32-bit residual stream: scaled embedding, grouped
// RMS norm, depth average (a weighted sum over the results of all earlier layers), rotary embedding on a
// part of each head with the append to a cache whose keys and values differ in size, the commit of an
// accepted draft path to such a cache, and the bookkeeping between two decode steps.
//
// No pointer to data of an earlier kernel is __restrict__ here: with programmatic dependent launch a kernel is resident
// before that data exists, and loads the compiler may take for invariant could move above pdl_wait().
#include "rd_common.cuh"

namespace {

constexpr int kNormMaxThreads = 1024;

// One block per token.  The row is formed in fp32 (embedding gather, or the weighted sum of `n_hist` stored
// rows), written to x when asked for, kept in shared memory, and normalised in groups of H / groups
// features: each group over its own sqrt(mean of squares + eps), the whole times w.
template <typename T, int VEC>
__global__ void __launch_bounds__(kNormMaxThreads) stream_norm_kernel(
    const T* table, const int64_t* ids, float embed_scale, const float* hist,
    int64_t hist_stride, const float* coeff, int n_hist, float* x_out, const T* w,
    T* y, int m_max, const int32_t* m_dev, int H, int groups, int parts, float eps) {
  extern __shared__ float smem[];
  float* row = smem;              // [H]
  float* part_sum = smem + H;     // [groups * parts]
  rd::pdl_launch_dependents();
  rd::pdl_wait();
  const int t = blockIdx.x;
  if (t >= rd::live_rows(m_dev, m_max)) return;
  const int tid = threadIdx.x, n_thr = blockDim.x;
  if (table != nullptr) {
    const T* src = table + ids[t] * (int64_t)H;
    for (int d = tid * VEC; d < H; d += n_thr * VEC) {
#pragma unroll
      for (int e = 0; e < VEC; ++e) row[d + e] = rd::Num<T>::to_f(src[d + e]) * embed_scale;
    }
  } else {
    const float* src = hist + (int64_t)t * H;
    for (int d = tid * VEC; d < H; d += n_thr * VEC) {
      float acc[VEC];
#pragma unroll
      for (int e = 0; e < VEC; ++e) acc[e] = 0.f;
      if (coeff == nullptr) {
        if constexpr (VEC == 4) {
          *reinterpret_cast<float4*>(acc) = *reinterpret_cast<const float4*>(src + d);
        } else {
          acc[0] = src[d];
        }
      } else {
#pragma unroll 4
        for (int j = 0; j < n_hist; ++j) {
          const float c = coeff[j];
          if constexpr (VEC == 4) {
            const float4 f = *reinterpret_cast<const float4*>(src + (int64_t)j * hist_stride + d);
            acc[0] = fmaf(c, f.x, acc[0]);
            acc[1] = fmaf(c, f.y, acc[1]);
            acc[2] = fmaf(c, f.z, acc[2]);
            acc[3] = fmaf(c, f.w, acc[3]);
          } else {
            acc[0] = fmaf(c, src[(int64_t)j * hist_stride + d], acc[0]);
          }
        }
      }
#pragma unroll
      for (int e = 0; e < VEC; ++e) row[d + e] = acc[e];
    }
  }
  __syncthreads();
  if (x_out != nullptr) {
    float* dst = x_out + (int64_t)t * H;
    for (int d = tid * VEC; d < H; d += n_thr * VEC) {
      if constexpr (VEC == 4)
        *reinterpret_cast<float4*>(dst + d) = *reinterpret_cast<const float4*>(row + d);
      else
        dst[d] = row[d];
    }
  }
  // sums of squares: every group is cut into `parts` interleaved shares, one warp each
  const int warp = tid >> 5, lane = tid & 31;
  const int gsize = H / groups;
  for (int u = warp; u < groups * parts; u += (n_thr / 32)) {
    const float* g0 = row + (u / parts) * gsize;
    float ss = 0.f;
    for (int d = (u % parts) * 32 + lane; d < gsize; d += 32 * parts) ss = fmaf(g0[d], g0[d], ss);
    ss = rd::warp_sum(ss);
    if (lane == 0) part_sum[u] = ss;
  }
  __syncthreads();
  // one scale per group, left in the place of its first share
  for (int g = tid; g < groups; g += n_thr) {
    float tot = 0.f;
    for (int p = 0; p < parts; ++p) tot += part_sum[g * parts + p];
    part_sum[g * parts] = 1.0f / sqrtf(tot / (float)gsize + eps);
  }
  __syncthreads();
  T* dst = y + (int64_t)t * H;
  const bool whole = gsize % VEC == 0;  // a vector lies in one group
  for (int d = tid * VEC; d < H; d += n_thr * VEC) {
    T o[VEC], g[VEC];
    if constexpr (VEC == 4 && sizeof(T) == 2)
      *reinterpret_cast<uint2*>(g) = *reinterpret_cast<const uint2*>(w + d);
    else if constexpr (VEC == 4)
      *reinterpret_cast<float4*>(g) = *reinterpret_cast<const float4*>(w + d);
    else
      g[0] = w[d];
    float rs = part_sum[(d / gsize) * parts];
#pragma unroll
    for (int e = 0; e < VEC; ++e) {
      if (!whole) rs = part_sum[((d + e) / gsize) * parts];
      o[e] = rd::Num<T>::from_f(row[d + e] * rs * rd::Num<T>::to_f(g[e]));
    }
    if constexpr (VEC == 4 && sizeof(T) == 2)
      *reinterpret_cast<uint2*>(dst + d) = *reinterpret_cast<const uint2*>(o);
    else if constexpr (VEC == 4)
      *reinterpret_cast<float4*>(dst + d) = *reinterpret_cast<const float4*>(o);
    else
      dst[d] = o[0];
  }
}

// One block per token.  proj row: q [nh*dim] | k [nkv*dim] | v [nkv*vdim] | ...; rotated q replaces q in place,
// rotated k and v go to the token's slot.  cos/sin: [n_pos, rot/2].
constexpr int kRotThreads = 256;

template <typename T>
__global__ void __launch_bounds__(kRotThreads) rotary_append_kernel(
    T* proj, int64_t ld, T* k_cache, T* v_cache, const int32_t* tok_row,
    const int32_t* tok_pos, const int32_t* tok_slot, const float* cos_t,
    const float* sin_t, int n_pos, int m_max, const int32_t* m_dev, int nh, int nkv, int dim,
    int vdim, int rot, int max_len) {
  rd::pdl_launch_dependents();
  rd::pdl_wait();
  const int t = blockIdx.x;
  if (t >= rd::live_rows(m_dev, m_max)) return;
  const int b = tok_row[t], slot = tok_slot[t];
  int pos = tok_pos[t];
  pos = pos < 0 ? 0 : (pos >= n_pos ? n_pos - 1 : pos);
  const int half = rot / 2;
  T* row = proj + (int64_t)t * ld;
  const float* c = cos_t + (int64_t)pos * half;
  const float* s = sin_t + (int64_t)pos * half;
  // rotated pairs of q and k heads
  for (int w = threadIdx.x; w < (nh + nkv) * half; w += kRotThreads) {
    const int head = w / half, i = w % half;
    T* src = row + head * dim;
    const float u = rd::Num<T>::to_f(src[i]), v = rd::Num<T>::to_f(src[i + half]);
    const T lo = rd::Num<T>::from_f(u * c[i] - v * s[i]), hi = rd::Num<T>::from_f(v * c[i] + u * s[i]);
    T* dst = head < nh ? src : k_cache + (((int64_t)b * nkv + (head - nh)) * max_len + slot) * dim;
    dst[i] = lo;
    dst[i + half] = hi;
  }
  // the rest of k, and v
  const int rest = dim - rot;
  for (int w = threadIdx.x; w < nkv * rest; w += kRotThreads) {
    const int head = w / rest, d = rot + w % rest;
    k_cache[(((int64_t)b * nkv + head) * max_len + slot) * dim + d] = row[(nh + head) * dim + d];
  }
  const T* v0 = row + (nh + nkv) * dim;
  for (int w = threadIdx.x; w < nkv * vdim; w += kRotThreads) {
    const int head = w / vdim, d = w % vdim;
    v_cache[(((int64_t)b * nkv + head) * max_len + slot) * vdim + d] = v0[w];
  }
}

// Moves the rows of an accepted draft path to the tail of their sequence: slot base + index[b, j] -> slot
// base + j for j < count[b] + 1.  index rises with j and index[b, j] >= j, so ascending order never reads a
// row it has already overwritten.  Grid (heads, B).
template <typename T>
__global__ void __launch_bounds__(128) cache_commit_kernel(T* cache, int nkv, int max_len, int dim,
                                                           const int32_t* kv_begin,
                                                           const int32_t* base_len,
                                                           const int32_t* unpacker, int W, int Lb,
                                                           const int32_t* n_accepted,
                                                           const int32_t* seq_in_beam) {
  rd::pdl_launch_dependents();
  rd::pdl_wait();
  const int b = blockIdx.y, h = blockIdx.x;
  const int32_t* u = unpacker + ((int64_t)b * W + seq_in_beam[b]) * Lb;
  T* rows = cache + (((int64_t)b * nkv + h) * max_len + kv_begin[b] + base_len[b]) * dim;
  const int n = n_accepted[b];
  for (int j = 0; j <= n && j < Lb; ++j) {
    const int src = u[j];
    if (src == j) continue;
    // a thread moves its own columns only, so no barrier is needed between the rows
    for (int d = threadIdx.x; d < dim; d += blockDim.x) rows[(int64_t)j * dim + d] = rows[(int64_t)src * dim + d];
  }
}

// After the next token of every row has been chosen: it is appended to the row's token buffer and the row's
// counters move on.
__global__ void decode_advance_kernel(const int64_t* next_tok, int64_t* token_buf, int64_t buf_ld,
                                      const int32_t* buf_begin, const int32_t* begin,
                                      int32_t* kv_len, int32_t* base_len,
                                      int32_t* slot, int limit, int B) {
  rd::pdl_launch_dependents();
  rd::pdl_wait();
  const int b = blockIdx.x * blockDim.x + threadIdx.x;
  if (b >= B) return;
  const int len = kv_len[b];
  int s = begin[b] + len;
  if (s >= limit) s = limit - 1;  // the host keeps rows shorter; stay inside the buffers in any case
  if (token_buf != nullptr) {
    const int64_t c = buf_begin[b] + len;
    if (c < buf_ld) token_buf[(int64_t)b * buf_ld + c] = next_tok[b];
  }
  base_len[b] = len;
  slot[b] = s;
  kv_len[b] = len + 1;
}

}  // namespace

#define RD_DISPATCH_T(dtype, ...)                  \
  if ((dtype) == RD_F32) {                         \
    using T = float;                               \
    __VA_ARGS__;                                   \
  } else if ((dtype) == RD_BF16) {                 \
    using T = __nv_bfloat16;                       \
    __VA_ARGS__;                                   \
  } else {                                         \
    return RD_ERR_DTYPE;                           \
  }

extern "C" int rd_stream_norm(int dtype, const void* table, const int64_t* ids, float embed_scale, const float* hist,
                              int64_t hist_stride, const float* coeff, int n_hist, float* x_out, const void* weight, void* y,
                              int m_max, const int32_t* m_dev, int H, int groups, float eps, void* stream) {
  RD_REQUIRE(weight && y && ((table && ids && !hist) || (!table && hist)), RD_ERR_ARG);
  RD_REQUIRE(m_max >= 1 && H >= 1 && groups >= 1 && H % groups == 0 && (table || n_hist >= 1), RD_ERR_SIZE);
  RD_REQUIRE(coeff || table || n_hist == 1, RD_ERR_ARG);
  const uintptr_t bits = (uintptr_t)hist | (uintptr_t)x_out | (uintptr_t)y | (uintptr_t)weight;
  const bool vec = H % 4 == 0 && bits % 16 == 0 && hist_stride % 4 == 0;
  int threads = ((vec ? H / 4 : H) + 31) / 32 * 32;
  // few tokens: the row's loads all in flight at once; many tokens: small blocks, several per SM
  const int most = m_max <= 2 * 148 ? kNormMaxThreads : 256;
  threads = threads > most ? most : threads;
  const int warps = threads / 32;
  const int parts = groups >= warps ? 1 : (warps + groups - 1) / groups;
  const size_t smem = ((size_t)H + (size_t)groups * parts) * sizeof(float);
  RD_REQUIRE(smem <= 200 * 1024, RD_ERR_SIZE);
  cudaError_t err = cudaSuccess;
  RD_DISPATCH_T(dtype, {
    auto kern = vec ? stream_norm_kernel<T, 4> : stream_norm_kernel<T, 1>;
    if (smem > 48 * 1024) {
      err = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
      RD_CHECK_CHAINED(err);
    }
    err = rd::launch_chained(kern, dim3(m_max), dim3(threads), smem, (cudaStream_t)stream, 1, (const T*)table, ids,
                             embed_scale, hist, hist_stride, coeff, n_hist, x_out, (const T*)weight, (T*)y, m_max, m_dev, H,
                             groups, parts, eps);
  });
  RD_CHECK_CHAINED(err);
  return RD_OK;
}

extern "C" int rd_rotary_append(int dtype, void* proj, int64_t ld, void* k_cache, void* v_cache, const int32_t* tok_row,
                                const int32_t* tok_pos, const int32_t* tok_slot, const float* cos_table, const float* sin_table,
                                int n_pos, int m_max, const int32_t* m_dev, int nh, int nkv, int dim, int vdim, int rot_dims,
                                int max_len, void* stream) {
  RD_REQUIRE(proj && k_cache && v_cache && tok_row && tok_pos && tok_slot, RD_ERR_ARG);
  RD_REQUIRE(m_max >= 1 && nh >= 1 && nkv >= 1 && dim >= 1 && vdim >= 1 && rot_dims >= 0 && rot_dims % 2 == 0 && rot_dims <= dim &&
                 max_len >= 1 && n_pos >= 1 && ld >= (int64_t)(nh + nkv) * dim + (int64_t)nkv * vdim,
             RD_ERR_SIZE);
  RD_REQUIRE(rot_dims == 0 || (cos_table && sin_table), RD_ERR_ARG);
  cudaError_t err = cudaSuccess;
  RD_DISPATCH_T(dtype, (err = rd::launch_chained(rotary_append_kernel<T>, dim3(m_max), dim3(kRotThreads), 0, (cudaStream_t)stream, 1,
                                                 (T*)proj, ld, (T*)k_cache, (T*)v_cache, tok_row, tok_pos, tok_slot, cos_table,
                                                 sin_table, n_pos, m_max, m_dev, nh, nkv, dim, vdim, rot_dims, max_len)));
  RD_CHECK_CHAINED(err);
  return RD_OK;
}

extern "C" int rd_cache_commit(int dtype, void* cache, int B, int nkv, int max_len, int dim, const int32_t* kv_begin,
                               const int32_t* base_len, const int32_t* unpacker, int W, int Lb, const int32_t* n_accepted,
                               const int32_t* seq_in_beam, void* stream) {
  RD_REQUIRE(cache && kv_begin && base_len && unpacker && n_accepted && seq_in_beam, RD_ERR_ARG);
  RD_REQUIRE(B >= 1 && B <= 65535 && nkv >= 1 && max_len >= 1 && dim >= 1 && W >= 1 && Lb >= 1, RD_ERR_SIZE);
  cudaError_t err = cudaSuccess;
  RD_DISPATCH_T(dtype, (err = rd::launch_chained(cache_commit_kernel<T>, dim3(nkv, B), dim3(128), 0, (cudaStream_t)stream, 1, (T*)cache,
                                                 nkv, max_len, dim, kv_begin, base_len, unpacker, W, Lb, n_accepted, seq_in_beam)));
  RD_CHECK_CHAINED(err);
  return RD_OK;
}

extern "C" int rd_decode_advance(const int64_t* next_tok, int64_t* token_buf, int64_t buf_ld, const int32_t* buf_begin,
                                 const int32_t* begin, int32_t* kv_len, int32_t* base_len, int32_t* slot, int limit, int B,
                                 void* stream) {
  RD_REQUIRE(next_tok && begin && kv_len && base_len && slot && (!token_buf || buf_begin), RD_ERR_ARG);
  RD_REQUIRE(B >= 1 && limit >= 1 && (!token_buf || buf_ld >= 1), RD_ERR_SIZE);
  cudaError_t err = rd::launch_chained(decode_advance_kernel, dim3((B + 127) / 128), dim3(128), 0, (cudaStream_t)stream, 1, next_tok,
                                       token_buf, buf_ld, buf_begin, begin, kv_len, base_len, slot, limit, B);
  RD_CHECK_CHAINED(err);
  return RD_OK;
}
