// What comes between an attention layer's input projections and its scores: rotary embedding (either pairing), norms of
// queries and keys, latents, and the append to the cache; and the gathering of the latents that a prompt's tokens see.
//
// No pointer to data of an earlier kernel is __restrict__ here (programmatic dependent launch, see rd_common.cuh).
#include "attention_window.cuh"

namespace {

using rd::Num;

// Features (lo, hi) of pair i.
struct Pairing {
  int half, neighbours;
  __device__ __forceinline__ int lo(int i) const { return neighbours ? 2 * i : i; }
  __device__ __forceinline__ int hi(int i) const { return neighbours ? 2 * i + 1 : i + half; }
};

__device__ __forceinline__ int clamp_pos(int pos, int n_pos) { return pos < 0 ? 0 : (pos >= n_pos ? n_pos - 1 : pos); }

// ------------------------------------------------------------------------------------------------ q, k, v heads
struct HeadArgs {
  int64_t ld;
  const int32_t *tok_row, *tok_pos, *tok_slot;
  const float *cos_t, *sin_t;
  int n_pos, m_max;
  const int32_t* m_dev;
  int nh, nkv, dim, vdim, rot, neighbours;
  float eps;
  int max_len;
};
constexpr int kHeadThreads = 256;

// One block per token, one warp per head at a time.
template <typename T>
__global__ void __launch_bounds__(kHeadThreads) rotary_norm_append_kernel(T* proj, T* k_cache, T* v_cache, const HeadArgs a) {
  rd::pdl_launch_dependents();
  rd::pdl_wait();
  const int t = blockIdx.x;
  if (t >= rd::live_rows(a.m_dev, a.m_max)) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int b = a.tok_row[t], slot = a.tok_slot[t], pos = clamp_pos(a.tok_pos[t], a.n_pos);
  const Pairing pair{a.rot / 2, a.neighbours};
  const float* c = a.cos_t + (int64_t)pos * pair.half;
  const float* s = a.sin_t + (int64_t)pos * pair.half;
  T* row = proj + (int64_t)t * a.ld;
  const int vd = a.vdim > 0 ? a.vdim : a.dim;
  for (int head = warp; head < a.nh + a.nkv; head += kHeadThreads / 32) {
    T* src = row + head * a.dim;
    const int kv = head - a.nh;
    T* dst = kv < 0 ? src : k_cache + (((int64_t)b * a.nkv + kv) * a.max_len + slot) * a.dim;
    T* v_dst = kv < 0 ? nullptr : v_cache + (((int64_t)b * a.nkv + kv) * a.max_len + slot) * vd;
    float f = 1.f;
    if (a.eps >= 0.f) {
      // a rotation does not change the sum of squares
      float ss = 0.f;
      for (int d = lane; d < a.dim; d += 32) {
        const float x = Num<T>::to_f(src[d]);
        ss = fmaf(x, x, ss);
      }
      f = 1.0f / sqrtf(rd::warp_sum(ss) / (float)a.dim + a.eps);
    }
    if (kv >= 0 && a.vdim == 0) {
      for (int d = lane; d < a.dim; d += 32) v_dst[d] = src[d];
    }
    for (int i = lane; i < pair.half; i += 32) {
      const int lo = pair.lo(i), hi = pair.hi(i);
      const float u = Num<T>::to_f(src[lo]), v = Num<T>::to_f(src[hi]);
      dst[lo] = Num<T>::from_f((u * c[i] - v * s[i]) * f);
      dst[hi] = Num<T>::from_f((v * c[i] + u * s[i]) * f);
    }
    for (int d = a.rot + lane; d < a.dim; d += 32) dst[d] = Num<T>::from_f(Num<T>::to_f(src[d]) * f);
    if (kv >= 0 && a.vdim > 0) {
      const T* v_src = row + (a.nh + a.nkv) * a.dim + kv * a.vdim;
      for (int d = lane; d < a.vdim; d += 32) v_dst[d] = v_src[d];
    }
  }
}

// ------------------------------------------------------------------------------------------------ latents
struct LatentArgs {
  int64_t ldq, ld_rot, rot_head, ld_dkv;
  const float* dkv;
  float eps;
  const int32_t *tok_row, *tok_pos, *tok_slot;
  const float *cos_t, *sin_t;
  int n_pos, m_max;
  const int32_t* m_dev;
  int nh, dim, rot_dim, rot, neighbours, rank, max_len;
};
constexpr int kLatentThreads = 256;

// One block per token.
template <typename T>
__global__ void __launch_bounds__(kLatentThreads) latent_append_kernel(const T* q, T* q_rot, const T* norm_w, T* cache, const LatentArgs a) {
  __shared__ float part[kLatentThreads / 32];
  rd::pdl_launch_dependents();
  rd::pdl_wait();
  const int t = blockIdx.x;
  if (t >= rd::live_rows(a.m_dev, a.m_max)) return;
  const int tid = threadIdx.x;
  const int b = a.tok_row[t], slot = a.tok_slot[t], pos = clamp_pos(a.tok_pos[t], a.n_pos);
  const Pairing pair{a.rot / 2, a.neighbours};
  const float* c = a.cos_t + (int64_t)pos * pair.half;
  const float* s = a.sin_t + (int64_t)pos * pair.half;
  const float* src = a.dkv + (int64_t)t * a.ld_dkv;
  T* dst = cache + ((int64_t)b * a.max_len + slot) * (a.rank + a.rot_dim);
  float ss = 0.f;
  for (int d = tid; d < a.rank; d += kLatentThreads) ss = fmaf(src[d], src[d], ss);
  ss = rd::warp_sum(ss);
  if ((tid & 31) == 0) part[tid >> 5] = ss;
  // the query heads' rotated features meanwhile
  const int rest = a.rot_dim - a.rot;
  for (int w = tid; w < a.nh * pair.half; w += kLatentThreads) {
    const int h = w / pair.half, i = w % pair.half;
    const T* from = q + (int64_t)t * a.ldq + (int64_t)h * (a.dim + a.rot_dim) + a.dim;
    T* to = q_rot + (int64_t)t * a.ld_rot + h * a.rot_head;
    const int lo = pair.lo(i), hi = pair.hi(i);
    const float u = Num<T>::to_f(from[lo]), v = Num<T>::to_f(from[hi]);
    to[lo] = Num<T>::from_f(u * c[i] - v * s[i]);
    to[hi] = Num<T>::from_f(v * c[i] + u * s[i]);
  }
  for (int w = tid; w < a.nh * rest; w += kLatentThreads) {
    const int h = w / rest, d = a.rot + w % rest;
    q_rot[(int64_t)t * a.ld_rot + h * a.rot_head + d] = q[(int64_t)t * a.ldq + (int64_t)h * (a.dim + a.rot_dim) + a.dim + d];
  }
  // the shared key part
  for (int i = tid; i < pair.half; i += kLatentThreads) {
    const int lo = pair.lo(i), hi = pair.hi(i);
    const float u = src[a.rank + lo], v = src[a.rank + hi];
    dst[a.rank + lo] = Num<T>::from_f(u * c[i] - v * s[i]);
    dst[a.rank + hi] = Num<T>::from_f(v * c[i] + u * s[i]);
  }
  for (int d = a.rot + tid; d < a.rot_dim; d += kLatentThreads) dst[a.rank + d] = Num<T>::from_f(src[a.rank + d]);
  __syncthreads();
  float tot = 0.f;
#pragma unroll
  for (int w = 0; w < kLatentThreads / 32; ++w) tot += part[w];
  const float f = 1.0f / sqrtf(tot / (float)a.rank + a.eps);
  for (int d = tid; d < a.rank; d += kLatentThreads) dst[d] = Num<T>::from_f(src[d] * f * Num<T>::to_f(norm_w[d]));
}

// The same for bf16, neighbouring pairs and sizes in multiples of 8, with every load 16 bytes wide: the latent stays in
// registers between its sum of squares and its store (rank <= 4 * kLatentThreads).
__global__ void __launch_bounds__(kLatentThreads) latent_append_vec_kernel(const __nv_bfloat16* q, __nv_bfloat16* q_rot, const __nv_bfloat16* norm_w,
                                                                           __nv_bfloat16* cache, const LatentArgs a) {
  __shared__ float part[kLatentThreads / 32];
  rd::pdl_launch_dependents();
  rd::pdl_wait();
  const int t = blockIdx.x;
  if (t >= rd::live_rows(a.m_dev, a.m_max)) return;
  const int tid = threadIdx.x;
  const int b = a.tok_row[t], slot = a.tok_slot[t], pos = clamp_pos(a.tok_pos[t], a.n_pos);
  const float* src = a.dkv + (int64_t)t * a.ld_dkv;
  const bool has = tid * 4 < a.rank;
  const float4 x = has ? *reinterpret_cast<const float4*>(src + tid * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
  const uint2 w = has ? *reinterpret_cast<const uint2*>(norm_w + tid * 4) : make_uint2(0u, 0u);
  float ss = rd::warp_sum(fmaf(x.x, x.x, fmaf(x.y, x.y, fmaf(x.z, x.z, x.w * x.w))));
  if ((tid & 31) == 0) part[tid >> 5] = ss;
  // four pairs of a query head, or of the key part (the last units)
  const int per = a.rot / 8;
  __nv_bfloat16* dst = cache + ((int64_t)b * a.max_len + slot) * (a.rank + a.rot_dim);
  for (int u = tid; u < (a.nh + 1) * per; u += kLatentThreads) {
    const int h = u / per, i = u % per;
    const float4 c = *reinterpret_cast<const float4*>(a.cos_t + (int64_t)pos * (a.rot / 2) + i * 4);
    const float4 s = *reinterpret_cast<const float4*>(a.sin_t + (int64_t)pos * (a.rot / 2) + i * 4);
    float v[8];
    __nv_bfloat16* to;
    if (h < a.nh) {
      const uint4 raw = *reinterpret_cast<const uint4*>(q + (int64_t)t * a.ldq + (int64_t)h * (a.dim + a.rot_dim) + a.dim + i * 8);
      const __nv_bfloat162* p2 = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float2 f = __bfloat1622float2(p2[e]);
        v[2 * e] = f.x, v[2 * e + 1] = f.y;
      }
      to = q_rot + (int64_t)t * a.ld_rot + h * a.rot_head + i * 8;
    } else {
      *reinterpret_cast<float4*>(v) = *reinterpret_cast<const float4*>(src + a.rank + i * 8);
      *reinterpret_cast<float4*>(v + 4) = *reinterpret_cast<const float4*>(src + a.rank + i * 8 + 4);
      to = dst + a.rank + i * 8;
    }
    const float cc[4] = {c.x, c.y, c.z, c.w}, sn[4] = {s.x, s.y, s.z, s.w};
    uint4 out;
    __nv_bfloat162* o2 = reinterpret_cast<__nv_bfloat162*>(&out);
#pragma unroll
    for (int e = 0; e < 4; ++e)
      o2[e] = __floats2bfloat162_rn(v[2 * e] * cc[e] - v[2 * e + 1] * sn[e], v[2 * e + 1] * cc[e] + v[2 * e] * sn[e]);
    *reinterpret_cast<uint4*>(to) = out;
  }
  __syncthreads();
  float tot = 0.f;
#pragma unroll
  for (int k = 0; k < kLatentThreads / 32; ++k) tot += part[k];
  const float f = 1.0f / sqrtf(tot / (float)a.rank + a.eps);
  if (has) {
    const __nv_bfloat162* w2 = reinterpret_cast<const __nv_bfloat162*>(&w);
    const float2 w0 = __bfloat1622float2(w2[0]), w1 = __bfloat1622float2(w2[1]);
    __nv_bfloat162 o[2] = {__floats2bfloat162_rn(x.x * f * w0.x, x.y * f * w0.y), __floats2bfloat162_rn(x.z * f * w1.x, x.w * f * w1.y)};
    *reinterpret_cast<uint2*>(dst + tid * 4) = *reinterpret_cast<uint2*>(o);
  }
}

// One warp per gathered row; V: the widest word that divides a row.
constexpr int kGatherWarps = 8;

template <typename V>
__global__ void __launch_bounds__(kGatherWarps * 32) latent_gather_kernel(const V* cache, int width, int max_len, const int32_t* row_start,
                                                                          const int32_t* kv_begin, const int32_t* base_len, int B,
                                                                          int mask_kind, int window, V* out, int rows_max,
                                                                          int32_t* out_begin, int32_t* n_out) {
  rd::pdl_launch_dependents();
  rd::pdl_wait();
  const int r = blockIdx.x * kGatherWarps + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  // which batch row holds gathered row r: the lanes take 32 batch rows at a time
  int at = 0, my_b = -1, my_j = 0;
  for (int b0 = 0; b0 < B; b0 += 32) {
    const int b = b0 + lane;
    int lo = 0, n = 0;
    if (b < B) {
      const int base = base_len[b], n_new = row_start[b + 1] - row_start[b];
      lo = rd_win::first_visible(mask_kind, window, base);
      lo = lo < 0 ? 0 : lo / RD_GATHER_ALIGN * RD_GATHER_ALIGN;
      n = n_new > 0 ? base + n_new - lo : 0;
    }
    int end = n;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int v = __shfl_up_sync(0xffffffffu, end, o);
      if (lane >= o) end += v;
    }
    const int begin = at + end - n;  // of this lane's batch row
    if (b < B && blockIdx.x == 0 && threadIdx.x < 32) out_begin[b] = begin - lo;
    const uint32_t hit = __ballot_sync(0xffffffffu, r >= begin && r < begin + n);
    const int who = hit ? __ffs(hit) - 1 : 0;
    const int j = __shfl_sync(0xffffffffu, lo + r - begin, who);
    if (hit) my_b = b0 + who, my_j = j;
    at += __shfl_sync(0xffffffffu, end, 31);
  }
  const int total = at + RD_GATHER_ALIGN - 1;
  if (blockIdx.x == 0 && threadIdx.x == 0) *n_out = total < rows_max ? total : rows_max;
  if (r >= total || r >= rows_max) return;
  V* dst = out + (int64_t)r * width;
  if (my_b < 0) {
    for (int d = lane; d < width; d += 32) dst[d] = V{};
    return;
  }
  const V* src = cache + ((int64_t)my_b * max_len + kv_begin[my_b] + my_j) * width;
  for (int d = lane; d < width; d += 32) dst[d] = src[d];
}

template <typename V>
int gather(const void* cache, int width, int max_len, const int32_t* row_start, const int32_t* kv_begin, const int32_t* base_len, int B,
           int mask_kind, int window, void* out, int rows_max, int32_t* out_begin, int32_t* n_out, cudaStream_t s) {
  cudaError_t err = rd::launch_chained(latent_gather_kernel<V>, dim3((rows_max + kGatherWarps - 1) / kGatherWarps), dim3(kGatherWarps * 32), 0, s,
                                       1, (const V*)cache, width, max_len, row_start, kv_begin, base_len, B, mask_kind, window, (V*)out,
                                       rows_max, out_begin, n_out);
  RD_CHECK_CHAINED(err);
  return RD_OK;
}

bool rotation_ok(int rot, int dim, const float* cos_t, const float* sin_t, int n_pos) {
  return rot >= 0 && rot % 2 == 0 && rot <= dim && n_pos >= 1 && (rot == 0 || (cos_t && sin_t));
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

extern "C" int rd_rotary_norm_append(int dtype, void* proj, int64_t ld, void* k_cache, void* v_cache, const int32_t* tok_row,
                                     const int32_t* tok_pos, const int32_t* tok_slot, const float* cos_table, const float* sin_table,
                                     int n_pos, int m_max, const int32_t* m_dev, int nh, int nkv, int dim, int vdim, int rot_dims,
                                     int neighbours, float eps, int max_len, void* stream) {
  RD_REQUIRE(proj && k_cache && v_cache && tok_row && tok_pos && tok_slot, RD_ERR_ARG);
  RD_REQUIRE(m_max >= 1 && nh >= 1 && nkv >= 1 && dim >= 1 && vdim >= 0 && max_len >= 1 &&
                 rotation_ok(rot_dims, dim, cos_table, sin_table, n_pos) && ld >= (int64_t)(nh + nkv) * dim + (int64_t)nkv * vdim,
             RD_ERR_SIZE);
  const HeadArgs a{ld, tok_row, tok_pos, tok_slot, cos_table, sin_table, n_pos, m_max, m_dev, nh, nkv, dim, vdim, rot_dims, neighbours, eps, max_len};
  cudaError_t err = cudaSuccess;
  RD_DISPATCH_T(dtype, (err = rd::launch_chained(rotary_norm_append_kernel<T>, dim3(m_max), dim3(kHeadThreads), 0, (cudaStream_t)stream, 1,
                                                 (T*)proj, (T*)k_cache, (T*)v_cache, a)));
  RD_CHECK_CHAINED(err);
  return RD_OK;
}

extern "C" int rd_latent_append(int dtype, const void* q, int64_t ldq, void* q_rot, int64_t ld_rot, int64_t rot_head, const float* dkv,
                                int64_t ld_dkv, const void* norm_weight, float eps, void* cache, const int32_t* tok_row,
                                const int32_t* tok_pos, const int32_t* tok_slot, const float* cos_table, const float* sin_table,
                                int n_pos, int m_max, const int32_t* m_dev, int nh, int dim, int rot_dim, int rot_dims, int neighbours,
                                int rank, int max_len, void* stream) {
  RD_REQUIRE(q && q_rot && dkv && norm_weight && cache && tok_row && tok_pos && tok_slot, RD_ERR_ARG);
  RD_REQUIRE(m_max >= 1 && nh >= 1 && dim >= 1 && rot_dim >= 0 && rank >= 1 && max_len >= 1 && ld_dkv >= rank + rot_dim &&
                 rotation_ok(rot_dims, rot_dim, cos_table, sin_table, n_pos) && ldq >= (int64_t)nh * (dim + rot_dim),
             RD_ERR_SIZE);
  const uintptr_t bits = (uintptr_t)q | (uintptr_t)q_rot | (uintptr_t)norm_weight | (uintptr_t)cache | (uintptr_t)dkv | (uintptr_t)cos_table | (uintptr_t)sin_table;
  const bool vec = dtype == RD_BF16 && neighbours && rot_dims == rot_dim && rot_dim > 0 && bits % 16 == 0 && ld_dkv % 4 == 0 &&
                   (ldq | ld_rot | rot_head | dim | rot_dim | rank) % 8 == 0 && rank <= 4 * kLatentThreads;
  const LatentArgs a{ldq, ld_rot, rot_head, ld_dkv, dkv, eps, tok_row, tok_pos, tok_slot, cos_table, sin_table, n_pos, m_max, m_dev,
                     nh, dim, rot_dim, rot_dims, neighbours, rank, max_len};
  cudaError_t err = cudaSuccess;
  if (vec)
    err = rd::launch_chained(latent_append_vec_kernel, dim3(m_max), dim3(kLatentThreads), 0, (cudaStream_t)stream, 1, (const __nv_bfloat16*)q,
                             (__nv_bfloat16*)q_rot, (const __nv_bfloat16*)norm_weight, (__nv_bfloat16*)cache, a);
  else
    RD_DISPATCH_T(dtype, (err = rd::launch_chained(latent_append_kernel<T>, dim3(m_max), dim3(kLatentThreads), 0, (cudaStream_t)stream, 1,
                                                 (const T*)q, (T*)q_rot, (const T*)norm_weight, (T*)cache, a)));
  RD_CHECK_CHAINED(err);
  return RD_OK;
}

extern "C" int rd_latent_gather(int dtype, const void* cache, int width, int max_len, const int32_t* row_start, const int32_t* kv_begin,
                                const int32_t* base_len, int B, int mask_kind, int window, void* out, int rows_max, int32_t* out_begin,
                                int32_t* n_out, void* stream) {
  RD_REQUIRE(cache && row_start && kv_begin && base_len && out && out_begin && n_out, RD_ERR_ARG);
  RD_REQUIRE(dtype == RD_F32 || dtype == RD_BF16, RD_ERR_DTYPE);
  RD_REQUIRE(width >= 1 && max_len >= 1 && B >= 1 && rows_max >= 1 && window >= 1 && (mask_kind == RD_MASK_WINDOW || mask_kind == RD_MASK_CHUNK),
             RD_ERR_SIZE);
  const int64_t bytes = (int64_t)width * (dtype == RD_F32 ? 4 : 2);
  cudaStream_t s = (cudaStream_t)stream;
  if (bytes % 16 == 0 && ((uintptr_t)cache | (uintptr_t)out) % 16 == 0)
    return gather<uint4>(cache, (int)(bytes / 16), max_len, row_start, kv_begin, base_len, B, mask_kind, window, out, rows_max, out_begin, n_out, s);
  if (bytes % 4 == 0)
    return gather<uint32_t>(cache, (int)(bytes / 4), max_len, row_start, kv_begin, base_len, B, mask_kind, window, out, rows_max, out_begin, n_out, s);
  return gather<uint16_t>(cache, (int)(bytes / 2), max_len, row_start, kv_begin, base_len, B, mask_kind, window, out, rows_max, out_begin, n_out, s);
}
