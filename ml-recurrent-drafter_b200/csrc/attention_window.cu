// Sliding-window attention with kept first tokens, grouped key/value heads, different key and value sizes,
// a free score scale and an output gate per head (see attention_window.cuh for the visibility rule).
//
//   attention_window_rowwise_kernel  any dtype and size: one warp per (query, head), online softmax over 32 keys
//                                    at a time, exact expf.  fp32 models and odd sizes.
//   attention_window_prefill_kernel,  bf16 on warp-level tensor cores (attention_window_tc.cuh): head sizes up to 128
//   attention_window_decode_kernel    in multiples of 8 (decode: values up to 256).
#include "attention_window_tc.cuh"

namespace {

constexpr int kRowWarps = 8;
constexpr int kMaxV = 16;  // value features per lane: vdim <= 512

template <typename T>
__global__ void __launch_bounds__(kRowWarps * 32) attention_window_rowwise_kernel(const rd_win::Args a) {
  rd::pdl_launch_dependents();
  rd::pdl_wait();
  const int b = blockIdx.z, h = blockIdx.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int rs = a.row_start[b];
  const int n_new = a.row_start[b + 1] - rs;
  const int i = blockIdx.x * kRowWarps + warp;
  if (i >= n_new) return;
  extern __shared__ float smem[];
  float* qs = smem + (size_t)warp * a.dim;
  const int t = rs + i;
  const int hk = h / (a.nh / a.nkv);
  const T* qrow = (const T*)a.q + (int64_t)t * a.ldq + (int64_t)h * a.dim;
  for (int d = lane; d < a.dim; d += 32) qs[d] = rd::Num<T>::to_f(qrow[d]);
  __syncwarp();
  const int64_t row0 = ((int64_t)b * a.nkv + hk) * a.max_len + a.kv_begin[b];
  const T* kb = (const T*)a.k_cache + row0 * a.dim;
  const T* vb = (const T*)a.v_cache + row0 * a.vdim;
  rd_win::Query qu;
  qu.init(a, a.base_len[b], rs, n_new, i);
  float m = -INFINITY, l = 0.f;
  float acc[kMaxV];
#pragma unroll
  for (int v = 0; v < kMaxV; ++v) acc[v] = 0.f;
  // the kept tokens, then the window
  const int kept_end = min(a.keep_first, qu.kv_end);
  for (int part = 0; part < 2; ++part) {
    const int j_lo = part == 0 ? 0 : qu.lo, j_hi = part == 0 ? kept_end : qu.kv_end;
    for (int j0 = j_lo; j0 < j_hi; j0 += 32) {
      const int j = j0 + lane;
      float s = -INFINITY;
      if (j < j_hi && qu.sees(a, j)) {
        const T* kr = kb + (int64_t)j * a.dim;
        float dot = 0.f;
        for (int d = 0; d < a.dim; ++d) dot = fmaf(qs[d], rd::Num<T>::to_f(kr[d]), dot);
        s = dot * a.scale;
      }
      const float mt = rd::warp_max(s);
      if (mt == -INFINITY) continue;
      const float m_new = fmaxf(m, mt);
      const float alpha = m == -INFINITY ? 0.f : expf(m - m_new);
      const float p = s == -INFINITY ? 0.f : expf(s - m_new);
      m = m_new;
      l = l * alpha + rd::warp_sum(p);
#pragma unroll
      for (int v = 0; v < kMaxV; ++v) acc[v] *= alpha;
      const int n = min(32, j_hi - j0);
      for (int jj = 0; jj < n; ++jj) {
        const float pj = __shfl_sync(0xffffffffu, p, jj);
        if (pj == 0.f) continue;
        const T* vr = vb + (int64_t)(j0 + jj) * a.vdim;
#pragma unroll
        for (int v = 0; v < kMaxV; ++v)
          if (v * 32 + lane < a.vdim) acc[v] = fmaf(pj, rd::Num<T>::to_f(vr[v * 32 + lane]), acc[v]);
      }
    }
  }
  float f = l > 0.f ? 1.0f / l : 0.f;
  if (a.gate != nullptr) f *= rd_win::sigmoid_exact(rd::Num<T>::to_f(((const T*)a.gate)[(int64_t)t * a.ld_gate + h]));
  T* orow = (T*)a.out + ((int64_t)t * a.nh + h) * a.vdim;
#pragma unroll
  for (int v = 0; v < kMaxV; ++v)
    if (v * 32 + lane < a.vdim) orow[v * 32 + lane] = rd::Num<T>::from_f(acc[v] * f);
}

template <typename T>
int launch_rowwise(const rd_win::Args& a, int B, int max_new, cudaStream_t s) {
  const size_t smem = (size_t)kRowWarps * a.dim * sizeof(float);
  RD_REQUIRE(smem <= 48 * 1024 && a.vdim <= kMaxV * 32, RD_ERR_SIZE);
  dim3 grid((max_new + kRowWarps - 1) / kRowWarps, a.nh, B);
  cudaError_t err = rd::launch_chained(attention_window_rowwise_kernel<T>, grid, dim3(kRowWarps * 32), smem, s, 1, a);
  RD_CHECK_CHAINED(err);
  return RD_OK;
}

}  // namespace

extern "C" int rd_attention_window(int dtype, const void* q, int64_t ldq, const void* k_cache, const void* v_cache,
                                   const void* gate, int64_t ld_gate, void* out, const int32_t* row_start,
                                   const int32_t* kv_begin, const int32_t* base_len, int B, int nh, int nkv, int dim, int vdim,
                                   int max_len, int max_new, int mode, const int32_t* tok_pos, const uint32_t* tree_mask,
                                   int mask_words, float scale, int window, int keep_first, int max_kv, void* stream) {
  RD_REQUIRE(q && k_cache && v_cache && out && row_start && kv_begin && base_len, RD_ERR_ARG);
  RD_REQUIRE(mode == RD_ATTN_CAUSAL || (mode == RD_ATTN_TREE && tree_mask && tok_pos && mask_words >= 1), RD_ERR_ARG);
  RD_REQUIRE(dtype == RD_F32 || dtype == RD_BF16, RD_ERR_DTYPE);
  RD_REQUIRE(B >= 1 && B <= 65535 && nh >= 1 && nh <= 65535 && nkv >= 1 && nh % nkv == 0 && dim >= 1 && vdim >= 1 && max_len >= 1 &&
                 max_new >= 1 && window >= 1 && keep_first >= 0 && ldq >= (int64_t)nh * dim,
             RD_ERR_SIZE);
  rd_win::Args a{q,       ldq,     k_cache, v_cache,   gate,       ld_gate, out, row_start, kv_begin, base_len, tok_pos,
                 tree_mask, mask_words, nh,   nkv, dim, vdim, max_len, mode, scale, window, keep_first};
  cudaStream_t s = (cudaStream_t)stream;
  if (dtype == RD_F32) return launch_rowwise<float>(a, B, max_new, s);
  const uintptr_t bits = (uintptr_t)q | (uintptr_t)k_cache | (uintptr_t)v_cache | (uintptr_t)out;
  if (dim % 8 == 0 && vdim % 8 == 0 && ldq % 8 == 0 && bits % 16 == 0 && dim <= 256 && vdim <= 256) {
    // two row tiles of queries per key/value head are still cheaper to read K and V for than one 128-query tile per head
    const bool decode = (nh / nkv) * max_new <= 2 * rd_win::kRows;
    if (decode) {
      if (dim <= 64 && vdim <= 64) return rd_win::launch_decode<64, 64>(a, B, max_new, max_kv, s);
      if (dim <= 128 && vdim <= 128) return rd_win::launch_decode<128, 128>(a, B, max_new, max_kv, s);
      return rd_win::launch_decode<256, 256>(a, B, max_new, max_kv, s);
    }
    if (dim <= 64 && vdim <= 64) return rd_win::launch_prefill<64, 64>(a, B, max_new, s);
    if (dim <= 64 && vdim <= 128) return rd_win::launch_prefill<64, 128>(a, B, max_new, s);
    if (dim <= 128 && vdim <= 64) return rd_win::launch_prefill<128, 64>(a, B, max_new, s);
    if (dim <= 128 && vdim <= 128) return rd_win::launch_prefill<128, 128>(a, B, max_new, s);
  }
  return launch_rowwise<__nv_bfloat16>(a, B, max_new, s);
}
