// Attention over a sliding window or a chunk with kept first tokens, grouped key/value heads, different key and value
// sizes, a free score scale, an output gate and a sink per head, and key features that all heads share (see
// attention_window.cuh for the visibility rule).
//
//   attention_window_rowwise_kernel  any dtype and size: one warp per (query, head), online softmax over 32 keys
//                                    at a time, exact expf.  fp32 models and odd sizes.
//   attention_window_prefill_kernel,  bf16 on warp-level tensor cores (attention_window_tc.cuh): head sizes up to 128
//   attention_window_decode_kernel    in multiples of 8 (decode: values up to 256).
#include "attention_window_tc.cuh"

namespace {

constexpr int kRowWarps = 8;

// kMaxV: value features per lane
template <typename T, int kMaxV>
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
  rd_win::RowKeys<T> keys;
  keys.init(a, b, hk);
  const int own = a.dim - a.tail_dim;  // key features that belong to the head
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
        const T* kr = keys.k + (int64_t)j * a.k_row;
        float dot = 0.f;
        for (int d = 0; d < own; ++d) dot = fmaf(qs[d], rd::Num<T>::to_f(kr[d]), dot);
        if (a.tail_dim > 0) {
          const T* tr = keys.tail + (int64_t)j * a.tail_row;
          for (int d = own; d < a.dim; ++d) dot = fmaf(qs[d], rd::Num<T>::to_f(tr[d - own]), dot);
        }
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
        const T* vr = keys.v + (int64_t)(j0 + jj) * a.v_row;
#pragma unroll
        for (int v = 0; v < kMaxV; ++v)
          if (v * 32 + lane < a.vdim) acc[v] = fmaf(pj, rd::Num<T>::to_f(vr[v * 32 + lane]), acc[v]);
      }
    }
  }
  float f = l > 0.f ? 1.0f / l : 0.f;
  if (a.sink != nullptr && l > 0.f) {
    const float s = a.sink[h], top = fmaxf(m, s), w = expf(m - top);
    f = w / (l * w + expf(s - top));
  }
  if (a.gate != nullptr) f *= rd_win::sigmoid_exact(rd::Num<T>::to_f(((const T*)a.gate)[(int64_t)t * a.ld_gate + h]));
  T* orow = (T*)a.out + ((int64_t)t * a.nh + h) * a.vdim;
#pragma unroll
  for (int v = 0; v < kMaxV; ++v)
    if (v * 32 + lane < a.vdim) orow[v * 32 + lane] = rd::Num<T>::from_f(acc[v] * f);
}

template <typename T, int kMaxV>
int launch_rowwise_v(const rd_win::Args& a, cudaStream_t s) {
  const size_t smem = (size_t)kRowWarps * a.dim * sizeof(float);
  RD_REQUIRE(smem <= 48 * 1024, RD_ERR_SIZE);
  dim3 grid((a.max_new + kRowWarps - 1) / kRowWarps, a.nh, a.B);
  cudaError_t err = rd::launch_chained(attention_window_rowwise_kernel<T, kMaxV>, grid, dim3(kRowWarps * 32), smem, s, 1, a);
  RD_CHECK_CHAINED(err);
  return RD_OK;
}

template <typename T>
int launch_rowwise(const rd_win::Args& a, cudaStream_t s) {
  if (a.vdim <= 8 * 32) return launch_rowwise_v<T, 8>(a, s);
  if (a.vdim <= 16 * 32) return launch_rowwise_v<T, 16>(a, s);
  RD_REQUIRE(a.vdim <= 32 * 32, RD_ERR_SIZE);
  return launch_rowwise_v<T, 32>(a, s);
}

}  // namespace

extern "C" int rd_attention_masked(const rd_attention_desc* desc, void* stream) {
  RD_REQUIRE(desc, RD_ERR_ARG);
  const rd_win::Args& a = *desc;
  RD_REQUIRE(a.q && a.k && a.v && a.out && a.row_start && a.kv_begin && a.base_len, RD_ERR_ARG);
  RD_REQUIRE(a.mode == RD_ATTN_CAUSAL || (a.mode == RD_ATTN_TREE && a.tree_mask && a.tok_pos && a.mask_words >= 1), RD_ERR_ARG);
  RD_REQUIRE(a.dtype == RD_F32 || a.dtype == RD_BF16, RD_ERR_DTYPE);
  RD_REQUIRE(a.mask_kind == RD_MASK_WINDOW || a.mask_kind == RD_MASK_CHUNK, RD_ERR_ARG);
  RD_REQUIRE(a.B >= 1 && a.B <= 65535 && a.nh >= 1 && a.nh <= 65535 && a.nkv >= 1 && a.nh % a.nkv == 0 && a.dim >= 1 && a.vdim >= 1 &&
                 a.max_new >= 1 && a.window >= 1 && a.keep_first >= 0 && a.ldq >= (int64_t)a.nh * a.dim && a.tail_dim >= 0 &&
                 a.tail_dim < a.dim && (a.tail_dim == 0 || a.k_tail),
             RD_ERR_SIZE);
  cudaStream_t s = (cudaStream_t)stream;
  if (a.dtype == RD_F32) return launch_rowwise<float>(a, s);
  const uintptr_t bits = (uintptr_t)a.q | (uintptr_t)a.k | (uintptr_t)a.v | (uintptr_t)a.out | (uintptr_t)(a.tail_dim ? a.k_tail : nullptr);
  const int64_t strides = a.ldq | a.k_batch | a.k_head | a.k_row | a.v_batch | a.v_head | a.v_row |
                          (a.tail_dim ? a.tail_batch | a.tail_row | a.tail_dim : 0);
  if (a.dim % 8 == 0 && a.vdim % 8 == 0 && strides % 8 == 0 && bits % 16 == 0 && a.dim <= 256 && a.vdim <= 256) {
    // two row tiles of queries per key/value head are still cheaper to read K and V for than one 128-query tile per head
    const bool decode = (a.nh / a.nkv) * a.max_new <= 2 * rd_win::kRows;
    if (decode) {
      if (a.dim <= 64 && a.vdim <= 64) return rd_win::launch_decode<64, 64>(a, s);
      if (a.dim <= 128 && a.vdim <= 128) return rd_win::launch_decode<128, 128>(a, s);
      return rd_win::launch_decode<256, 256>(a, s);
    }
    if (a.dim <= 64 && a.vdim <= 64) return rd_win::launch_prefill<64, 64>(a, s);
    if (a.dim <= 64 && a.vdim <= 128) return rd_win::launch_prefill<64, 128>(a, s);
    if (a.dim <= 128 && a.vdim <= 64) return rd_win::launch_prefill<128, 64>(a, s);
    if (a.dim <= 128 && a.vdim <= 128) return rd_win::launch_prefill<128, 128>(a, s);
  }
  return launch_rowwise<__nv_bfloat16>(a, s);
}

extern "C" int rd_attention_desc_bytes(void) { return (int)sizeof(rd_attention_desc); }

extern "C" int rd_attention_window(int dtype, const void* q, int64_t ldq, const void* k_cache, const void* v_cache,
                                   const void* gate, int64_t ld_gate, void* out, const int32_t* row_start,
                                   const int32_t* kv_begin, const int32_t* base_len, int B, int nh, int nkv, int dim, int vdim,
                                   int max_len, int max_new, int mode, const int32_t* tok_pos, const uint32_t* tree_mask,
                                   int mask_words, float scale, int window, int keep_first, int max_kv, void* stream) {
  RD_REQUIRE(max_len >= 1, RD_ERR_SIZE);
  rd_attention_desc a{};
  a.q = q, a.ldq = ldq;
  a.k = k_cache, a.k_row = dim, a.k_head = (int64_t)max_len * dim, a.k_batch = a.k_head * nkv;
  a.v = v_cache, a.v_row = vdim, a.v_head = (int64_t)max_len * vdim, a.v_batch = a.v_head * nkv;
  a.gate = gate, a.ld_gate = ld_gate;
  a.out = out;
  a.row_start = row_start, a.kv_begin = kv_begin, a.base_len = base_len, a.tok_pos = tok_pos;
  a.tree_mask = tree_mask, a.mask_words = mask_words;
  a.dtype = dtype, a.B = B, a.nh = nh, a.nkv = nkv, a.dim = dim, a.vdim = vdim, a.max_new = max_new, a.max_kv = max_kv, a.mode = mode;
  a.mask_kind = RD_MASK_WINDOW, a.window = window, a.keep_first = keep_first, a.scale = scale;
  return rd_attention_masked(&a, stream);
}
