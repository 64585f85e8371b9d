// Matrix-memory recurrence with exponential gates (mLSTM).  Per row and head a state S [dim, vdim], a
// normaliser n [dim] and a running maximum m, all fp32:
//   i = cap tanh((zi + bi) / cap),  f = logsigmoid(cap tanh((zf + bf) / cap)),  m' = max(f + m, i)
//   S' = e^(f + m - m') S + e^(i - m') k v^T,  n' = e^(f + m - m') n + e^(i - m') k
//   o = S'^T q / (max(|n' . q|, e^(-m')) + 1e-6),  q scaled by dim^(-1/2)
// followed by the RMS norm of every head's o, the norm weight and the output gate sigmoid(g).
#include <cooperative_groups.h>

#include "mlstm_common.cuh"

namespace cg = cooperative_groups;

namespace {

using namespace rd_mlstm;

struct MlstmArgs {
  const void* proj;     // [m, ld]: q [nh*dim] | k [nh*dim] | v [nh*vdim] | g [nh*vdim]
  int64_t ld;
  const float* gates;   // [m, ld_gates]: zi [nh] | zf [nh]
  int64_t ld_gates;
  const float* bias_i;  // [nh]
  const float* bias_f;
  float cap;
  const void* norm_w;   // [nh*vdim]
  float eps;
  void* out;            // [m, nh*vdim]; null: the state only
  float* S;             // [B, nh, dim, vdim]
  float* n;             // [B, nh, dim]
  float* m;             // [B, nh]
  const int32_t* row_start;
  const int32_t* base_len;   // a row whose base_len is 0 starts from the zero state, whatever memory holds
  // optional indirection (commit of an accepted draft path): row b runs the tokens
  // row_start[b] + path[(b * W + seq[b]) * Lb + j], j = 0 .. count[b]
  const int32_t* path;
  int W, Lb;
  const int32_t* seq;
  const int32_t* count;
  int nh, dim, vdim, slice;  // slice: value columns per CTA
};

constexpr int kScanThreads = 256;

// Token after token.  Cluster of CTAs per (head, row), each with `slice` value columns; the head's sum of
// squares is exchanged through distributed shared memory.  The state slice stays in shared memory when the
// row brings several tokens (smem_state), otherwise it passes through registers once.
template <typename T, int VEC>
__global__ void __launch_bounds__(kScanThreads) mlstm_scan_kernel(const MlstmArgs a, int smem_state) {
  cg::cluster_group cluster = cg::this_cluster();
  extern __shared__ __align__(16) float smem[];
  rd::pdl_launch_dependents();
  rd::pdl_wait();
  const int b = blockIdx.z, h = blockIdx.y;
  const int rank = (int)cluster.block_rank(), n_ranks = (int)cluster.num_blocks();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int rs = a.row_start[b];
  const int n_tok = a.path ? min(a.count[b] + 1, a.Lb) : a.row_start[b + 1] - rs;
  if (n_tok <= 0) return;  // the same for every CTA of the cluster
  const int32_t* path = a.path ? a.path + ((int64_t)b * a.W + a.seq[b]) * a.Lb : nullptr;
  const int dim = a.dim, vdim = a.vdim;
  const int c0 = rank * a.slice;
  const int cols = max(0, min(a.slice, vdim - c0));
  const int col_units = cols / VEC;                          // VEC divides cols when VEC == 4
  const int lanes_c = a.slice / VEC;                         // threads along the columns
  const int rows_par = kScanThreads / lanes_c;               // threads along the rows
  const int tc = tid % lanes_c, tr = tid / lanes_c;
  const bool active = tc < col_units && tr < rows_par;

  const int dim4 = (dim + 3) & ~3;         // keeps the state slice on a 16-byte boundary
  float* q_s = smem;                       // [dim]
  float* k_s = q_s + dim4;                 // [dim]
  float* n_s = k_s + dim4;                 // [dim]
  float* red = n_s + dim4;                 // [rows_par][slice]
  float* warp_red = red + rows_par * a.slice;  // [8]
  float* ssq = warp_red + 8;               // [2]: this CTA's sum of squares, double-buffered over the tokens
  float* S_s = ssq + 2 + 6;                // [dim][slice] when smem_state

  const bool fresh = a.base_len[b] == 0;
  float* S_g = a.S + ((int64_t)b * a.nh + h) * dim * vdim + c0;
  float* n_g = a.n + ((int64_t)b * a.nh + h) * dim;
  for (int d = tid; d < dim; d += kScanThreads) n_s[d] = fresh ? 0.f : n_g[d];
  float m = fresh ? 0.f : a.m[(int64_t)b * a.nh + h];
  if (smem_state && active) {
    for (int r = tr; r < dim; r += rows_par)
#pragma unroll
      for (int e = 0; e < VEC; ++e) S_s[r * a.slice + tc * VEC + e] = fresh ? 0.f : S_g[(int64_t)r * vdim + tc * VEC + e];
  }
  const float qscale = rsqrtf((float)dim);
  const float bi = a.bias_i[h], bf = a.bias_f[h];

  for (int it = 0; it < n_tok; ++it) {
    const int t = rs + (path ? path[it] : it);
    const T* row = (const T*)a.proj + (int64_t)t * a.ld;
    const T* qp = row + (int64_t)h * dim;
    const T* kp = row + (int64_t)(a.nh + h) * dim;
    const T* vp = row + (int64_t)2 * a.nh * dim + (int64_t)h * vdim + c0;
    for (int d = tid; d < dim; d += kScanThreads) {
      q_s[d] = rd::Num<T>::to_f(qp[d]) * qscale;
      k_s[d] = rd::Num<T>::to_f(kp[d]);
    }
    const float zi = soft_cap(a.gates[(int64_t)t * a.ld_gates + h] + bi, a.cap);
    const float zf = log_sigmoid(soft_cap(a.gates[(int64_t)t * a.ld_gates + a.nh + h] + bf, a.cap));
    const float m_new = fmaxf(zf + m, zi);
    const float fa = expf(zf + m - m_new), fb = expf(zi - m_new);
    m = m_new;
    float v[VEC];
#pragma unroll
    for (int e = 0; e < VEC; ++e) v[e] = active ? rd::Num<T>::to_f(vp[tc * VEC + e]) * fb : 0.f;
    __syncthreads();
    // state update and S^T q of this thread's rows
    float o[VEC];
#pragma unroll
    for (int e = 0; e < VEC; ++e) o[e] = 0.f;
    if (active) {
      if (smem_state) {
        float* sp = S_s + tc * VEC;
        for (int r = tr; r < dim; r += rows_par) {
          const float kk = k_s[r], qq = q_s[r];
          float s[VEC];
          if constexpr (VEC == 4) {
            *reinterpret_cast<float4*>(s) = *reinterpret_cast<const float4*>(sp + r * a.slice);
          } else {
            s[0] = sp[r * a.slice];
          }
#pragma unroll
          for (int e = 0; e < VEC; ++e) {
            s[e] = fmaf(fa, s[e], kk * v[e]);
            o[e] = fmaf(s[e], qq, o[e]);
          }
          if constexpr (VEC == 4) {
            *reinterpret_cast<float4*>(sp + r * a.slice) = *reinterpret_cast<const float4*>(s);
          } else {
            sp[r * a.slice] = s[0];
          }
        }
      } else {
        const bool zero = fresh && it == 0;
        float* sp = S_g + tc * VEC;
#pragma unroll 8
        for (int r = tr; r < dim; r += rows_par) {
          const float kk = k_s[r], qq = q_s[r];
          float s[VEC];
          if constexpr (VEC == 4) {
            *reinterpret_cast<float4*>(s) = zero ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4*>(sp + (int64_t)r * vdim);
          } else {
            s[0] = zero ? 0.f : sp[(int64_t)r * vdim];
          }
#pragma unroll
          for (int e = 0; e < VEC; ++e) {
            s[e] = fmaf(fa, s[e], kk * v[e]);
            o[e] = fmaf(s[e], qq, o[e]);
          }
          if constexpr (VEC == 4) {
            *reinterpret_cast<float4*>(sp + (int64_t)r * vdim) = *reinterpret_cast<const float4*>(s);
          } else {
            sp[(int64_t)r * vdim] = s[0];
          }
        }
      }
    }
    // normaliser: every CTA of the cluster keeps its own copy
    float nq = 0.f;
    for (int d = tid; d < dim; d += kScanThreads) {
      const float nn = fmaf(fa, n_s[d], fb * k_s[d]);
      n_s[d] = nn;
      nq = fmaf(nn, q_s[d], nq);
    }
    if (a.out != nullptr) {
      nq = rd::warp_sum(nq);
      if (lane == 0) warp_red[warp] = nq;
      if (active) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) red[tr * a.slice + tc * VEC + e] = o[e];
      }
      __syncthreads();
      float dot = 0.f;
#pragma unroll
      for (int w = 0; w < kScanThreads / 32; ++w) dot += warp_red[w];
      const float inv = 1.0f / (fmaxf(fabsf(dot), expf(-m)) + kDenEps);
      // column c of this CTA belongs to thread c (slice <= kScanThreads)
      float oc = 0.f;
      if (tid < cols) {
        for (int r = 0; r < rows_par; ++r) oc += red[r * a.slice + tid];
        oc *= inv;
      }
      float ss = rd::warp_sum(tid < cols ? oc * oc : 0.f);
      __syncthreads();  // warp_red has been read
      if (lane == 0) warp_red[warp] = ss;
      __syncthreads();
      if (tid == 0) {
        float tot = 0.f;
#pragma unroll
        for (int w = 0; w < kScanThreads / 32; ++w) tot += warp_red[w];
        ssq[it & 1] = tot;
      }
      // everyone's share is written; also: every CTA has read n and m before any of them is written back
      cluster.sync();
      float tot = 0.f;
      for (int r = 0; r < n_ranks; ++r) tot += *cluster.map_shared_rank(&ssq[it & 1], r);
      if (tid < cols) {
        const float rms = 1.0f / sqrtf(tot / (float)vdim + a.eps);
        const int col = h * vdim + c0 + tid;
        const float g = rd::Num<T>::to_f(row[(int64_t)2 * a.nh * dim + (int64_t)a.nh * vdim + col]);
        const float y = oc * rms * rd::Num<T>::to_f(((const T*)a.norm_w)[col]) / (1.0f + expf(-g));
        ((T*)a.out)[(int64_t)t * a.nh * vdim + col] = rd::Num<T>::from_f(y);
      }
    } else {
      __syncthreads();  // q_s / k_s are rewritten by the next token
    }
  }
  if (smem_state && active) {
    for (int r = tr; r < dim; r += rows_par)
#pragma unroll
      for (int e = 0; e < VEC; ++e) S_g[(int64_t)r * vdim + tc * VEC + e] = S_s[r * a.slice + tc * VEC + e];
  }
  // peers may still read this CTA's shared memory, and have read n and m before they change
  cluster.sync();
  if (rank == 0) {
    for (int d = tid; d < dim; d += kScanThreads) n_g[d] = n_s[d];
    if (tid == 0) a.m[(int64_t)b * a.nh + h] = m;
  }
}

template <typename T>
int launch_scan(const MlstmArgs& a0, int B, int max_new, cudaStream_t s) {
  MlstmArgs a = a0;
  const bool vec = a.vdim % 4 == 0 && ((uintptr_t)a.S & 15) == 0;
  // value columns per CTA: at most 8 CTAs per head, at least 32 columns each, at most one column per thread
  int ranks = 1;
  while (ranks < 8 && a.vdim / (ranks * 2) >= 32) ranks *= 2;
  int slice = (a.vdim + ranks - 1) / ranks;
  slice = (slice + 3) / 4 * 4;
  RD_REQUIRE(slice <= kScanThreads, RD_ERR_SIZE);
  a.slice = slice;
  const int lanes_c = vec ? slice / 4 : slice;
  const int rows_par = kScanThreads / lanes_c;
  const size_t fixed = ((size_t)3 * ((a.dim + 3) & ~3) + (size_t)rows_par * slice + 16) * sizeof(float);
  const size_t state = (size_t)a.dim * slice * sizeof(float);
  const int smem_state = max_new > 1 && fixed + state <= 200 * 1024;
  const size_t smem = fixed + (smem_state ? state : 0);
  RD_REQUIRE(smem <= 200 * 1024, RD_ERR_SIZE);
  auto kern = vec ? mlstm_scan_kernel<T, 4> : mlstm_scan_kernel<T, 1>;
  if (smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    RD_CHECK_CHAINED(e);
  }
  cudaError_t err = rd::launch_chained(kern, dim3(ranks, a.nh, B), dim3(kScanThreads), smem, s, ranks, a, smem_state);
  RD_CHECK_CHAINED(err);
  return RD_OK;
}

// Packed draft trees: every new token continues the row's state along its own path of ancestors (tree_mask, itself
// included; ascending packed index is root to leaf), and the state is left as it was.  With the path's tokens 1 .. k,
//   num = e^(sum f + m - m_k) S^T q + sum_j e^(f_(j+1) + .. + f_k + i_j - m_k) (q . k_j) v_j
// and the denominator likewise.  A CTA holds 64 value columns of the state in shared memory; a warp takes four tokens
// at a time.  Writes o in fp32; launch_norm_gate() follows.
constexpr int kTreeCols = 64;
constexpr int kTreeTok = 4;
constexpr int kTreeWarps = 8;

template <typename T>
__global__ void __launch_bounds__(kTreeWarps * 32) mlstm_tree_kernel(const MlstmArgs a, const uint32_t* tree_mask,
                                                                    int mask_words, float* o_out) {
  extern __shared__ __align__(16) float smem[];
  rd::pdl_launch_dependents();
  rd::pdl_wait();
  const int b = blockIdx.z, h = blockIdx.y, c0 = blockIdx.x * kTreeCols;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int rs = a.row_start[b], n_tok = a.row_start[b + 1] - rs;
  if (n_tok <= 0) return;
  const int dim = a.dim, vdim = a.vdim;
  float* S_s = smem;                                      // [dim][kTreeCols]
  float* q_s = S_s + dim * kTreeCols + warp * dim * kTreeTok;  // [dim][kTreeTok]
  const bool fresh = a.base_len[b] == 0;
  const float* S_g = a.S + ((int64_t)b * a.nh + h) * dim * vdim;
  const float* n_g = a.n + ((int64_t)b * a.nh + h) * dim;
  for (int i = tid; i < dim * kTreeCols; i += kTreeWarps * 32) {
    const int d = i / kTreeCols, c = c0 + i % kTreeCols;
    S_s[i] = (c < vdim && !fresh) ? S_g[(int64_t)d * vdim + c] : 0.f;
  }
  __syncthreads();
  const float m0 = fresh ? 0.f : a.m[(int64_t)b * a.nh + h];
  const float qscale = rsqrtf((float)dim);
  const float bi = a.bias_i[h], bf = a.bias_f[h];
  const int ca = c0 + lane * 2;  // this lane's two value columns
  for (int i0 = warp * kTreeTok; i0 < n_tok; i0 += kTreeWarps * kTreeTok) {
    float nq[kTreeTok];
#pragma unroll
    for (int u = 0; u < kTreeTok; ++u) {
      const T* qp = (const T*)a.proj + (int64_t)(rs + min(i0 + u, n_tok - 1)) * a.ld + (int64_t)h * dim;
      float acc = 0.f;
      for (int d = lane; d < dim; d += 32) {
        const float qv = rd::Num<T>::to_f(qp[d]) * qscale;
        q_s[d * kTreeTok + u] = qv;
        acc = fmaf(qv, fresh ? 0.f : n_g[d], acc);
      }
      nq[u] = rd::warp_sum(acc);
    }
    __syncwarp();
    float x[kTreeTok][2];
#pragma unroll
    for (int u = 0; u < kTreeTok; ++u) x[u][0] = x[u][1] = 0.f;
    for (int d = 0; d < dim; ++d) {
      const float2 s2 = *reinterpret_cast<const float2*>(S_s + d * kTreeCols + lane * 2);
      const float4 q4 = *reinterpret_cast<const float4*>(q_s + d * kTreeTok);
      const float qv[4] = {q4.x, q4.y, q4.z, q4.w};
#pragma unroll
      for (int u = 0; u < kTreeTok; ++u) {
        x[u][0] = fmaf(s2.x, qv[u], x[u][0]);
        x[u][1] = fmaf(s2.y, qv[u], x[u][1]);
      }
    }
#pragma unroll
    for (int u = 0; u < kTreeTok; ++u) {
      const int i = i0 + u;
      if (i >= n_tok) break;
      const uint32_t* mask = tree_mask + (int64_t)(rs + i) * mask_words;
      int anc[RD_MAX_BEAM_LENGTH];
      float fg[RD_MAX_BEAM_LENGTH], ig[RD_MAX_BEAM_LENGTH];
      int depth = 0;
      float m = m0, sum_f = 0.f;
      for (int wd = 0; wd < mask_words; ++wd) {
        uint32_t bits = mask[wd];
        while (bits != 0u && depth < RD_MAX_BEAM_LENGTH) {
          const int jn = wd * 32 + __ffs(bits) - 1;
          bits &= bits - 1u;
          const float* gp = a.gates + (int64_t)(rs + jn) * a.ld_gates + h;
          const float ii = soft_cap(gp[0] + bi, a.cap), ff = log_sigmoid(soft_cap(gp[a.nh] + bf, a.cap));
          m = fmaxf(ff + m, ii);
          sum_f += ff;
#pragma unroll
          for (int e = 0; e < RD_MAX_BEAM_LENGTH; ++e)
            if (e == depth) {
              anc[e] = jn;
              fg[e] = ff;
              ig[e] = ii;
            }
          ++depth;
        }
      }
      const float inter = expf(sum_f + m0 - m);
      float y0 = x[u][0] * inter, y1 = x[u][1] * inter, den = nq[u] * inter;
      float tail = 0.f;  // sum of the log forget gates after token e of the path
#pragma unroll
      for (int e = RD_MAX_BEAM_LENGTH - 1; e >= 0; --e) {
        if (e >= depth) continue;
        const T* row = (const T*)a.proj + (int64_t)(rs + anc[e]) * a.ld;
        const T* kp = row + (int64_t)(a.nh + h) * dim;
        float dot = 0.f;
        for (int d = lane; d < dim; d += 32) dot = fmaf(q_s[d * kTreeTok + u], rd::Num<T>::to_f(kp[d]), dot);
        const float p = rd::warp_sum(dot) * expf(tail + ig[e] - m);
        tail += fg[e];
        den += p;
        const T* vp = row + (int64_t)2 * a.nh * dim + (int64_t)h * vdim;
        if (ca < vdim) y0 = fmaf(p, rd::Num<T>::to_f(vp[ca]), y0);
        if (ca + 1 < vdim) y1 = fmaf(p, rd::Num<T>::to_f(vp[ca + 1]), y1);
      }
      const float inv = 1.0f / (fmaxf(fabsf(den), expf(-m)) + kDenEps);
      float* dst = o_out + ((int64_t)(rs + i) * a.nh + h) * vdim;
      if (ca < vdim) dst[ca] = y0 * inv;
      if (ca + 1 < vdim) dst[ca + 1] = y1 * inv;
    }
    __syncwarp();
  }
}

template <typename T>
int launch_tree(const MlstmArgs& a, int B, int m_max, const uint32_t* tree_mask, int mask_words, float* o, cudaStream_t s) {
  const size_t smem = (size_t)a.dim * (kTreeCols + kTreeWarps * kTreeTok) * sizeof(float);
  RD_REQUIRE(smem <= 200 * 1024, RD_ERR_SIZE);
  auto kern = mlstm_tree_kernel<T>;
  if (smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    RD_CHECK_CHAINED(e);
  }
  cudaError_t err = rd::launch_chained(kern, dim3((a.vdim + kTreeCols - 1) / kTreeCols, a.nh, B), dim3(kTreeWarps * 32), smem, s, 1, a,
                                       tree_mask, mask_words, o);
  RD_CHECK_CHAINED(err);
  const T* gp = (const T*)a.proj + (int64_t)2 * a.nh * a.dim + (int64_t)a.nh * a.vdim;
  return launch_norm_gate<T>(o, gp, a.ld, a.norm_w, a.out, a.eps, m_max, a.row_start, B, a.nh, a.vdim, s);
}

}  // namespace

extern "C" int rd_mlstm_tree(int dtype, const void* proj, int64_t ld, const float* gates, int64_t ld_gates, const float* bias_i,
                             const float* bias_f, float gate_cap, const void* norm_weight, float eps, void* out, const float* S,
                             const float* n, const float* m, const int32_t* row_start, const int32_t* base_len, int B, int nh,
                             int dim, int vdim, int m_max, const uint32_t* tree_mask, int mask_words, float* workspace,
                             int64_t workspace_bytes, void* stream) {
  RD_REQUIRE(proj && gates && bias_i && bias_f && S && n && m && row_start && base_len && norm_weight && out && tree_mask && workspace,
             RD_ERR_ARG);
  RD_REQUIRE(B >= 1 && B <= 65535 && nh >= 1 && nh <= 65535 && dim >= 1 && vdim >= 1 && m_max >= 1 && gate_cap > 0.f &&
                 mask_words >= 1 && ld >= 2 * (int64_t)nh * (dim + vdim) && ld_gates >= 2 * nh,
             RD_ERR_SIZE);
  RD_REQUIRE(workspace_bytes >= (int64_t)m_max * nh * vdim * (int64_t)sizeof(float), RD_ERR_CAPACITY);
  MlstmArgs a{proj, ld,  gates, ld_gates,  bias_i,   bias_f, gate_cap, norm_weight, eps, out, const_cast<float*>(S), const_cast<float*>(n),
              const_cast<float*>(m), row_start, base_len, nullptr, 0, 0, nullptr, nullptr, nh, dim, vdim, 0};
  if (dtype == RD_F32) return launch_tree<float>(a, B, m_max, tree_mask, mask_words, workspace, (cudaStream_t)stream);
  if (dtype == RD_BF16) return launch_tree<__nv_bfloat16>(a, B, m_max, tree_mask, mask_words, workspace, (cudaStream_t)stream);
  return RD_ERR_DTYPE;
}

extern "C" int rd_mlstm_scan(int dtype, const void* proj, int64_t ld, const float* gates, int64_t ld_gates, const float* bias_i,
                             const float* bias_f, float gate_cap, const void* norm_weight, float eps, void* out, float* S,
                             float* n, float* m, const int32_t* row_start, const int32_t* base_len, int B, int nh, int dim,
                             int vdim, int max_new, const int32_t* path, int W, int Lb, const int32_t* seq,
                             const int32_t* count, void* stream) {
  RD_REQUIRE(proj && gates && bias_i && bias_f && S && n && m && row_start && base_len && (norm_weight || !out), RD_ERR_ARG);
  RD_REQUIRE(B >= 1 && B <= 65535 && nh >= 1 && nh <= 65535 && dim >= 1 && vdim >= 1 && max_new >= 1 && gate_cap > 0.f &&
                 ld >= 2 * (int64_t)nh * (dim + vdim) && ld_gates >= 2 * nh,
             RD_ERR_SIZE);
  RD_REQUIRE(!path || (seq && count && W >= 1 && Lb >= 1), RD_ERR_ARG);
  MlstmArgs a{proj, ld,  gates, ld_gates,  bias_i,   bias_f, gate_cap, norm_weight, eps,   out, S,  n,
              m,    row_start, base_len, path, W, Lb, seq, count, nh, dim, vdim, 0};
  if (dtype == RD_F32) return launch_scan<float>(a, B, max_new, (cudaStream_t)stream);
  if (dtype == RD_BF16) return launch_scan<__nv_bfloat16>(a, B, max_new, (cudaStream_t)stream);
  return RD_ERR_DTYPE;
}
