// What the masked attention kernels share: which keys a query sees, and where to look for them.
//
// A row's keys lie in the slots kv_begin + j, j = 0 .. base_len + n_new - 1.  A cached key and, among causal new tokens, a
// new key sits at position j; a new key of a packed draft tree sits at the position its token was given.  A query at
// position p sees a key at position s (that causality or the tree lets it see) iff s >= first_visible(p) or s < keep_first.
#pragma once
#include "rd_common.cuh"

namespace rd_win {

typedef rd_attention_desc Args;

// First position that a sliding window of `window` positions ending at p, or p's own chunk of `window` positions, holds.
__host__ __device__ __forceinline__ int first_visible(int kind, int window, int p) {
  return kind == RD_MASK_CHUNK ? p / window * window : p - window + 1;
}

// Softmax of one query finished with its sink: m, l = running maximum (log2 units) and sum of 2^(score - m); returns what
// the accumulated values are multiplied by.
__device__ __forceinline__ float finish_softmax(float m, float l, const float* sink, int h) {
  if (!(l > 0.f)) return 0.f;
  if (sink == nullptr) return 1.0f / l;
  const float s = sink[h] * 1.4426950408889634f;
  const float top = fmaxf(m, s), f = exp2f(m - top);
  return f / (l * f + exp2f(s - top));
}

__device__ __forceinline__ float sigmoid_exact(float z) { return 1.0f / (1.0f + expf(-z)); }

// One query of one row.
struct Query {
  int p;        // position
  int base, n_new, i;
  int kv_end;   // keys j >= kv_end are never visible
  int first;    // first visible position past the kept ones
  int lo;       // keys keep_first <= j < lo are never visible
  const uint32_t* mask;   // tree mode
  const int32_t* new_pos;  // tree mode: positions of the row's new tokens

  __device__ __forceinline__ void init(const Args& a, int base_, int rs, int n_new_, int i_) {
    base = base_;
    n_new = n_new_;
    i = i_;
    if (a.mode == RD_ATTN_TREE) {
      mask = a.tree_mask + (int64_t)(rs + i) * a.mask_words;
      new_pos = a.tok_pos + rs;
      p = new_pos[i];
      kv_end = base + n_new;
      first = first_visible(a.mask_kind, a.window, p);
      lo = min(first, base);
    } else {
      mask = nullptr;
      new_pos = nullptr;
      p = base + i;
      kv_end = p + 1;
      first = first_visible(a.mask_kind, a.window, p);
      lo = first;
    }
    if (lo < a.keep_first) lo = a.keep_first;
  }
  __device__ __forceinline__ bool sees(const Args& a, int j) const {
    if (j >= kv_end) return false;
    int s = j;
    if (mask != nullptr && j >= base) {
      const int jn = j - base;
      if (!((mask[jn >> 5] >> (jn & 31)) & 1u)) return false;
      s = new_pos[jn];
    }
    return s >= first || s < a.keep_first;
  }
};

// This row's first key and value under key/value head g, and the shared last features of its first key.
template <typename T>
struct RowKeys {
  const T *k, *v, *tail;
  __device__ __forceinline__ void init(const Args& a, int b, int g) {
    const int64_t begin = a.kv_begin[b];
    k = (const T*)a.k + b * a.k_batch + g * a.k_head + begin * a.k_row;
    v = (const T*)a.v + b * a.v_batch + g * a.v_head + begin * a.v_row;
    tail = a.tail_dim > 0 ? (const T*)a.k_tail + b * a.tail_batch + begin * a.tail_row : nullptr;
  }
};

}  // namespace rd_win
