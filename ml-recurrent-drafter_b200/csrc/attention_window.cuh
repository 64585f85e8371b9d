// What the sliding-window attention kernels share: which keys a query sees, and where to look for them.
//
// A row's keys lie in the cache slots kv_begin + j, j = 0 .. base_len + n_new - 1.  A cached key and, among
// causal new tokens, a new key sits at position j; a new key of a packed draft tree sits at the position
// its token was given.  A query at position p sees a key at position s (that causality or the tree lets it
// see) iff p - s < window or s < keep_first.
#pragma once
#include "rd_common.cuh"

namespace rd_win {

struct Args {
  const void* q;        // [m, ldq]: head h of token t at q + t * ldq + h * dim
  int64_t ldq;
  const void* k_cache;  // [B, nkv, max_len, dim]
  const void* v_cache;  // [B, nkv, max_len, vdim]
  const void* gate;     // optional [m, ld_gate]: head h's output is multiplied by sigmoid(gate[t, h])
  int64_t ld_gate;
  void* out;            // [m, nh * vdim]
  const int32_t* row_start;
  const int32_t* kv_begin;
  const int32_t* base_len;
  const int32_t* tok_pos;  // tree mode: position of every new token
  const uint32_t* tree_mask;
  int mask_words;
  int nh, nkv, dim, vdim, max_len, mode;
  float scale;
  int window, keep_first;
};

__device__ __forceinline__ float sigmoid_exact(float z) { return 1.0f / (1.0f + expf(-z)); }

// One query of one row.
struct Query {
  int p;        // position
  int base, n_new, i;
  int kv_end;   // keys j >= kv_end are never visible
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
      lo = min(p - a.window + 1, base);
    } else {
      mask = nullptr;
      new_pos = nullptr;
      p = base + i;
      kv_end = p + 1;
      lo = p - a.window + 1;
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
    return p - s < a.window || s < a.keep_first;
  }
};

}  // namespace rd_win
