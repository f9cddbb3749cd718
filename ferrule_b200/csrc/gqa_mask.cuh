// Which cached tokens a query sees: its position-aligned chunk, or a sliding window with the first tokens of the sequence or with
// the blocks before it.  The visible keys of a row are head() ones - kept tokens [0, head()), or the mean rows of the first
// head() blocks of `pool` tokens - followed by the tokens [first(), pos].
//
// Mean rows lie outside the paged pool, one after the other for every sequence slot.
#pragma once
#include "ferrule_b200.h"

namespace fb {

struct KeySpan {
  int chunk;     // > 0: chunks of this many positions
  int window;    // otherwise: the last `window` tokens
  int keep;      // and tokens below `keep`
  int pool;      // > 0: and blocks of this many tokens that lie wholly before the window
  __host__ __device__ int first(int pos) const {
    if (chunk > 0) return pos / chunk * chunk;
    return pos >= window ? pos - window + 1 : 0;
  }
  __host__ __device__ int head(int pos) const {
    const int f = first(pos);
    if (pool > 0) return f / pool;
    return keep < f ? keep : f;
  }
};

// rows of mean keys and values
template <typename T>
struct PooledRows {
  const T* base;
  long long rows;
  int stride, slot_div;
  const int* slot_of;
  // first row of a sequence, -1: it has none
  __device__ __forceinline__ long long first(int seq) const {
    const int s = slot_of[seq];
    const long long r = s >= 0 ? static_cast<long long>(s / slot_div) * stride : -1;
    return r >= 0 && r + stride <= rows ? r : -1;
  }
};

template <typename T>
inline PooledRows<T> pooled_rows(const FbGqaArgs* a) {
  return {static_cast<const T*>(a->pooled), a->pooled_rows, a->pooled_stride, a->slot_div, a->slot_of};
}
inline KeySpan key_span(const FbGqaArgs* a) { return {a->chunk, a->window, a->keep_first, a->pooled ? a->pool_tokens : 0}; }

// what the attention kernels require of the mask, the query and cache rows and the output form
inline bool gqa_form_ok(const FbGqaArgs* a) {
  const long long out_width = a->talk ? a->vdim_pad : a->value_width;
  return (a->chunk > 0 || a->window > 0) && a->keep_first >= 0 && (a->maps == 1 || a->maps == 2) && a->key_width > 0 &&
         a->key_width % 8 == 0 && a->key_width % a->maps == 0 && (a->key_stride == 0 || a->key_stride == a->key_width) &&
         a->v_offset % 8 == 0 && a->v_offset >= (a->key_stride ? static_cast<long long>(a->kv_heads) * a->key_stride : a->key_width) &&
         a->pool_ld >= a->v_offset + static_cast<long long>(a->kv_heads) * a->vdim_pad &&
         (a->value_stride == 0 ? a->value_width == static_cast<long long>(a->kv_heads) * a->vdim_pad
                               : a->value_stride == a->vdim_pad && a->value_width == a->vdim_pad) &&
         (a->value_stride != 0 || a->maps == 1) && (!a->talk || a->value_stride == 0) && a->softcap >= 0.f &&
         (!a->pooled || (a->chunk == 0 && a->keep_first == 0 && a->pool_tokens > 0 && a->pooled_stride > 0 && a->slot_div > 0 &&
                         a->slot_of && a->pooled_rows > 0 && !a->slopes)) &&
         a->ldq >= static_cast<long long>(a->heads) * a->maps * a->key_width &&
         a->ldo >= static_cast<long long>(a->heads) * out_width &&
         (!a->gate || a->ldg >= static_cast<long long>(a->heads) * a->vdim_pad);
}
// for kernels without pooled blocks, soft cap and shared values
inline bool gqa_plain_form(const FbGqaArgs* a) { return !a->pooled && a->softcap == 0.f && a->value_stride != 0; }

}  // namespace fb
