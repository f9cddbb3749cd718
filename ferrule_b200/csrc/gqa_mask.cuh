// Which cached tokens a query sees: its position-aligned chunk, or a sliding window and the first tokens of the sequence.
// The visible tokens of a row are kept ones [0, head()) followed by [first(), pos].
#pragma once
#include "ferrule_b200.h"

namespace fb {

struct KeySpan {
  int chunk;     // > 0: chunks of this many positions
  int window;    // otherwise: the last `window` tokens
  int keep;      // and tokens below `keep`
  __host__ __device__ int first(int pos) const {
    if (chunk > 0) return pos / chunk * chunk;
    return pos >= window ? pos - window + 1 : 0;
  }
  __host__ __device__ int head(int pos) const {
    const int f = first(pos);
    return keep < f ? keep : f;
  }
};

// what the attention kernels require of the mask, the query and cache rows and the output form
inline bool gqa_form_ok(const FbGqaArgs* a) {
  return (a->chunk > 0 || a->window > 0) && a->keep_first >= 0 && (a->maps == 1 || a->maps == 2) && a->key_width > 0 &&
         a->key_width % 8 == 0 && a->key_width % a->maps == 0 && (a->key_stride == 0 || a->key_stride == a->key_width) &&
         a->v_offset % 8 == 0 && a->v_offset >= (a->key_stride ? static_cast<long long>(a->kv_heads) * a->key_stride : a->key_width) &&
         a->pool_ld >= a->v_offset + static_cast<long long>(a->kv_heads) * a->vdim_pad &&
         a->ldq >= static_cast<long long>(a->heads) * a->maps * a->key_width &&
         a->ldo >= static_cast<long long>(a->heads) * a->vdim_pad &&
         (!a->gate || a->ldg >= static_cast<long long>(a->heads) * a->vdim_pad);
}

}  // namespace fb
