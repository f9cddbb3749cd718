// Everything between the input projection and window attention in one launch: biases, query and key RMS norm per head, the
// factors of the scores, mixing of scores across heads, cache append.
//
// score_h = sum_g M[h, g] q_g . k_kv(g) is linear in the queries, so heads are mixed here: row h of the output holds, side by
// side for every kv head, the sum of M[h, g] q_g over the heads g of that kv head, and meets the concatenated keys of all kv
// heads.  Without mixing a head with several maps writes one row per map, its query in the map's columns and zeros elsewhere.
//
// One CTA per token; norms, factors and sums in fp32, rounded once on the way out.
#include "act_type.cuh"
#include "common.cuh"
#include "ferrule_b200.h"
#include "launch.cuh"

namespace fb {

constexpr int kHpThreads = 256;

template <typename T>
struct HeadPrepParams {
  const T* q;
  const T* k;
  const T* v;
  long long ldp;
  const float* q_bias;
  const float* k_bias;
  const float* q_norm;
  const float* k_norm;
  const float* q_mix;
  T* q_out;
  long long ldqo;
  const long long* write_slot;
  T* pool;
  long long pool_rows, pool_ld;
  int heads, kv_heads, maps, dim, dim_pad, vdim_pad;
  float eps;
  DeviceStatus* status;
};

template <typename T, bool MIX>
__global__ void __launch_bounds__(kHpThreads)
head_prep_kernel(const HeadPrepParams<T> p) {
  pdl_launch_dependents();
  extern __shared__ __align__(16) float hp_sm[];
  const int nq = p.heads * p.maps, nk = p.kv_heads * p.maps, dp = p.dim_pad, vecs = dp / 8;
  float* sq = hp_sm;                       // [nq][dim_pad]
  float* sk = sq + nq * dp;                // [nk][dim_pad]
  float* inv = sk + nk * dp;               // [nq + nk]
  float* coef = inv + nq + nk;             // mix: [heads][heads]
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, nw = kHpThreads / 32;
  if (MIX)
    for (int i = tid; i < p.heads * p.heads; i += kHpThreads) coef[i] = p.q_mix[i];
  pdl_wait();
  const long long r = blockIdx.x, slot = p.write_slot[r];
  const bool keep = slot >= 0 && slot < p.pool_rows;
  if (!keep && slot != -1 && tid == 0) report_status(p.status, kStatusBadIndex, 0xE20, r, static_cast<uint32_t>(slot));
  T* row = p.pool + (keep ? slot : 0) * p.pool_ld;
  T* vrow = row + nk * dp;
  for (int i = tid; i < (nq + nk) * vecs; i += kHpThreads) {
    const bool is_q = i < nq * vecs;
    const int e = (is_q ? i : i - nq * vecs) * 8;
    const float* bias = is_q ? p.q_bias : p.k_bias;
    float x[8], b[8];
    act_load8((is_q ? p.q : p.k) + r * p.ldp + e, x);
    if (bias) {
      act_load8(bias + e, b);
#pragma unroll
      for (int j = 0; j < 8; ++j) x[j] += b[j];
    }
    act_store8((is_q ? sq : sk) + e, x);
    if (!is_q && !p.v && keep) act_store8(vrow + e, x);      // the values are the keys as projected
  }
  if (p.v && keep)
    for (int e = tid * 8; e < p.kv_heads * p.vdim_pad; e += kHpThreads * 8) {
      float x[8];
      act_load8(p.v + r * p.ldp + e, x);
      act_store8(vrow + e, x);
    }
  __syncthreads();
  for (int h = warp; h < nq + nk; h += nw) {
    const float* x = h < nq ? sq + h * dp : sk + (h - nq) * dp;
    float ss = 0.f;
    for (int d = lane; d < dp; d += 32) ss = fmaf(x[d], x[d], ss);
    ss = warp_sum(ss);
    if (lane == 0) inv[h] = 1.f / sqrtf(ss / p.dim + p.eps);
  }
  __syncthreads();
  if (keep)
    for (int i = tid; i < nk * vecs; i += kHpThreads) {
      const int h = i / vecs, d = (i - h * vecs) * 8;
      float x[8], w[8];
      act_load8(sk + h * dp + d, x);
      act_load8(p.k_norm + d, w);
      const float f = inv[nq + h];
#pragma unroll
      for (int j = 0; j < 8; ++j) x[j] *= f * w[j];
      act_store8(row + h * dp + d, x);
    }
  T* out = p.q_out + r * p.ldqo;
  if constexpr (MIX) {
    // an item is kHb output heads x one kv head x 8 features: every query vector is read once for all of them
    constexpr int kHb = 4;
    const int per = p.heads / p.kv_heads, gv = p.kv_heads * vecs, items = (p.heads + kHb - 1) / kHb * gv;
    for (int i = tid; i < items; i += kHpThreads) {
      const int hb = i / gv, c = i - hb * gv, kv = c / vecs, d = (c - kv * vecs) * 8, h0 = hb * kHb;
      float acc[kHb][8] = {}, w[8];
      act_load8(p.q_norm + d, w);
      for (int g = kv * per; g < kv * per + per; ++g) {
        float x[8];
        act_load8(sq + g * dp + d, x);
#pragma unroll
        for (int b = 0; b < kHb; ++b) {
          const float f = coef[min(h0 + b, p.heads - 1) * p.heads + g] * inv[g];
#pragma unroll
          for (int j = 0; j < 8; ++j) acc[b][j] = fmaf(f, x[j], acc[b][j]);
        }
      }
#pragma unroll
      for (int b = 0; b < kHb; ++b) {
        if (h0 + b >= p.heads) break;
#pragma unroll
        for (int j = 0; j < 8; ++j) acc[b][j] *= w[j];
        act_store8(out + (static_cast<long long>(h0 + b) * gv + c) * 8, acc[b]);
      }
    }
  } else {
    const int items = nq * p.maps * vecs;
    for (int i = tid; i < items; i += kHpThreads) {
      const int c = i / vecs, d = (i - c * vecs) * 8, h = c / p.maps;
      float x[8] = {};
      if (c - h * p.maps == h % p.maps) {
        float w[8];
        act_load8(sq + h * dp + d, x);
        act_load8(p.q_norm + d, w);
        const float f = inv[h] * p.q_mix[h / p.maps];
#pragma unroll
        for (int j = 0; j < 8; ++j) x[j] *= f * w[j];
      }
      act_store8(out + static_cast<long long>(i) * 8, x);
    }
  }
}

template <typename T, bool MIX>
static int run_head_prep(const FbHeadPrepArgs* a, cudaStream_t s) {
  HeadPrepParams<T> p{};
  p.q = static_cast<const T*>(a->q); p.k = static_cast<const T*>(a->k); p.v = static_cast<const T*>(a->v); p.ldp = a->ldp;
  p.q_bias = a->q_bias; p.k_bias = a->k_bias; p.q_norm = a->q_norm; p.k_norm = a->k_norm; p.q_mix = a->q_mix;
  p.q_out = static_cast<T*>(a->q_out); p.ldqo = a->ldqo;
  p.write_slot = a->write_slot; p.pool = static_cast<T*>(a->pool); p.pool_rows = a->pool_rows; p.pool_ld = a->pool_ld;
  p.heads = a->heads; p.kv_heads = a->kv_heads; p.maps = a->maps;
  p.dim = a->dim; p.dim_pad = a->dim_pad; p.vdim_pad = a->vdim_pad; p.eps = a->eps;
  p.status = static_cast<DeviceStatus*>(a->status);
  const size_t n = static_cast<size_t>(a->heads + a->kv_heads) * a->maps;
  const size_t smem = (n * a->dim_pad + n + (MIX ? static_cast<size_t>(a->heads) * a->heads : 0)) * sizeof(float);
  if (smem > 200 * 1024) return FB_ERR_LIMIT;
  static bool attr = false;
  if (!attr) {
    if (cudaFuncSetAttribute(head_prep_kernel<T, MIX>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024) != cudaSuccess)
      return FB_ERR_LAUNCH;
    attr = true;
  }
  launch_pdl(head_prep_kernel<T, MIX>, dim3(a->rows), dim3(kHpThreads), smem, s, p);
  return cudaGetLastError() == cudaSuccess ? FB_OK : FB_ERR_LAUNCH;
}

}  // namespace fb

using namespace fb;

extern "C" int fb_head_prep(const FbHeadPrepArgs* a, void* stream) {
  if (!a || !a->q || !a->k || !a->q_norm || !a->k_norm || !a->q_mix || !a->q_out || !a->write_slot || !a->pool || a->rows <= 0 ||
      a->heads <= 0 || a->kv_heads <= 0 || a->heads % a->kv_heads || (a->maps != 1 && a->maps != 2) || (a->mix && a->maps != 1) ||
      a->dim <= 0 || a->dim_pad < a->dim || a->dim_pad % 8 || a->vdim_pad <= 0 || a->vdim_pad % 8 || a->pool_rows <= 0)
    return FB_ERR_SHAPE;
  if (!a->v && (a->maps != 1 || a->vdim_pad != a->dim_pad)) return FB_ERR_SHAPE;
  const long long kw = static_cast<long long>(a->mix ? a->kv_heads : a->maps) * a->dim_pad;
  if (a->ldqo < a->heads * a->maps * kw || a->ldp < static_cast<long long>(a->heads) * a->maps * a->dim_pad ||
      a->pool_ld < static_cast<long long>(a->kv_heads) * (a->maps * a->dim_pad + a->vdim_pad))
    return FB_ERR_SHAPE;
  const uintptr_t bits = reinterpret_cast<uintptr_t>(a->q) | reinterpret_cast<uintptr_t>(a->k) | reinterpret_cast<uintptr_t>(a->v) |
                         reinterpret_cast<uintptr_t>(a->q_out) | reinterpret_cast<uintptr_t>(a->pool) |
                         reinterpret_cast<uintptr_t>(a->q_bias) | reinterpret_cast<uintptr_t>(a->k_bias) |
                         reinterpret_cast<uintptr_t>(a->q_norm) | reinterpret_cast<uintptr_t>(a->k_norm);
  if ((bits & 15) || a->ldp % 8 || a->ldqo % 8 || a->pool_ld % 8) return FB_ERR_ALIGN;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (a->fp32) return a->mix ? run_head_prep<float, true>(a, s) : run_head_prep<float, false>(a, s);
  return a->mix ? run_head_prep<__nv_bfloat16, true>(a, s) : run_head_prep<__nv_bfloat16, false>(a, s);
}
