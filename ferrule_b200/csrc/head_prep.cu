// Everything between the input projection and window attention in one launch: biases, rotation, query and key RMS norm per head,
// the factors of the scores, mixing of scores across heads, cache append; in decode steps also the mean rows of the blocks of
// tokens that this step completes (fb_pool_blocks: the same for any batch, in a launch of its own).
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
struct PoolParams {
  const T* pool;
  long long pool_rows, pool_ld;
  T* pooled;
  long long pooled_rows;
  const int* positions;
  const int* row_seq;
  const int* block_table;
  const int* slot_of;
  int rows, width, num_seqs, max_blocks, page_size, pool_tokens, pooled_stride, slot_div;
  DeviceStatus* status;
};

constexpr int kPoolBatch = 8;

// the mean cache row of the block that ends with batch row r, if one does: eight columns per thread
template <typename T>
__device__ __forceinline__ void pool_block(const PoolParams<T>& p, int r) {
  const int pos = p.positions[r], P = p.pool_tokens;
  if (pos < 0 || (pos + 1) % P) return;
  const int seq = p.row_seq[r], b = pos / P;
  const int slot = seq >= 0 && seq < p.num_seqs ? p.slot_of[seq] : -1;
  if (slot < 0) return;                                          // a row of no sequence
  const long long dst = static_cast<long long>(slot / p.slot_div) * p.pooled_stride + b;
  if (b >= p.pooled_stride || dst >= p.pooled_rows || pos >= p.max_blocks * p.page_size) {
    if (threadIdx.x == 0) report_status(p.status, kStatusBadIndex, 0xE30, r, pos);
    return;
  }
  const int* pages = p.block_table + static_cast<long long>(seq) * p.max_blocks;
  const int t0 = pos + 1 - P;
  for (int c = threadIdx.x * 8; c < p.width; c += blockDim.x * 8) {
    float sum[8] = {};
    for (int k = 0; k < P; k += kPoolBatch) {
      // the rows of a batch are requested together (past the block's end: its last row again, not counted)
      Raw8<T> raw[kPoolBatch];
      bool ok[kPoolBatch];
#pragma unroll
      for (int e = 0; e < kPoolBatch; ++e) {
        const int t = min(t0 + k + e, pos), page = pages[t / p.page_size];
        const long long row = static_cast<long long>(page) * p.page_size + t % p.page_size;
        ok[e] = page >= 0 && row < p.pool_rows;
        raw[e].load_written(p.pool + (ok[e] ? row : 0) * p.pool_ld + c);
      }
#pragma unroll
      for (int e = 0; e < kPoolBatch; ++e) {
        if (!ok[e]) report_status(p.status, kStatusBadIndex, 0xE31, seq, t0 + k + e);
        const float w = ok[e] && k + e < P ? 1.f : 0.f;
        float x[8];
        raw[e].get(x);
#pragma unroll
        for (int j = 0; j < 8; ++j) sum[j] = fmaf(w, x[j], sum[j]);
      }
    }
#pragma unroll
    for (int j = 0; j < 8; ++j) sum[j] /= P;
    act_store8(p.pooled + dst * p.pool_ld + c, sum);
  }
}

template <typename T>
__global__ void __launch_bounds__(128)
pool_blocks_kernel(const PoolParams<T> p) {
  pdl_launch_dependents();
  pdl_wait();
  pool_block(p, blockIdx.x);
}

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
  const float* cos_t;
  const float* sin_t;
  const int* positions;
  int half, max_pos;
  PoolParams<T> blocks;
  DeviceStatus* status;
};

// eight features of a head from d0 on, rotated: feature d turns with d + half
__device__ __forceinline__ void turned8(const float* x, int d0, int half, const float* cs, const float* sn, float (&o)[8]) {
#pragma unroll
  for (int j = 0; j < 8; ++j) {
    const int d = d0 + j;
    if (d < half) o[j] = x[d] * cs[d] - x[d + half] * sn[d];
    else if (d < 2 * half) o[j] = x[d] * cs[d - half] + x[d - half] * sn[d - half];
    else o[j] = x[d];
  }
}

template <typename T, bool MIX>
__global__ void __launch_bounds__(kHpThreads)
head_prep_kernel(const HeadPrepParams<T> p) {
  pdl_launch_dependents();
  extern __shared__ __align__(16) float hp_sm[];
  const int nq = p.heads * p.maps, nk = p.kv_heads * p.maps, dp = p.dim_pad, vecs = dp / 8;
  float* sq = hp_sm;                       // [nq][dim_pad]
  float* sk = sq + nq * dp;                // [nk][dim_pad]
  float* inv = sk + nk * dp;               // [nq + nk]
  float* coef = inv + nq + nk;             // mix: [heads][heads]; else cosines and sines
  float* cs = coef;
  float* sn = cs + p.half;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, nw = kHpThreads / 32;
  if (MIX)
    for (int i = tid; i < p.heads * p.heads; i += kHpThreads) coef[i] = p.q_mix[i];
  pdl_wait();
  const long long r = blockIdx.x, slot = p.write_slot[r];
  const bool keep = slot >= 0 && slot < p.pool_rows;
  if (!keep && slot != -1 && tid == 0) report_status(p.status, kStatusBadIndex, 0xE20, r, static_cast<uint32_t>(slot));
  if (p.half) {
    int pos = p.positions[r];
    if (pos < 0 || pos >= p.max_pos) {
      if (tid == 0) report_status(p.status, kStatusBadIndex, 0xE21, r, pos);
      pos = 0;
    }
    for (int i = tid; i < p.half; i += kHpThreads) {
      cs[i] = p.cos_t[static_cast<long long>(pos) * p.half + i];
      sn[i] = p.sin_t[static_cast<long long>(pos) * p.half + i];
    }
  }
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
  auto weighted = [&](float (&x)[8], const float* norm, int d, float f) {
    float w[8];
    if (norm) act_load8(norm + d, w);
#pragma unroll
    for (int j = 0; j < 8; ++j) x[j] *= norm ? f * w[j] : f;
  };
  if (keep)
    for (int i = tid; i < nk * vecs; i += kHpThreads) {
      const int h = i / vecs, d = (i - h * vecs) * 8;
      float x[8];
      if (p.half) turned8(sk + h * dp, d, p.half, cs, sn, x);        // (turning keeps the root mean square)
      else act_load8(sk + h * dp + d, x);
      weighted(x, p.k_norm, d, inv[nq + h]);
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
        if (p.half) turned8(sq + h * dp, d, p.half, cs, sn, x);
        else act_load8(sq + h * dp + d, x);
        weighted(x, p.q_norm, d, inv[h] * p.q_mix[h / p.maps]);
      }
      act_store8(out + static_cast<long long>(i) * 8, x);
    }
    if (p.blocks.pooled && keep) {
      __syncthreads();                     // this step's own cache row is complete
      pool_block(p.blocks, static_cast<int>(r));
    }
  }
}

// The same without mixing, one map per head and rotations whose half is a multiple of 8, in registers: LPH lanes share a head, a lane
// holds a pair of 8-element vectors that turn together, or one vector of the part that is not rotated.
template <typename T, int LPH, bool BLOCKS>
__global__ void __launch_bounds__(kHpThreads)
head_turn_kernel(const HeadPrepParams<T> p) {
  pdl_launch_dependents();
  const int pairs = p.half / 8, per_head = pairs + (p.dim_pad - 2 * p.half) / 8, heads = p.heads + p.kv_heads;
  const int tid = threadIdx.x, v = tid % LPH;
  const bool pair = v < pairs;
  const int at = pair ? v * 8 : 2 * p.half + (v - pairs) * 8;                // first feature of this lane's vector
  pdl_wait();
  const long long r = blockIdx.x, slot = p.write_slot[r];
  const bool keep = slot >= 0 && slot < p.pool_rows;
  if (!keep && slot != -1 && tid == 0) report_status(p.status, kStatusBadIndex, 0xE22, r, static_cast<uint32_t>(slot));
  T* row = p.pool + (keep ? slot : 0) * p.pool_ld;
  float c[8] = {}, s[8] = {};
  if (p.half) {
    int pos = p.positions[r];
    if (pos < 0 || pos >= p.max_pos) {
      if (tid == 0) report_status(p.status, kStatusBadIndex, 0xE21, r, pos);
      pos = 0;
    }
    if (pair) {
      act_load8(p.cos_t + static_cast<long long>(pos) * p.half + at, c);
      act_load8(p.sin_t + static_cast<long long>(pos) * p.half + at, s);
    }
  }
  constexpr int kStep = kHpThreads / LPH;
  for (int h0 = 0; h0 < heads; h0 += kStep) {
    const int h = h0 + tid / LPH, hk = h - p.heads;
    const bool is_q = hk < 0, in = h < heads && v < per_head;
    const T* src = is_q ? p.q + r * p.ldp + h * p.dim_pad : p.k + r * p.ldp + hk * p.dim_pad;
    const float* bias = is_q ? p.q_bias : p.k_bias;
    const float* norm = is_q ? p.q_norm : p.k_norm;
    float u[8] = {}, w[8] = {}, b[8];
    if (in) {
      act_load8(src + at, u);
      if (pair) act_load8(src + at + p.half, w);
      if (bias) {
        bias += (is_q ? h : hk) * p.dim_pad + at;
        act_load8(bias, b);
#pragma unroll
        for (int j = 0; j < 8; ++j) u[j] += b[j];
        if (pair) {
          act_load8(bias + p.half, b);
#pragma unroll
          for (int j = 0; j < 8; ++j) w[j] += b[j];
        }
      }
    }
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < 8; ++j) ss = fmaf(u[j], u[j], fmaf(w[j], w[j], ss));
#pragma unroll
    for (int o = 1; o < LPH; o <<= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if (!in || (!is_q && !keep)) continue;
    const float f = 1.f / sqrtf(ss / p.dim + p.eps) * (is_q ? p.q_mix[h] : 1.f);
    T* dst = (is_q ? p.q_out + r * p.ldqo + h * p.dim_pad : row + hk * p.dim_pad) + at;
    float o[8], n[8];
    // the norm's weights belong to the features behind the turn
#pragma unroll
    for (int j = 0; j < 8; ++j) o[j] = (pair ? fmaf(u[j], c[j], -w[j] * s[j]) : u[j]) * f;
    if (norm) {
      act_load8(norm + at, n);
#pragma unroll
      for (int j = 0; j < 8; ++j) o[j] *= n[j];
    }
    act_store8(dst, o);
    if (!pair) continue;
#pragma unroll
    for (int j = 0; j < 8; ++j) o[j] = fmaf(w[j], c[j], u[j] * s[j]) * f;
    if (norm) {
      act_load8(norm + at + p.half, n);
#pragma unroll
      for (int j = 0; j < 8; ++j) o[j] *= n[j];
    }
    act_store8(dst + p.half, o);
  }
  if (!keep) return;
  T* vrow = row + p.kv_heads * p.dim_pad;
  for (int e = tid * 8; e < p.kv_heads * p.vdim_pad; e += kHpThreads * 8) {
    float x[8];
    act_load8(p.v + r * p.ldp + e, x);
    act_store8(vrow + e, x);
  }
  if constexpr (BLOCKS) {
    __syncthreads();                       // this step's own cache row is complete
    pool_block(p.blocks, static_cast<int>(r));
  }
}

template <typename T, int LPH>
static int launch_head_turn(const HeadPrepParams<T>& p, int rows, cudaStream_t s) {
  if (p.blocks.pooled) launch_pdl(head_turn_kernel<T, LPH, true>, dim3(rows), dim3(kHpThreads), 0, s, p);
  else launch_pdl(head_turn_kernel<T, LPH, false>, dim3(rows), dim3(kHpThreads), 0, s, p);
  return cudaGetLastError() == cudaSuccess ? FB_OK : FB_ERR_LAUNCH;
}

template <typename T>
static PoolParams<T> pool_params(const FbPoolArgs* a) {
  return {static_cast<const T*>(a->pool), a->pool_rows, a->pool_ld, static_cast<T*>(a->pooled), a->pooled_rows, a->positions,
          a->row_seq, a->block_table, a->slot_of, a->rows, a->width, a->num_seqs, a->max_blocks, a->page_size, a->pool_tokens,
          a->pooled_stride, a->slot_div, static_cast<DeviceStatus*>(a->status)};
}
static bool pool_args_ok(const FbPoolArgs* a) {
  return a->pool && a->pooled && a->positions && a->row_seq && a->block_table && a->slot_of && a->rows > 0 && a->pool_rows > 0 &&
         a->pooled_rows > 0 && a->width > 0 && a->width % 8 == 0 && a->width <= a->pool_ld && a->pool_ld % 8 == 0 &&
         a->num_seqs > 0 && a->max_blocks > 0 && a->page_size > 0 && a->pool_tokens > 0 && a->pooled_stride > 0 &&
         a->slot_div > 0 && !(reinterpret_cast<uintptr_t>(a->pool) & 15) && !(reinterpret_cast<uintptr_t>(a->pooled) & 15);
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
  p.cos_t = a->cos_t; p.sin_t = a->sin_t; p.positions = a->positions; p.half = a->half; p.max_pos = a->max_pos;
  if (a->blocks) p.blocks = pool_params<T>(a->blocks);
  const int lanes = a->half / 8 + (a->dim_pad - 2 * a->half) / 8;
  if (!MIX && a->maps == 1 && a->v && a->half % 8 == 0 && lanes <= 32) {
    if (lanes <= 4) return launch_head_turn<T, 4>(p, a->rows, s);
    if (lanes <= 8) return launch_head_turn<T, 8>(p, a->rows, s);
    if (lanes <= 16) return launch_head_turn<T, 16>(p, a->rows, s);
    return launch_head_turn<T, 32>(p, a->rows, s);
  }
  const size_t n = static_cast<size_t>(a->heads + a->kv_heads) * a->maps;
  const size_t smem = (n * a->dim_pad + n + (MIX ? static_cast<size_t>(a->heads) * a->heads : 2 * a->half)) * sizeof(float);
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
  if (!a || !a->q || !a->k || (a->mix && (!a->q_norm || !a->k_norm)) || !a->q_mix || !a->q_out || !a->write_slot || !a->pool || a->rows <= 0 ||
      a->heads <= 0 || a->kv_heads <= 0 || a->heads % a->kv_heads || (a->maps != 1 && a->maps != 2) || (a->mix && a->maps != 1) ||
      a->dim <= 0 || a->dim_pad < a->dim || a->dim_pad % 8 || a->vdim_pad <= 0 || a->vdim_pad % 8 || a->pool_rows <= 0)
    return FB_ERR_SHAPE;
  if (!a->v && (a->maps != 1 || a->vdim_pad != a->dim_pad)) return FB_ERR_SHAPE;
  if (a->half < 0 || (a->half && (a->mix || 2 * a->half > a->dim || !a->cos_t || !a->sin_t || !a->positions || a->max_pos <= 0)))
    return FB_ERR_SHAPE;
  if (a->blocks && (a->mix || !pool_args_ok(a->blocks) || a->blocks->rows != a->rows || a->blocks->fp32 != a->fp32 ||
                    a->blocks->pool != a->pool))
    return FB_ERR_SHAPE;
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

extern "C" int fb_pool_blocks(const FbPoolArgs* a, void* stream) {
  if (!a || !pool_args_ok(a)) return FB_ERR_SHAPE;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (a->fp32) launch_pdl(pool_blocks_kernel<float>, dim3(a->rows), dim3(128), 0, s, pool_params<float>(a));
  else launch_pdl(pool_blocks_kernel<__nv_bfloat16>, dim3(a->rows), dim3(128), 0, s, pool_params<__nv_bfloat16>(a));
  return cudaGetLastError() == cudaSuccess ? FB_OK : FB_ERR_LAUNCH;
}
