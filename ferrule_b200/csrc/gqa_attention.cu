// Grouped-query attention inside position-aligned chunks or sliding windows (gqa_mask.cuh), over paged keys and values.
//
// Query head h reads key / value head h / (H / G).  A cache row holds [G][maps][dim_pad] keys | [G][vdim_pad] values (heads
// padded to multiples of 8, padding is zero).
//
//   fb_gqa_prep       everything between the projection and the attention in one launch: query and key RMS norm over the
//                     whole projection, rotation of the leading dimensions (halves paired), value norm per head, mixing
//                     with the first mixing layer's values of the token (read from that layer's cache row), cache append
//   fb_value_mix      outputs of every head on the values of every kv head -> outputs whose softmax weights are mixed across heads
//   fb_gqa_attention  attention in 32-bit arithmetic, one CTA per (query row, head): models that run in fp32, and head sizes
//                     the tensor-core kernels do not take.  Query rows as wide as the keys they meet (all kv heads' keys
//                     when scores are mixed across heads), distance bias, soft cap, mean rows of the blocks before the window,
//                     values of all kv heads for every query row, difference of two maps, output gate
#include "act_type.cuh"
#include "common.cuh"
#include "ferrule_b200.h"
#include "gqa_mask.cuh"
#include "launch.cuh"

namespace fb {

template <typename T>
struct GqaParams {
  T* q;
  long long ldq;
  const T* k;
  const T* v;
  long long ldkv;
  const float* q_norm;
  const float* k_norm;
  const float* cos_t;
  const float* sin_t;
  int max_pos, half;
  const int* positions;
  const long long* write_slot;
  T* pool;
  long long pool_rows, pool_ld;
  const T* first_pool;
  long long first_off;
  float v_mix;
  const int* block_table;
  const int* row_seq;
  const int* row_pos;
  int num_seqs, max_blocks, page_size;
  KeySpan span;
  int maps, key_width, key_stride, v_offset, value_width, value_stride, value_slice;
  float softcap;
  PooledRows<T> pooled;
  const float* slopes;
  const T* gate;
  long long ldg;
  float diff_lambda, diff_scale;
  float scale, eps;
  T* out;
  long long ldo;
  int rows, heads, kv_heads, dim, dim_pad, vdim, vdim_pad;
  DeviceStatus* status;
};

// normalised rows of `heads` heads in shared memory -> rotated, into `dst` (8 elements per step)
template <typename T>
__device__ __forceinline__ void rotate_store(const float* row, int heads, const GqaParams<T>& p, const float* cs,
                                             const float* sn, T* dst) {
  const int vecs = p.dim_pad / 8;
  for (int i = threadIdx.x; i < heads * vecs; i += blockDim.x) {
    const int d0 = (i % vecs) * 8;
    const float* h = row + (i / vecs) * p.dim_pad;
    float o[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const int d = d0 + j;
      if (d < p.half) o[j] = h[d] * cs[d] - h[d + p.half] * sn[d];
      else if (d < 2 * p.half) o[j] = h[d] * cs[d - p.half] + h[d - p.half] * sn[d - p.half];
      else o[j] = h[d];
    }
    act_store8(dst + static_cast<long long>(i) * 8, o);
  }
}

template <typename T>
__global__ void __launch_bounds__(256)
gqa_prep_kernel(const GqaParams<T> p) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ float sm[];
  __shared__ float red[2][32];
  const int nq = p.heads * p.dim_pad, nk = p.kv_heads * p.dim_pad;
  float* sq = sm;
  float* sk = sq + nq;
  float* cs = sk + nk;
  float* sn = cs + p.half;
  const long long r = blockIdx.x;
  int pos = p.positions[r];
  if (pos < 0 || pos >= p.max_pos) {
    if (threadIdx.x == 0) report_status(p.status, kStatusBadIndex, 0xD60, r, pos);
    pos = 0;
  }
  const long long slot = p.write_slot[r];
  const bool keep = slot >= 0 && slot < p.pool_rows;
  if (!keep && slot != -1 && threadIdx.x == 0) report_status(p.status, kStatusBadIndex, 0xD61, r, static_cast<uint32_t>(slot));
  float ssq = 0.f, ssk = 0.f;
  for (int i = threadIdx.x * 8; i < nq; i += blockDim.x * 8) {
    float v[8];
    act_load8(p.q + r * p.ldq + i, v);
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      ssq = fmaf(v[j], v[j], ssq);
      sq[i + j] = v[j];
    }
  }
  for (int i = threadIdx.x * 8; i < nk; i += blockDim.x * 8) {
    float v[8];
    act_load8(p.k + r * p.ldkv + i, v);
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      ssk = fmaf(v[j], v[j], ssk);
      sk[i + j] = v[j];
    }
  }
  for (int i = threadIdx.x; i < p.half; i += blockDim.x) {
    cs[i] = p.cos_t[static_cast<long long>(pos) * p.half + i];
    sn[i] = p.sin_t[static_cast<long long>(pos) * p.half + i];
  }
  ssq = cta_sum(ssq, red[0]);
  ssk = cta_sum(ssk, red[1]);
  const float iq = 1.f / sqrtf(ssq / (p.heads * p.dim) + p.eps), ik = 1.f / sqrtf(ssk / (p.kv_heads * p.dim) + p.eps);
  for (int i = threadIdx.x; i < nq; i += blockDim.x) sq[i] *= iq * p.q_norm[i];
  for (int i = threadIdx.x; i < nk; i += blockDim.x) sk[i] *= ik * p.k_norm[i];
  __syncthreads();
  rotate_store(sq, p.heads, p, cs, sn, p.q + r * p.ldq);
  if (!keep) return;
  T* row = p.pool + slot * p.pool_ld;
  rotate_store(sk, p.kv_heads, p, cs, sn, row);
  // values: one warp per head
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  for (int g = warp; g < p.kv_heads; g += nw) {
    const T* v = p.v + r * p.ldkv + g * p.vdim_pad;
    float ss = 0.f;
    for (int d = lane; d < p.vdim; d += 32) {
      const float x = act_load(v + d);
      ss = fmaf(x, x, ss);
    }
    const float inv = 1.f / sqrtf(warp_sum(ss) / p.vdim + p.eps);
    T* dst = row + nk + g * p.vdim_pad;
    const T* first = p.first_pool ? p.first_pool + slot * p.pool_ld + p.first_off + g * p.vdim_pad : nullptr;
    for (int d = lane; d < p.vdim_pad; d += 32) {
      float x = d < p.vdim ? act_load(v + d) * inv : 0.f;
      if (first) x = fmaf(p.v_mix, act_load(first + d), (1.f - p.v_mix) * x);
      act_store(dst + d, x);
    }
  }
}

// The same with everything in registers, for rotations whose half is a multiple of 8: an item is a pair of 8-element vectors
// that turn together, or one vector of the part that is not rotated.  NI items per thread.
template <typename T, int NI>
__global__ void __launch_bounds__(256)
gqa_prep_vec_kernel(const GqaParams<T> p) {
  pdl_launch_dependents();
  const int pairs = p.half / 8, per_head = pairs + (p.dim_pad - 2 * p.half) / 8;
  const int q_items = p.heads * per_head, items = q_items + p.kv_heads * per_head;
  const int nk = p.kv_heads * p.dim_pad;
  __shared__ float red[2][32];
  pdl_wait();
  const long long r = blockIdx.x;
  int pos = p.positions[r];
  const long long slot = p.write_slot[r];
  float u[NI][8], w[NI][8], ssq = 0.f, ssk = 0.f;
  int off[NI];                                                       // first element of the item in its matrix row
#pragma unroll
  for (int k = 0; k < NI; ++k) {
    const int i = threadIdx.x + k * 256;
#pragma unroll
    for (int j = 0; j < 8; ++j) u[k][j] = w[k][j] = 0.f;
    off[k] = -1;
    if (i >= items) continue;
    const bool is_q = i < q_items;
    const int n = is_q ? i : i - q_items, v = n % per_head;
    off[k] = n / per_head * p.dim_pad + (v < pairs ? v * 8 : 2 * p.half + (v - pairs) * 8);
    const T* src = is_q ? p.q + r * p.ldq : p.k + r * p.ldkv;
    act_load8(src + off[k], u[k]);
    if (v < pairs) act_load8(src + off[k] + p.half, w[k]);
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < 8; ++j) ss = fmaf(u[k][j], u[k][j], fmaf(w[k][j], w[k][j], ss));
    (is_q ? ssq : ssk) += ss;
  }
  if (pos < 0 || pos >= p.max_pos) {
    if (threadIdx.x == 0) report_status(p.status, kStatusBadIndex, 0xD60, r, pos);
    pos = 0;
  }
  const bool keep = slot >= 0 && slot < p.pool_rows;
  if (!keep && slot != -1 && threadIdx.x == 0) report_status(p.status, kStatusBadIndex, 0xD61, r, static_cast<uint32_t>(slot));
  T* row = p.pool + (keep ? slot : 0) * p.pool_ld;
  // values: one warp per head, independent of the row sums
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (keep) {
    for (int g = warp; g < p.kv_heads; g += 8) {
      const T* v = p.v + r * p.ldkv + g * p.vdim_pad;
      const T* first = p.first_pool ? p.first_pool + slot * p.pool_ld + p.first_off + g * p.vdim_pad : nullptr;
      float ss = 0.f, x[8], f[8];
      if (p.vdim_pad <= 256) {
        const int d = lane * 8;
        const bool in = d < p.vdim_pad;
#pragma unroll
        for (int j = 0; j < 8; ++j) x[j] = f[j] = 0.f;
        if (in) act_load8(v + d, x);
        if (in && first) act_load8(first + d, f);
#pragma unroll
        for (int j = 0; j < 8; ++j) ss = fmaf(x[j], x[j], ss);
        const float inv = 1.f / sqrtf(warp_sum(ss) / p.vdim + p.eps), own = first ? 1.f - p.v_mix : 1.f;
#pragma unroll
        for (int j = 0; j < 8; ++j) x[j] = fmaf(p.v_mix, f[j], own * (x[j] * inv));
        if (in) act_store8(row + nk + g * p.vdim_pad + d, x);
      } else {
        for (int d = lane * 8; d < p.vdim_pad; d += 256) {
          act_load8(v + d, x);
#pragma unroll
          for (int j = 0; j < 8; ++j) ss = fmaf(x[j], x[j], ss);
        }
        const float inv = 1.f / sqrtf(warp_sum(ss) / p.vdim + p.eps), own = first ? 1.f - p.v_mix : 1.f;
        for (int d = lane * 8; d < p.vdim_pad; d += 256) {
          act_load8(v + d, x);
#pragma unroll
          for (int j = 0; j < 8; ++j) f[j] = 0.f;
          if (first) act_load8(first + d, f);
#pragma unroll
          for (int j = 0; j < 8; ++j) x[j] = fmaf(p.v_mix, f[j], own * (x[j] * inv));
          act_store8(row + nk + g * p.vdim_pad + d, x);
        }
      }
    }
  }
  ssq = cta_sum(ssq, red[0]);
  ssk = cta_sum(ssk, red[1]);
  const float iq = 1.f / sqrtf(ssq / (p.heads * p.dim) + p.eps), ik = 1.f / sqrtf(ssk / (p.kv_heads * p.dim) + p.eps);
#pragma unroll
  for (int k = 0; k < NI; ++k) {
    if (off[k] < 0) continue;
    const int i = threadIdx.x + k * 256;
    const bool is_q = i < q_items;
    if (!is_q && !keep) continue;
    const int v = (is_q ? i : i - q_items) % per_head;
    const float inv = is_q ? iq : ik;
    const float* nw = (is_q ? p.q_norm : p.k_norm) + off[k];
    T* dst = (is_q ? p.q + r * p.ldq : row) + off[k];
    float a[8];
    act_load8(nw, a);
#pragma unroll
    for (int j = 0; j < 8; ++j) u[k][j] *= inv * a[j];
    if (v < pairs) {
      float c[8], s[8], o[8];
      act_load8(nw + p.half, a);
      act_load8(p.cos_t + static_cast<long long>(pos) * p.half + v * 8, c);
      act_load8(p.sin_t + static_cast<long long>(pos) * p.half + v * 8, s);
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        w[k][j] *= inv * a[j];
        o[j] = fmaf(u[k][j], c[j], -w[k][j] * s[j]);
      }
      act_store8(dst, o);
#pragma unroll
      for (int j = 0; j < 8; ++j) o[j] = fmaf(w[k][j], c[j], u[k][j] * s[j]);
      act_store8(dst + p.half, o);
    } else {
      act_store8(dst, u[k]);
    }
  }
}

// CTA = (query row, head, slice of the value columns); DPL: value features per lane.  A head with two maps attends twice over the same values.
template <typename T, int DPL>
__global__ void __launch_bounds__(128)
gqa_attention_kernel(const GqaParams<T> p) {
  pdl_launch_dependents();
  pdl_wait();
  extern __shared__ float sm[];                 // [key_width] query, [maps][columns] outputs
  __shared__ float sm_m[4], sm_l[4], red[32];
  __shared__ float sm_o[4][DPL * 32];
  float* sq = sm;
  float* res = sm + p.key_width;
  const int r = blockIdx.x, h = blockIdx.y, g = h / (p.heads / p.kv_heads);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int seq = p.row_seq[r], pos = p.row_pos[r];
  int len = pos + 1;
  if (seq < 0 || seq >= p.num_seqs) {
    if (threadIdx.x == 0) report_status(p.status, kStatusBadIndex, 0xD70, r, seq);
    len = 0;
  }
  len = min(len, p.max_blocks * p.page_size);
  const int first = len > 0 ? p.span.first(pos) : 0, kept = len > 0 ? p.span.head(pos) : 0;
  const int n_keys = kept + max(len - first, 0);
  const float slope = p.slopes ? p.slopes[h] : 0.f;
  // with two maps a query row is zero outside its own half
  const int part = p.key_width / p.maps, col0 = blockIdx.z * p.value_slice, cols = min(p.value_slice, p.value_width - col0);
  const long long voff = p.v_offset + static_cast<long long>(g) * p.value_stride + col0;
  const long long mean_row = kept > 0 && p.span.pool > 0 ? p.pooled.first(seq) : -1;
  if (kept > 0 && p.span.pool > 0 && mean_row < 0 && threadIdx.x == 0) report_status(p.status, kStatusBadIndex, 0xD72, r, seq);
  for (int map = 0; map < p.maps; ++map) {
    const T* qr = p.q + r * p.ldq + (static_cast<long long>(h) * p.maps + map) * p.key_width + map * part;
    const long long koff = static_cast<long long>(g) * p.key_stride + map * part;
    __syncthreads();
    for (int d = threadIdx.x; d < part; d += blockDim.x) sq[d] = act_load(qr + d);
    __syncthreads();
    float o[DPL];
#pragma unroll
    for (int j = 0; j < DPL; ++j) o[j] = 0.f;
    float m = -INFINITY, l = 0.f;
    for (int i = warp; i < n_keys; i += 4) {
      const int t = i < kept ? i : first + i - kept;
      const T* row;
      if (i < kept && p.span.pool > 0) {
        if (mean_row < 0) continue;
        row = p.pooled.base + (mean_row + i) * p.pool_ld;
      } else {
        const int page = p.block_table[static_cast<long long>(seq) * p.max_blocks + t / p.page_size];
        const long long slot = static_cast<long long>(page) * p.page_size + t % p.page_size;
        if (page < 0 || slot >= p.pool_rows) {
          if (lane == 0) report_status(p.status, kStatusBadIndex, 0xD71, seq, t);
          continue;
        }
        row = p.pool + slot * p.pool_ld;
      }
      float s = 0.f, v[DPL];
#pragma unroll
      for (int j = 0; j < DPL; ++j) {
        const int d = lane + 32 * j;
        v[j] = d < cols ? act_load(row + voff + d) : 0.f;
      }
#pragma unroll 4
      for (int d = lane; d < part; d += 32) s = fmaf(sq[d], act_load(row + koff + d), s);
      s = warp_sum(s) * p.scale;
      if (p.softcap > 0.f) s = p.softcap * tanhf(s / p.softcap);
      s = fmaf(-slope, static_cast<float>(pos - t), s);
      if (s > m) {
        const float a = expf(m - s);
        m = s;
        l *= a;
#pragma unroll
        for (int j = 0; j < DPL; ++j) o[j] *= a;
      }
      const float w = expf(s - m);
      l += w;
#pragma unroll
      for (int j = 0; j < DPL; ++j) o[j] = fmaf(w, v[j], o[j]);
    }
    if (lane == 0) { sm_m[warp] = m; sm_l[warp] = l; }
#pragma unroll
    for (int j = 0; j < DPL; ++j) sm_o[warp][lane + 32 * j] = o[j];
    __syncthreads();
    const float M = fmaxf(fmaxf(sm_m[0], sm_m[1]), fmaxf(sm_m[2], sm_m[3]));
    float w[4], L = 0.f;
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      w[k] = sm_m[k] == -INFINITY ? 0.f : expf(sm_m[k] - M);
      L += w[k] * sm_l[k];
    }
    const float f = L > 0.f ? 1.f / L : 0.f;
    for (int d = threadIdx.x; d < cols; d += blockDim.x)
      res[map * cols + d] =
          (w[0] * sm_o[0][d] + w[1] * sm_o[1][d] + w[2] * sm_o[2][d] + w[3] * sm_o[3][d]) * f;
  }
  // every thread finishes the columns it wrote itself
  float inv = 1.f;
  if (p.maps == 2) {
    float ss = 0.f;
    for (int d = threadIdx.x; d < cols; d += blockDim.x) {
      res[d] -= p.diff_lambda * res[cols + d];
      ss = fmaf(res[d], res[d], ss);
    }
    inv = p.diff_scale / sqrtf(cta_sum(ss, red) / p.vdim + p.eps);
  }
  T* dst = p.out + r * p.ldo + static_cast<long long>(h) * p.value_width + col0;
  const T* gate = p.gate ? p.gate + r * p.ldg + static_cast<long long>(h) * p.vdim_pad + col0 : nullptr;
  for (int d = threadIdx.x; d < cols; d += blockDim.x)
    act_store(dst + d, res[d] * inv * (gate ? sigmoid_f(act_load(gate + d)) : 1.f));
}

// outputs of all heads on the values of one kv head -> mixed outputs of that kv head's own heads.  A thread takes 8 columns of a
// row and kv head, for up to kVmHeads of its heads at a time.
constexpr int kVmThreads = 256, kVmHeads = 4;

template <typename T>
__global__ void __launch_bounds__(kVmThreads)
value_mix_kernel(const T* __restrict__ o, long long ldv, const float* __restrict__ talk, T* __restrict__ out, long long ldo,
                 int rows, int heads, int kv_heads, int vp) {
  pdl_launch_dependents();
  extern __shared__ float share[];               // [heads of the output][heads]
  const int per = heads / kv_heads, vecs = vp / 8, blocks = (per + kVmHeads - 1) / kVmHeads;
  for (int i = threadIdx.x; i < heads * heads; i += kVmThreads) share[i] = talk[i];
  __syncthreads();
  pdl_wait();
  const long long total = static_cast<long long>(rows) * kv_heads * vecs * blocks;
  for (long long i = static_cast<long long>(blockIdx.x) * kVmThreads + threadIdx.x; i < total;
       i += static_cast<long long>(gridDim.x) * kVmThreads) {
    // neighbouring threads: columns, then kv heads, then blocks of heads, then rows
    const long long t = i / vecs, u = t / kv_heads, r = u / blocks;
    const int d = static_cast<int>(i - t * vecs) * 8, c = static_cast<int>(t - u * kv_heads), j0 = static_cast<int>(u - r * blocks) * kVmHeads;
    const T* src = o + r * ldv + c * vp + d;
    float acc[kVmHeads][8] = {};
#pragma unroll 8
    for (int g = 0; g < heads; ++g) {
      float x[8];
      act_load8(src + static_cast<long long>(g) * kv_heads * vp, x);
#pragma unroll
      for (int h = 0; h < kVmHeads; ++h) {
        const float w = share[(c * per + min(j0 + h, per - 1)) * heads + g];
#pragma unroll
        for (int j = 0; j < 8; ++j) acc[h][j] = fmaf(w, x[j], acc[h][j]);
      }
    }
#pragma unroll
    for (int h = 0; h < kVmHeads; ++h)
      if (j0 + h < per) act_store8(out + r * ldo + static_cast<long long>(c * per + j0 + h) * vp + d, acc[h]);
  }
}

template <typename T>
static int launch_value_mix(const void* o, long long ldv, const float* talk, void* out, long long ldo, int rows, int heads,
                            int kv_heads, int vp, cudaStream_t s) {
  const size_t smem = static_cast<size_t>(heads) * heads * sizeof(float);
  if (smem > 200 * 1024) return FB_ERR_LIMIT;
  static bool attr = false;
  if (!attr) {
    if (cudaFuncSetAttribute(value_mix_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024) != cudaSuccess)
      return FB_ERR_LAUNCH;
    attr = true;
  }
  const int blocks = (heads / kv_heads + kVmHeads - 1) / kVmHeads;
  const long long total = static_cast<long long>(rows) * kv_heads * (vp / 8) * blocks, ctas = (total + kVmThreads - 1) / kVmThreads;
  launch_pdl(value_mix_kernel<T>, dim3(static_cast<unsigned>(ctas < 148 * 16 ? ctas : 148 * 16)), dim3(kVmThreads), smem, s,
             static_cast<const T*>(o), ldv, talk, static_cast<T*>(out), ldo, rows, heads, kv_heads, vp);
  return cudaGetLastError() == cudaSuccess ? FB_OK : FB_ERR_LAUNCH;
}

template <typename T>
static void fill_gqa(const FbGqaArgs* a, GqaParams<T>& p) {
  p.q = static_cast<T*>(a->q); p.ldq = a->ldq;
  p.k = static_cast<const T*>(a->k); p.v = static_cast<const T*>(a->v); p.ldkv = a->ldkv;
  p.q_norm = a->q_norm; p.k_norm = a->k_norm; p.cos_t = a->cos_t; p.sin_t = a->sin_t;
  p.max_pos = a->max_pos; p.half = a->rot_dims / 2;
  p.positions = a->positions; p.write_slot = a->write_slot;
  p.pool = static_cast<T*>(a->pool); p.pool_rows = a->pool_rows; p.pool_ld = a->pool_ld;
  p.first_pool = static_cast<const T*>(a->first_pool); p.first_off = a->first_off; p.v_mix = a->v_mix;
  p.block_table = a->block_table; p.row_seq = a->row_seq; p.row_pos = a->row_pos;
  p.num_seqs = a->num_seqs; p.max_blocks = a->max_blocks; p.page_size = a->page_size;
  p.span = key_span(a);
  p.pooled = pooled_rows<T>(a);
  p.value_width = a->value_width; p.value_stride = a->value_stride; p.softcap = a->softcap;
  p.maps = a->maps; p.key_width = a->key_width; p.key_stride = a->key_stride; p.v_offset = a->v_offset;
  p.slopes = a->slopes; p.gate = static_cast<const T*>(a->gate); p.ldg = a->ldg;
  p.diff_lambda = a->diff_lambda; p.diff_scale = a->diff_scale;
  p.scale = a->scale; p.eps = a->eps;
  p.out = static_cast<T*>(a->out); p.ldo = a->ldo;
  p.rows = a->rows; p.heads = a->heads; p.kv_heads = a->kv_heads;
  p.dim = a->dim; p.dim_pad = a->dim_pad; p.vdim = a->vdim; p.vdim_pad = a->vdim_pad;
  p.status = static_cast<DeviceStatus*>(a->status);
}

static bool gqa_sizes_ok(const FbGqaArgs* a) {
  return a && a->q && a->pool && a->rows > 0 && a->heads > 0 && a->heads <= 65535 && a->kv_heads > 0 &&
         a->heads % a->kv_heads == 0 && a->dim > 0 && a->vdim > 0 && a->dim_pad >= a->dim && a->vdim_pad >= a->vdim &&
         a->dim_pad % 8 == 0 && a->vdim_pad % 8 == 0 && a->pool_rows > 0 && a->pool_ld % 8 == 0 &&
         a->ldq % 8 == 0;
}

template <typename T>
static int run_prep(const FbGqaArgs* a, cudaStream_t s) {
  GqaParams<T> p{};
  fill_gqa(a, p);
  const int per_head = p.half / 8 + (p.dim_pad - 2 * p.half) / 8, items = (p.heads + p.kv_heads) * per_head;
  const uintptr_t bits = reinterpret_cast<uintptr_t>(a->v) | reinterpret_cast<uintptr_t>(a->first_pool);
  if (p.half % 8 == 0 && items <= 1024 && (bits & 15) == 0 && a->first_off % 8 == 0) {
    const dim3 grid(a->rows), block(256);
    if (items <= 256) launch_pdl(gqa_prep_vec_kernel<T, 1>, grid, block, 0, s, p);
    else if (items <= 512) launch_pdl(gqa_prep_vec_kernel<T, 2>, grid, block, 0, s, p);
    else launch_pdl(gqa_prep_vec_kernel<T, 4>, grid, block, 0, s, p);
    return cudaGetLastError() == cudaSuccess ? FB_OK : FB_ERR_LAUNCH;
  }
  const size_t smem = (static_cast<size_t>(a->heads + a->kv_heads) * a->dim_pad + a->rot_dims) * sizeof(float);
  if (smem > 200 * 1024) return FB_ERR_LIMIT;
  static bool attr = false;
  if (!attr) {
    if (cudaFuncSetAttribute(gqa_prep_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024) != cudaSuccess)
      return FB_ERR_LAUNCH;
    attr = true;
  }
  launch_pdl(gqa_prep_kernel<T>, dim3(a->rows), dim3(256), smem, s, p);
  return cudaGetLastError() == cudaSuccess ? FB_OK : FB_ERR_LAUNCH;
}

template <typename T, int DPL>
static int launch_attention(GqaParams<T>& p, cudaStream_t s) {
  p.value_slice = min(p.value_width, DPL * 32);
  const int slices = (p.value_width + p.value_slice - 1) / p.value_slice;
  if (slices > 1 && p.maps != 1) return FB_ERR_LIMIT;
  const size_t smem = (static_cast<size_t>(p.key_width) + p.maps * p.value_slice) * sizeof(float);
  if (smem > 200 * 1024) return FB_ERR_LIMIT;
  static bool attr = false;
  if (!attr) {
    if (cudaFuncSetAttribute(gqa_attention_kernel<T, DPL>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024) != cudaSuccess)
      return FB_ERR_LAUNCH;
    attr = true;
  }
  launch_pdl(gqa_attention_kernel<T, DPL>, dim3(p.rows, p.heads, slices), dim3(128), smem, s, p);
  return cudaGetLastError() == cudaSuccess ? FB_OK : FB_ERR_LAUNCH;
}

template <typename T>
static int run_attention(const FbGqaArgs* a, cudaStream_t s) {
  GqaParams<T> p{};
  fill_gqa(a, p);
  const int d = (a->value_width + 31) / 32;
  if (d <= 2) return launch_attention<T, 2>(p, s);
  if (d <= 4) return launch_attention<T, 4>(p, s);
  if (d <= 8) return launch_attention<T, 8>(p, s);
  return launch_attention<T, 16>(p, s);
}

}  // namespace fb

using namespace fb;

extern "C" int fb_gqa_prep(const FbGqaArgs* a, void* stream) {
  if (!gqa_sizes_ok(a) || !a->k || !a->v || !a->q_norm || !a->k_norm || !a->positions || !a->write_slot || a->max_pos <= 0 ||
      a->pool_ld < static_cast<long long>(a->kv_heads) * (a->dim_pad + a->vdim_pad) ||
      a->ldq < static_cast<long long>(a->heads) * a->dim_pad || a->rot_dims < 0 || a->rot_dims % 2 || a->rot_dims > a->dim || (a->rot_dims && (!a->cos_t || !a->sin_t)))
    return FB_ERR_SHAPE;
  if (a->ldkv % 8 || a->first_off < 0 || a->first_off + static_cast<long long>(a->kv_heads) * a->vdim_pad > a->pool_ld)
    return FB_ERR_SHAPE;
  const uintptr_t bits = reinterpret_cast<uintptr_t>(a->q) | reinterpret_cast<uintptr_t>(a->k) |
                         reinterpret_cast<uintptr_t>(a->pool);
  if (bits & 15) return FB_ERR_ALIGN;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  return a->fp32 ? run_prep<float>(a, s) : run_prep<__nv_bfloat16>(a, s);
}

extern "C" int fb_gqa_attention(const FbGqaArgs* a, void* stream) {
  if (!gqa_sizes_ok(a) || !a->out || !a->block_table || !a->row_seq || !a->row_pos || a->num_seqs <= 0 || a->max_blocks <= 0 ||
      a->page_size <= 0 || !gqa_form_ok(a) || a->talk || a->value_width > 16384)
    return FB_ERR_SHAPE;
  if (a->maps == 2 && a->vdim > 512) return FB_ERR_LIMIT;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  return a->fp32 ? run_attention<float>(a, s) : run_attention<__nv_bfloat16>(a, s);
}

extern "C" int fb_value_mix(const void* o, long long ldv, const float* talk, void* out, long long ldo, int rows, int heads,
                            int kv_heads, int vdim_pad, int fp32, void* stream) {
  if (!o || !talk || !out || rows <= 0 || heads <= 0 || kv_heads <= 0 || heads % kv_heads || kv_heads > 65535 || vdim_pad <= 0 ||
      vdim_pad % 8 || ldv < static_cast<long long>(heads) * kv_heads * vdim_pad || ldo < static_cast<long long>(heads) * vdim_pad)
    return FB_ERR_SHAPE;
  if ((reinterpret_cast<uintptr_t>(o) & 15) || (reinterpret_cast<uintptr_t>(out) & 15) || ldv % 8 || ldo % 8) return FB_ERR_ALIGN;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  return fp32 ? launch_value_mix<float>(o, ldv, talk, out, ldo, rows, heads, kv_heads, vdim_pad, s)
              : launch_value_mix<__nv_bfloat16>(o, ldv, talk, out, ldo, rows, heads, kv_heads, vdim_pad, s);
}
