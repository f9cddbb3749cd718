// Row operators of layer-list models (per-layer mixers beside a feed-forward, 32-bit residual stream): embedding with
// the first norm, the layer tail (gated residual additions of both sublayers, expert reduction, next norm), latent
// cache append, logit soft cap, and the attention over a latent cache in full 32 bits.
//
// The residual stream is fp32 [rows, ldx]; activations are bf16 or fp32 (`T`).  Row pitches are padded to a multiple
// of 8 elements and the padding columns hold zeros, so any model width takes the 16-byte path.
#include "act_type.cuh"
#include "common.cuh"
#include "ferrule_b200.h"
#include "launch.cuh"

namespace fb {

// ---------------------------------------------------------------------------------
// x[r] = table[ids[r]] (fp32), h[r] = RMSNorm(x[r]) * g.  norm_stride 0: g is one number for all coordinates
// ---------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(256)
embed_norm_kernel(const int* __restrict__ ids, const T* __restrict__ table, long long ldt, int vocab,
                  float* __restrict__ x, long long ldx, const float* __restrict__ norm_w, int norm_stride,
                  T* __restrict__ h, long long ldh, int dim, int dim_pad, float eps, DeviceStatus* st) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float red[32];
  extern __shared__ float row[];
  const int r = blockIdx.x;
  int id = ids[r];
  if (id < 0 || id >= vocab) {
    if (threadIdx.x == 0) report_status(st, kStatusBadIndex, 0xB00, r, id);
    id = 0;
  }
  float ss = 0.f;
  for (int i = threadIdx.x * 8; i < dim_pad; i += blockDim.x * 8) {
    float v[8];
    act_load8(table + id * ldt + i, v);
    act_store8(x + r * ldx + i, v);
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      row[i + j] = v[j];
      ss += v[j] * v[j];
    }
  }
  ss = cta_sum(ss, red);
  const float inv = 1.f / sqrtf(ss / dim + eps);
  for (int i = threadIdx.x * 8; i < dim_pad; i += blockDim.x * 8) {
    float o[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) o[j] = i + j < dim ? row[i + j] * inv * norm_w[(i + j) * norm_stride] : 0.f;
    act_store8(h + r * ldh + i, o);
  }
}

// ---------------------------------------------------------------------------------
// Layer tail: x += sigmoid(gate1 + bias1) * mix + sigmoid(gate2 + bias2) * sum_s ffn[r * slots + s]  (each gate
// optional, each sublayer optional), h = RMSNorm(x) * g for whatever comes next.
// ---------------------------------------------------------------------------------
template <typename T>
struct TailParams {
  float* x;
  long long ldx;
  const T* mix;        // [rows, ldm]
  long long ldm;
  const T* gate1;      // pre-activation, bias added here
  long long ldg1;
  const float* bias1;
  const T* ffn;        // [rows * slots, ldf]: `topk` weighted expert rows of every token
  long long ldf;
  int slots, topk;
  const T* gate2;
  long long ldg2;
  const float* bias2;
  const float* norm_w;
  int norm_stride;
  T* h;
  long long ldh;
  int dim, dim_pad;
  float eps;
};

template <typename T>
__global__ void __launch_bounds__(256)
gated_residual_norm_kernel(const TailParams<T> p) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float red[32];
  extern __shared__ float row[];
  const long long r = blockIdx.x;
  float ss = 0.f;
  for (int i = threadIdx.x * 8; i < p.dim_pad; i += blockDim.x * 8) {
    float v[8], a[8], g[8];
    act_load8(p.x + r * p.ldx + i, v);
    if (p.mix) {
      act_load8(p.mix + r * p.ldm + i, a);
      if (p.gate1) {
        act_load8(p.gate1 + r * p.ldg1 + i, g);
#pragma unroll
        for (int j = 0; j < 8; ++j) a[j] *= sigmoid_f(g[j] + p.bias1[i + j]);
      }
#pragma unroll
      for (int j = 0; j < 8; ++j) v[j] += a[j];
    }
    if (p.ffn) {
      float f[8];
#pragma unroll
      for (int j = 0; j < 8; ++j) f[j] = 0.f;
      for (int s = 0; s < p.topk; ++s) {
        act_load8(p.ffn + (r * p.slots + s) * p.ldf + i, a);
#pragma unroll
        for (int j = 0; j < 8; ++j) f[j] += a[j];
      }
      if (p.gate2) {
        act_load8(p.gate2 + r * p.ldg2 + i, g);
#pragma unroll
        for (int j = 0; j < 8; ++j) f[j] *= sigmoid_f(g[j] + p.bias2[i + j]);
      }
#pragma unroll
      for (int j = 0; j < 8; ++j) v[j] += f[j];
    }
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      if (i + j >= p.dim) v[j] = 0.f;
      row[i + j] = v[j];
      ss += v[j] * v[j];
    }
    act_store8(p.x + r * p.ldx + i, v);
  }
  ss = cta_sum(ss, red);
  const float inv = 1.f / sqrtf(ss / p.dim + p.eps);
  for (int i = threadIdx.x * 8; i < p.dim_pad; i += blockDim.x * 8) {
    float o[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) o[j] = i + j < p.dim ? row[i + j] * inv * p.norm_w[(i + j) * p.norm_stride] : 0.f;
    act_store8(p.h + r * p.ldh + i, o);
  }
}

// ---------------------------------------------------------------------------------
// Latent cache append: c = RMSNorm(rows[:, :rank]) * w into the pool row of the token.  `row_dim` >= rank is the
// pool's row width (padding columns are written as zeros).  One warp per row.
// ---------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(128)
latent_append_kernel(const T* __restrict__ src, long long lds, int rank, int row_dim, const float* __restrict__ norm_w,
                     float eps, const long long* __restrict__ write_slot, T* __restrict__ pool, long long pool_rows,
                     int rows, DeviceStatus* st) {
  pdl_launch_dependents();
  pdl_wait();
  const int r = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (r >= rows) return;
  const long long slot = write_slot[r];
  if (slot < 0 || slot >= pool_rows) {
    if (slot != -1 && lane == 0) report_status(st, kStatusBadIndex, 0xB10, r, static_cast<uint32_t>(slot));
    return;
  }
  const T* s = src + r * lds;
  float ss = 0.f;
  for (int i = lane; i < rank; i += 32) {
    const float v = act_load(s + i);
    ss += v * v;
  }
  ss = warp_sum(ss);
  const float inv = 1.f / sqrtf(ss / rank + eps);
  T* d = pool + slot * row_dim;
  for (int i = lane; i < row_dim; i += 32) act_store(d + i, i < rank ? act_load(s + i) * inv * norm_w[i] : 0.f);
}

// ---------------------------------------------------------------------------------
// Latent layers with rotated parts: one CTA per token normalises the query latent in place (when the layer has one) and
// appends [normalised latent | turned key part | zeros] to the cache; neighbouring dimensions turn together.
// fb_latent_turn writes the turned query parts into the query rows of the attention, after the latent product.
// ---------------------------------------------------------------------------------
template <typename T>
struct LatentPrepParams {
  T* cq;                    // [rows, ldp]: rank_q wide, normalised in place; null: none
  const T* ckv;             // [rows, ldp]: rank, then rot
  long long ldp;
  int rank_q, rank, rot, row_dim, rot_off;
  const float* q_w;
  const float* kv_w;
  const float* cos_t;       // [max_pos, rot / 2]
  const float* sin_t;
  int max_pos;
  const int* positions;
  const long long* write_slot;
  T* pool;
  long long pool_rows;
  float eps;
  DeviceStatus* status;
};

__device__ __forceinline__ int checked_pos(int pos, int max_pos, int r, DeviceStatus* st) {
  if (pos >= 0 && pos < max_pos) return pos;
  if (threadIdx.x == 0) report_status(st, kStatusBadIndex, 0xB30, r, pos);
  return 0;
}

constexpr int kLpVecs = 2;

template <typename T, bool VEC>
__global__ void __launch_bounds__(256)
latent_prep_kernel(const LatentPrepParams<T> p) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float red[2][32];
  const long long r = blockIdx.x, slot = p.write_slot[r];
  const int pos = p.rot ? checked_pos(p.positions[r], p.max_pos, blockIdx.x, p.status) : 0;
  const bool keep = slot >= 0 && slot < p.pool_rows;
  if (!keep && slot != -1 && threadIdx.x == 0) report_status(p.status, kStatusBadIndex, 0xB31, r, static_cast<uint32_t>(slot));
  T* q = p.cq ? p.cq + r * p.ldp : nullptr;
  const T* c = p.ckv + r * p.ldp;
  T* d = p.pool + (keep ? slot : 0) * p.row_dim;
  const int half = p.rot / 2;
  float sq = 0.f, sc = 0.f;
  if constexpr (VEC) {
    // widths are multiples of 8: a thread holds up to kLpVecs vectors of the query latent and one of everything else
    float x[kLpVecs][8], y[8], o[8];
#pragma unroll
    for (int k = 0; k < kLpVecs; ++k) {
      const int i = (k * 256 + threadIdx.x) * 8;
#pragma unroll
      for (int j = 0; j < 8; ++j) x[k][j] = 0.f;
      if (q && i < p.rank_q) act_load8(q + i, x[k]);
    }
    const int i = threadIdx.x * 8;
#pragma unroll
    for (int j = 0; j < 8; ++j) y[j] = 0.f;
    if (i < p.rank + p.rot) act_load8(c + i, y);
#pragma unroll
    for (int k = 0; k < kLpVecs; ++k)
#pragma unroll
      for (int j = 0; j < 8; ++j) sq = fmaf(x[k][j], x[k][j], sq);
    if (i < p.rank)
#pragma unroll
      for (int j = 0; j < 8; ++j) sc = fmaf(y[j], y[j], sc);
    sq = cta_sum(sq, red[0]);
    sc = cta_sum(sc, red[1]);
    const float fq = q ? 1.f / sqrtf(sq / p.rank_q + p.eps) : 0.f, fc = 1.f / sqrtf(sc / p.rank + p.eps);
#pragma unroll
    for (int k = 0; k < kLpVecs; ++k) {
      const int e = (k * 256 + threadIdx.x) * 8;
      if (!q || e >= p.rank_q) continue;
      act_load8(p.q_w + e, o);
#pragma unroll
      for (int j = 0; j < 8; ++j) o[j] *= x[k][j] * fq;
      act_store8(q + e, o);
    }
    if (!keep) return;
    if (i < p.rank) {
      act_load8(p.kv_w + i, o);
#pragma unroll
      for (int j = 0; j < 8; ++j) o[j] *= y[j] * fc;
      act_store8(d + i, o);
    } else if (i < p.rank + p.rot) {
      const long long t = static_cast<long long>(pos) * half + (i - p.rank) / 2;
#pragma unroll
      for (int j = 0; j < 8; j += 2) {
        const float cs = p.cos_t[t + j / 2], sn = p.sin_t[t + j / 2];
        o[j] = y[j] * cs - y[j + 1] * sn;
        o[j + 1] = y[j + 1] * cs + y[j] * sn;
      }
      act_store8(d + p.rot_off + i - p.rank, o);
    }
    // padding columns
#pragma unroll
    for (int j = 0; j < 8; ++j) o[j] = 0.f;
    const int gap = p.rot_off - p.rank, end = p.rot_off + p.rot;
    if (p.rot && i < gap) act_store8(d + p.rank + i, o);
    if (end + i < p.row_dim) act_store8(d + end + i, o);
    return;
  }
  if (q)
    for (int i = threadIdx.x; i < p.rank_q; i += blockDim.x) {
      const float v = act_load(q + i);
      sq = fmaf(v, v, sq);
    }
  for (int i = threadIdx.x; i < p.rank; i += blockDim.x) {
    const float v = act_load(c + i);
    sc = fmaf(v, v, sc);
  }
  sq = cta_sum(sq, red[0]);
  sc = cta_sum(sc, red[1]);
  if (q) {
    const float f = 1.f / sqrtf(sq / p.rank_q + p.eps);
    for (int i = threadIdx.x; i < p.rank_q; i += blockDim.x) act_store(q + i, act_load(q + i) * f * p.q_w[i]);
  }
  if (!keep) return;
  const float f = 1.f / sqrtf(sc / p.rank + p.eps);
  for (int i = threadIdx.x; i < p.row_dim; i += blockDim.x) {
    const int e = i - p.rot_off;
    if (i < p.rank) {
      act_store(d + i, act_load(c + i) * f * p.kv_w[i]);
    } else if (e >= 0 && e < p.rot) {
      const float cs = p.cos_t[static_cast<long long>(pos) * half + e / 2], sn = p.sin_t[static_cast<long long>(pos) * half + e / 2];
      const float own = act_load(c + p.rank + e), other = act_load(c + p.rank + (e ^ 1));
      act_store(d + i, e & 1 ? own * cs + other * sn : own * cs - other * sn);
    } else {
      act_store(d + i, 0.f);
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(256)
latent_turn_kernel(const T* __restrict__ src, long long lds, int heads, int rot, const float* __restrict__ cos_t,
                   const float* __restrict__ sin_t, int max_pos, const int* __restrict__ positions, T* __restrict__ q,
                   long long ldq, int row_dim, int rot_off, DeviceStatus* st) {
  pdl_launch_dependents();
  pdl_wait();
  const long long r = blockIdx.x;
  const int pos = checked_pos(positions[r], max_pos, blockIdx.x, st), half = rot / 2;
  for (int i = threadIdx.x; i < heads * half; i += blockDim.x) {
    const int h = i / half, e = i - h * half;
    const float cs = cos_t[static_cast<long long>(pos) * half + e], sn = sin_t[static_cast<long long>(pos) * half + e];
    const float u = act_load(src + r * lds + h * rot + 2 * e), v = act_load(src + r * lds + h * rot + 2 * e + 1);
    T* d = q + r * ldq + static_cast<long long>(h) * row_dim + rot_off + 2 * e;
    act_store(d, u * cs - v * sn);
    act_store(d + 1, v * cs + u * sn);
  }
}

// logits <- cap * tanh(logits / cap)
__global__ void __launch_bounds__(256)
softcap_kernel(float* __restrict__ logits, long long ldl, int vocab, float cap) {
  pdl_launch_dependents();
  pdl_wait();
  float* l = logits + blockIdx.y * ldl;
  for (int i = blockIdx.x * blockDim.x + threadIdx.x; i < vocab; i += gridDim.x * blockDim.x)
    l[i] = cap * tanhf(l[i] / cap);
}

// state_in <- state_out, state_out <- the next of the slot's `buffers` buffers (decode steps that run back to back on
// the device, without the host between them)
__global__ void state_rotate_kernel(int* state_in, int* state_out, int n, int buffers) {
  pdl_launch_dependents();
  pdl_wait();
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= n) return;
  const int o = state_out[i];
  if (o < 0) return;
  state_in[i] = o;
  state_out[i] = o / buffers * buffers + (o % buffers + 1) % buffers;
}

// ---------------------------------------------------------------------------------
// Attention over a latent cache with 32-bit arithmetic throughout: one CTA per (query row, head), four warps walk the
// visible tokens in turn, one online softmax per warp, merged at the end.  DPL = latent features per lane.  Serves
// models that run in fp32, and bf16 latents wider than the tensor-core kernels take.
// ---------------------------------------------------------------------------------
template <typename T>
struct LatentParams {
  const T* q;               // [rows, heads, dl]
  long long ldq;
  const T* kv;              // [pool_rows, dl]
  long long pool_rows;
  const int* block_table;
  int max_blocks, page_size, num_seqs;
  const int* row_seq;
  const int* row_pos;
  int heads, dl, window;
  float scale;
  const T* gate;            // optional [rows, ldg]: output of head h is multiplied by sigmoid(gate[row][h])
  long long ldg;
  T* out;                   // [rows, heads, dl]
  long long ldo;
  DeviceStatus* status;
};

template <typename T, int DPL>
__global__ void __launch_bounds__(128)
latent_attention_kernel(const LatentParams<T> p) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float sm_m[4], sm_l[4];
  __shared__ float sm_o[4][DPL * 32];
  const int r = blockIdx.x, h = blockIdx.y;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int seq = p.row_seq[r];
  int len = p.row_pos[r] + 1;
  if (seq < 0 || seq >= p.num_seqs) {
    if (threadIdx.x == 0) report_status(p.status, kStatusBadIndex, 0xB20, r, seq);
    len = 0;
  }
  len = min(len, p.max_blocks * p.page_size);
  float q[DPL], o[DPL];
#pragma unroll
  for (int j = 0; j < DPL; ++j) {
    const int d = lane + 32 * j;
    q[j] = d < p.dl ? act_load(p.q + r * p.ldq + static_cast<long long>(h) * p.dl + d) : 0.f;
    o[j] = 0.f;
  }
  float m = -INFINITY, l = 0.f;
  const int first = p.window > 0 && len > p.window ? len - p.window : 0;
  for (int t = first + warp; t < len; t += 4) {
    const int page = p.block_table[static_cast<long long>(seq) * p.max_blocks + t / p.page_size];
    const long long slot = static_cast<long long>(page) * p.page_size + t % p.page_size;
    if (page < 0 || slot >= p.pool_rows) {
      if (lane == 0) report_status(p.status, kStatusBadIndex, 0xB21, seq, t);
      continue;
    }
    const T* c = p.kv + slot * p.dl;
    float v[DPL], s = 0.f;
#pragma unroll
    for (int j = 0; j < DPL; ++j) {
      const int d = lane + 32 * j;
      v[j] = d < p.dl ? act_load(c + d) : 0.f;
      s = fmaf(q[j], v[j], s);
    }
    s = warp_sum(s) * p.scale;
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
  float f = L > 0.f ? 1.f / L : 0.f;
  if (p.gate) f *= sigmoid_f(act_load(p.gate + r * p.ldg + h));
  for (int d = threadIdx.x; d < p.dl; d += blockDim.x)
    act_store(p.out + r * p.ldo + static_cast<long long>(h) * p.dl + d,
              (w[0] * sm_o[0][d] + w[1] * sm_o[1][d] + w[2] * sm_o[2][d] + w[3] * sm_o[3][d]) * f);
}

}  // namespace fb

using namespace fb;

static int ok_launch() { return cudaGetLastError() == cudaSuccess ? FB_OK : FB_ERR_LAUNCH; }
static bool aligned16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }
constexpr int kMaxRowDim = 12160;      // one fp32 row plus the reduction words in 48 KB of shared memory

template <typename T>
static int launch_embed_norm(const int* ids, const void* table, long long ldt, int vocab, float* x, long long ldx,
                             const float* norm_w, int norm_stride, void* h, long long ldh, int rows, int dim,
                             int dim_pad, float eps, void* status, cudaStream_t s) {
  launch_pdl(embed_norm_kernel<T>, dim3(rows), dim3(256), dim_pad * sizeof(float), s, ids,
             static_cast<const T*>(table), ldt, vocab, x, ldx, norm_w, norm_stride, static_cast<T*>(h), ldh, dim, dim_pad,
             eps, static_cast<DeviceStatus*>(status));
  return ok_launch();
}

extern "C" int fb_embed_norm(const int* ids, const void* table, long long ldt, int vocab, float* x, long long ldx,
                             const float* norm_w, int norm_stride, void* h, long long ldh, int rows, int dim,
                             int dim_pad, float eps, int fp32, void* status, void* stream) {
  if (!ids || !table || !x || !norm_w || !h || rows <= 0 || dim <= 0 || dim_pad < dim || dim_pad % 8 || dim_pad > kMaxRowDim)
    return FB_ERR_SHAPE;
  if (ldt < dim_pad || ldx < dim_pad || ldh < dim_pad || vocab <= 0) return FB_ERR_SHAPE;
  if (ldt % 8 || ldx % 8 || ldh % 8 || !aligned16(table) || !aligned16(x) || !aligned16(h)) return FB_ERR_ALIGN;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  return fp32 ? launch_embed_norm<float>(ids, table, ldt, vocab, x, ldx, norm_w, norm_stride, h, ldh, rows, dim, dim_pad,
                                         eps, status, s)
              : launch_embed_norm<__nv_bfloat16>(ids, table, ldt, vocab, x, ldx, norm_w, norm_stride, h, ldh, rows, dim,
                                                 dim_pad, eps, status, s);
}

template <typename T>
static int launch_tail(const FbLayerTailArgs* a, cudaStream_t s) {
  TailParams<T> p{};
  p.x = a->x; p.ldx = a->ldx;
  p.mix = static_cast<const T*>(a->mix); p.ldm = a->ldm;
  p.gate1 = static_cast<const T*>(a->gate1); p.ldg1 = a->ldg1; p.bias1 = a->bias1;
  p.ffn = static_cast<const T*>(a->ffn); p.ldf = a->ldf; p.slots = a->slots; p.topk = a->topk;
  p.gate2 = static_cast<const T*>(a->gate2); p.ldg2 = a->ldg2; p.bias2 = a->bias2;
  p.norm_w = a->norm_w; p.norm_stride = a->norm_stride;
  p.h = static_cast<T*>(a->h); p.ldh = a->ldh;
  p.dim = a->dim; p.dim_pad = a->dim_pad; p.eps = a->eps;
  launch_pdl(gated_residual_norm_kernel<T>, dim3(a->rows), dim3(256), a->dim_pad * sizeof(float), s, p);
  return ok_launch();
}

extern "C" int fb_gated_residual_norm(const FbLayerTailArgs* a, void* stream) {
  if (!a || !a->x || !a->h || !a->norm_w || a->rows <= 0 || a->dim <= 0 || a->dim_pad < a->dim || a->dim_pad % 8 ||
      a->dim_pad > kMaxRowDim)
    return FB_ERR_SHAPE;
  if (a->ldx < a->dim_pad || a->ldh < a->dim_pad || a->ldx % 8 || a->ldh % 8) return FB_ERR_SHAPE;
  if ((a->mix && (a->ldm < a->dim_pad || a->ldm % 8)) || (a->ffn && (a->ldf < a->dim_pad || a->ldf % 8 || a->slots < a->topk)))
    return FB_ERR_SHAPE;
  if ((a->gate1 && (!a->bias1 || a->ldg1 < a->dim_pad || a->ldg1 % 8)) ||
      (a->gate2 && (!a->bias2 || a->ldg2 < a->dim_pad || a->ldg2 % 8)))
    return FB_ERR_SHAPE;
  if (!aligned16(a->x) || !aligned16(a->h) || !aligned16(a->mix) || !aligned16(a->ffn) || !aligned16(a->gate1) ||
      !aligned16(a->gate2))
    return FB_ERR_ALIGN;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  return a->fp32 ? launch_tail<float>(a, s) : launch_tail<__nv_bfloat16>(a, s);
}

extern "C" int fb_latent_append(const void* src, long long lds, int rank, int row_dim, const float* norm_w, float eps,
                                const long long* write_slot, void* pool, long long pool_rows, int rows, int fp32,
                                void* status, void* stream) {
  if (!src || !norm_w || !write_slot || !pool || rank <= 0 || row_dim < rank || rows <= 0 || pool_rows <= 0)
    return FB_ERR_SHAPE;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  DeviceStatus* st = static_cast<DeviceStatus*>(status);
  const dim3 grid((rows + 3) / 4);
  if (fp32)
    launch_pdl(latent_append_kernel<float>, grid, dim3(128), 0, s, static_cast<const float*>(src), lds, rank, row_dim,
               norm_w, eps, write_slot, static_cast<float*>(pool), pool_rows, rows, st);
  else
    launch_pdl(latent_append_kernel<__nv_bfloat16>, grid, dim3(128), 0, s, static_cast<const __nv_bfloat16*>(src), lds,
               rank, row_dim, norm_w, eps, write_slot, static_cast<__nv_bfloat16*>(pool), pool_rows, rows, st);
  return ok_launch();
}

template <typename T>
static int launch_latent_prep(const FbLatentPrepArgs* a, cudaStream_t s) {
  LatentPrepParams<T> p{static_cast<T*>(a->cq), static_cast<const T*>(a->ckv), a->ldp, a->rank_q, a->rank, a->rot, a->row_dim,
                        a->rot_off, a->q_w, a->kv_w, a->cos_t, a->sin_t, a->max_pos, a->positions, a->write_slot,
                        static_cast<T*>(a->pool), a->pool_rows, a->eps, static_cast<DeviceStatus*>(a->status)};
  const bool vec = a->rank % 8 == 0 && a->rot % 8 == 0 && a->rot_off % 8 == 0 && a->row_dim % 8 == 0 && a->ldp % 8 == 0 &&
                   a->rank + a->rot <= 2048 && a->row_dim <= 2048 &&
                   (!a->cq || (a->rank_q % 8 == 0 && a->rank_q <= kLpVecs * 2048)) && aligned16(a->cq) && aligned16(a->ckv) &&
                   aligned16(a->q_w) && aligned16(a->kv_w) && aligned16(a->pool);
  if (vec) launch_pdl(latent_prep_kernel<T, true>, dim3(a->rows), dim3(256), 0, s, p);
  else launch_pdl(latent_prep_kernel<T, false>, dim3(a->rows), dim3(256), 0, s, p);
  return ok_launch();
}

extern "C" int fb_latent_prep(const FbLatentPrepArgs* a, void* stream) {
  if (!a || !a->ckv || !a->kv_w || !a->write_slot || !a->pool || a->rows <= 0 || a->rank <= 0 || a->rot < 0 || a->rot % 2 ||
      a->row_dim < a->rank || (a->cq && (a->rank_q <= 0 || !a->q_w)) || a->pool_rows <= 0 ||
      (a->rot && (a->rot_off < a->rank || a->rot_off + a->rot > a->row_dim || !a->cos_t || !a->sin_t || !a->positions || a->max_pos <= 0)))
    return FB_ERR_SHAPE;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  return a->fp32 ? launch_latent_prep<float>(a, s) : launch_latent_prep<__nv_bfloat16>(a, s);
}

extern "C" int fb_latent_turn(const void* src, long long lds, int heads, int rot, const float* cos_t, const float* sin_t, int max_pos,
                              const int* positions, void* q, long long ldq, int row_dim, int rot_off, int rows, int fp32,
                              void* status, void* stream) {
  if (!src || !cos_t || !sin_t || !positions || !q || rows <= 0 || heads <= 0 || rot <= 0 || rot % 2 || max_pos <= 0 ||
      rot_off < 0 || rot_off + rot > row_dim || ldq < static_cast<long long>(heads) * row_dim || lds < static_cast<long long>(heads) * rot)
    return FB_ERR_SHAPE;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  DeviceStatus* st = static_cast<DeviceStatus*>(status);
  if (fp32)
    launch_pdl(latent_turn_kernel<float>, dim3(rows), dim3(256), 0, s, static_cast<const float*>(src), lds, heads, rot, cos_t, sin_t,
               max_pos, positions, static_cast<float*>(q), ldq, row_dim, rot_off, st);
  else
    launch_pdl(latent_turn_kernel<__nv_bfloat16>, dim3(rows), dim3(256), 0, s, static_cast<const __nv_bfloat16*>(src), lds, heads,
               rot, cos_t, sin_t, max_pos, positions, static_cast<__nv_bfloat16*>(q), ldq, row_dim, rot_off, st);
  return ok_launch();
}

extern "C" int fb_softcap(float* logits, long long ldl, int rows, int vocab, float cap, void* stream) {
  if (!logits || rows <= 0 || rows > 65535 || vocab <= 0 || !(cap > 0.f)) return FB_ERR_SHAPE;
  int bx = (vocab + 1023) / 1024;
  launch_pdl(softcap_kernel, dim3(bx, rows), dim3(256), 0, static_cast<cudaStream_t>(stream), logits, ldl, vocab, cap);
  return ok_launch();
}

extern "C" int fb_state_rotate(int* state_in, int* state_out, int n, int buffers, void* stream) {
  if (!state_in || !state_out || n <= 0 || buffers < 2) return FB_ERR_SHAPE;
  launch_pdl(state_rotate_kernel, dim3((n + 127) / 128), dim3(128), 0, static_cast<cudaStream_t>(stream), state_in,
             state_out, n, buffers);
  return ok_launch();
}

template <typename T>
static int launch_latent(const FbAttnArgs* a, cudaStream_t s) {
  LatentParams<T> p{};
  p.q = static_cast<const T*>(a->q); p.ldq = a->ldq;
  p.kv = static_cast<const T*>(a->kv); p.pool_rows = a->pool_rows;
  p.block_table = a->block_table; p.max_blocks = a->max_blocks; p.page_size = a->page_size; p.num_seqs = a->num_seqs;
  p.row_seq = a->row_seq; p.row_pos = a->row_pos;
  p.heads = a->heads; p.dl = a->kv_lora; p.window = a->window; p.scale = a->softmax_scale;
  p.gate = static_cast<const T*>(a->gate); p.ldg = a->ldg;
  p.out = static_cast<T*>(a->out); p.ldo = a->ldo;
  p.status = static_cast<DeviceStatus*>(a->status);
  const dim3 grid(a->rows, a->heads);
  const int dpl = (a->kv_lora + 31) / 32;
  if (dpl <= 2) launch_pdl(latent_attention_kernel<T, 2>, grid, dim3(128), 0, s, p);
  else if (dpl <= 4) launch_pdl(latent_attention_kernel<T, 4>, grid, dim3(128), 0, s, p);
  else if (dpl <= 8) launch_pdl(latent_attention_kernel<T, 8>, grid, dim3(128), 0, s, p);
  else if (dpl <= 16) launch_pdl(latent_attention_kernel<T, 16>, grid, dim3(128), 0, s, p);
  else launch_pdl(latent_attention_kernel<T, 32>, grid, dim3(128), 0, s, p);
  return ok_launch();
}

extern "C" int fb_latent_attention(const FbAttnArgs* a, int fp32, void* stream) {
  if (!a || !a->q || !a->kv || !a->out || !a->block_table || !a->row_seq || !a->row_pos) return FB_ERR_SHAPE;
  if (a->rows <= 0 || a->heads <= 0 || a->heads > 65535 || a->kv_lora <= 0 || a->kv_lora > 1024 || a->rope_dim != 0 || a->window < 0 ||
      a->page_size <= 0 || a->max_blocks <= 0 || a->num_seqs <= 0 || a->pool_rows <= 0 || (a->gate && a->ldg < a->heads))
    return FB_ERR_SHAPE;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  return fp32 ? launch_latent<float>(a, s) : launch_latent<__nv_bfloat16>(a, s);
}
