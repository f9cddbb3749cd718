// Row operators of pre-norm blocks (32-bit residual stream, one RMS norm in front of every sublayer).
//
//   fb_pre_norm_step    one kernel between two sublayers: x = table[id] * scale, or x + what the sublayer before left (projected rows,
//                       or a token's expert rows and its gated shared expert), then the next sublayer's input
//                       h = x / rms(x) * w, and with a token shift h + (h of the previous token - h) * s
//   fb_group_norm_rows  RMS norm of equal parts of activation rows (the output norm of a head-decay scan)
//
// The shift needs the row before: of the same sequence in this batch, or what the sequence's state holds (fp32, normalised,
// before its own shift).  A CTA walks kShiftRows consecutive rows and forms the row in front of them once more, so rows with
// a predecessor in the batch are read by two CTAs: such steps write the new stream to another buffer than they read.  When
// every sequence brings one row, all predecessors are in the state.  A row's result depends on its own sequence only.
#include "act_type.cuh"
#include "common.cuh"
#include "ferrule_b200.h"
#include "launch.cuh"
#include "row_norm.cuh"

namespace fb {

constexpr int kShiftRows = 4;

template <typename T>
struct PreNormParams {
  const float* x;
  float* x_out;
  long long ldx;
  const int* ids;
  const T* table;
  long long ldt;
  int vocab;
  float scale;
  const T* y;
  long long ldy;
  const T* ffn;
  long long ldf;
  int slots, topk;
  const T* shared;
  long long lds;
  const float* shared_gate;
  long long ldsg;
  const float* norm_w;
  T* act;
  long long lda;
  const float* shift;
  float* plane;
  const int* row_seq;
  const int* seq_start;
  const int* state_in;
  const int* state_out;
  int n_states, n_seqs;
  int rows, dim, dim_pad, per_cta, single;
  float eps;
  DeviceStatus* status;
};

// the stream row after the previous sublayer
template <typename T, int VPT>
__device__ __forceinline__ void stream_row(const PreNormParams<T>& p, long long r, float (&v)[VPT][8]) {
  int id = 0;
  if (p.ids) {
    id = p.ids[r];
    if (id < 0 || id >= p.vocab) {
      if (threadIdx.x == 0) report_status(p.status, kStatusBadIndex, 0xE40, r, id);
      id = 0;
    }
  }
  const float gate = p.shared ? sigmoid_f(p.shared_gate[r * p.ldsg]) : 0.f;
#pragma unroll
  for (int k = 0; k < VPT; ++k) {
    const int i = (k * blockDim.x + threadIdx.x) * 8;
#pragma unroll
    for (int j = 0; j < 8; ++j) v[k][j] = 0.f;
    if (i >= p.dim_pad) continue;
    float a[8];
    if (p.ids) {
      act_load8(p.table + id * p.ldt + i, v[k]);
#pragma unroll
      for (int j = 0; j < 8; ++j) v[k][j] *= p.scale;
    } else {
      act_load8(p.x + r * p.ldx + i, v[k]);
    }
    if (p.y) {
      act_load8(p.y + r * p.ldy + i, a);
#pragma unroll
      for (int j = 0; j < 8; ++j) v[k][j] += a[j];
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
      if (p.shared) {
        act_load8(p.shared + r * p.lds + i, a);
#pragma unroll
        for (int j = 0; j < 8; ++j) f[j] = fmaf(gate, a[j], f[j]);
      }
#pragma unroll
      for (int j = 0; j < 8; ++j) v[k][j] += f[j];
    }
#pragma unroll
    for (int j = 0; j < 8; ++j)
      if (i + j >= p.dim) v[k][j] = 0.f;
  }
}

template <typename T, int VPT>
__global__ void __launch_bounds__(kRowThreads)
pre_norm_step_kernel(const PreNormParams<T> p) {
  pdl_launch_dependents();
  __shared__ float red[2][64];
  const GroupScratch g{nullptr, nullptr, red};
  const int r0 = blockIdx.x * p.per_cta, r1 = min(r0 + p.per_cta, p.rows);
  int turn = 0;
  float w[VPT][8], before[VPT][8], v[VPT][8], h[VPT][8];
#pragma unroll
  for (int k = 0; k < VPT; ++k) {
    const int i = (k * blockDim.x + threadIdx.x) * 8;
#pragma unroll
    for (int j = 0; j < 8; ++j) w[k][j] = before[k][j] = 0.f;
    if (p.act && i < p.dim_pad) act_load8(p.norm_w + i, w[k]);
  }
  auto normed = [&]() {
    group_norm<VPT>(v, p.dim, 1, p.eps, g, turn, h);
    turn ^= 1;
#pragma unroll
    for (int k = 0; k < VPT; ++k)
#pragma unroll
      for (int j = 0; j < 8; ++j) h[k][j] *= w[k][j];
  };
  pdl_wait();
  for (int r = r0; r < r1; ++r) {
    int seq = 0, first = r, last = r, sin = -1, sout = -1;
    if (p.shift) {
      seq = p.single ? r : p.row_seq[r];
      bool ok = seq >= 0 && seq < p.n_seqs;
      if (ok) {
        first = p.seq_start[seq];
        last = p.seq_start[seq + 1] - 1;
        sin = p.state_in[seq];
        sout = p.state_out[seq];
        ok = first >= 0 && first <= r && r <= last && last < p.rows && sin < p.n_states && sout < p.n_states &&
             !(sin >= 0 && sin == sout) && (!p.single || first == last);
      }
      if (!ok) {
        if (threadIdx.x == 0) report_status(p.status, kStatusBadIndex, 0xE41, r, seq);
        first = last = r;
        sin = sout = -1;
      }
      if (first == r) {
#pragma unroll
        for (int k = 0; k < VPT; ++k) {
          const int i = (k * blockDim.x + threadIdx.x) * 8;
#pragma unroll
          for (int j = 0; j < 8; ++j) before[k][j] = 0.f;
          if (sin >= 0 && i < p.dim_pad) act_load8(p.plane + static_cast<long long>(sin) * p.dim_pad + i, before[k]);
        }
      } else if (r == r0) {
        stream_row<T, VPT>(p, r - 1, v);
        normed();
#pragma unroll
        for (int k = 0; k < VPT; ++k)
#pragma unroll
          for (int j = 0; j < 8; ++j) before[k][j] = h[k][j];
      }
    }
    stream_row<T, VPT>(p, r, v);
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
      const int i = (k * blockDim.x + threadIdx.x) * 8;
      if (i < p.dim_pad) act_store8(p.x_out + r * p.ldx + i, v[k]);
    }
    if (!p.act) continue;
    normed();
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
      const int i = (k * blockDim.x + threadIdx.x) * 8;
      if (i >= p.dim_pad) continue;
      if (!p.shift) {
        act_store8(p.act + r * p.lda + i, h[k]);
        continue;
      }
      float s[8], o[8];
      act_load8(p.shift + i, s);
#pragma unroll
      for (int j = 0; j < 8; ++j) o[j] = fmaf(before[k][j] - h[k][j], s[j], h[k][j]);
      act_store8(p.act + r * p.lda + i, o);
      if (r == last && sout >= 0) act_store8(p.plane + static_cast<long long>(sout) * p.dim_pad + i, h[k]);
#pragma unroll
      for (int j = 0; j < 8; ++j) before[k][j] = h[k][j];
    }
  }
}

template <typename T, int VPT>
__global__ void __launch_bounds__(kRowThreads)
group_norm_rows_kernel(const T* __restrict__ x, long long ldx, const float* __restrict__ w_in, T* __restrict__ out, long long ldo,
                       int dim, int dim_pad, int groups, int n_sums, float eps) {
  pdl_launch_dependents();
  extern __shared__ float group_sm[];
  __shared__ float red[2][64];
  const GroupScratch g{group_sm, group_sm + n_sums, red};
  const long long r = blockIdx.x;
  pdl_wait();
  float v[VPT][8];
#pragma unroll
  for (int k = 0; k < VPT; ++k) {
    const int i = (k * blockDim.x + threadIdx.x) * 8;
#pragma unroll
    for (int j = 0; j < 8; ++j) v[k][j] = 0.f;
    if (i < dim_pad) act_load8(x + r * ldx + i, v[k]);
#pragma unroll
    for (int j = 0; j < 8; ++j)
      if (i + j >= dim) v[k][j] = 0.f;
  }
  group_norm<VPT>(v, dim, groups, eps, g, 0, v);
#pragma unroll
  for (int k = 0; k < VPT; ++k) {
    const int i = (k * blockDim.x + threadIdx.x) * 8;
    if (i >= dim_pad) continue;
    float w[8];
    act_load8(w_in + i, w);
#pragma unroll
    for (int j = 0; j < 8; ++j) v[k][j] *= w[j];
    act_store8(out + r * ldo + i, v[k]);
  }
}

}  // namespace fb

using namespace fb;

static int ok_launch() { return cudaGetLastError() == cudaSuccess ? FB_OK : FB_ERR_LAUNCH; }
static bool aligned16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

template <typename T>
static int launch_pre_norm(const FbPreNormArgs* a, cudaStream_t s) {
  PreNormParams<T> p{};
  p.x = a->x; p.x_out = a->x_out; p.ldx = a->ldx;
  p.ids = a->ids; p.table = static_cast<const T*>(a->table); p.ldt = a->ldt; p.vocab = a->vocab; p.scale = a->scale;
  p.y = static_cast<const T*>(a->y); p.ldy = a->ldy;
  p.ffn = static_cast<const T*>(a->ffn); p.ldf = a->ldf; p.slots = a->slots; p.topk = a->topk;
  p.shared = static_cast<const T*>(a->shared); p.lds = a->lds; p.shared_gate = a->shared_gate; p.ldsg = a->ldsg;
  p.norm_w = a->norm_w; p.act = static_cast<T*>(a->act); p.lda = a->lda;
  p.shift = a->shift; p.plane = a->plane; p.row_seq = a->row_seq; p.seq_start = a->seq_start;
  p.state_in = a->state_in; p.state_out = a->state_out; p.n_states = a->n_states; p.n_seqs = a->n_seqs;
  p.rows = a->rows; p.dim = a->dim; p.dim_pad = a->dim_pad; p.eps = a->eps;
  p.single = a->n_seqs == a->rows;
  p.per_cta = a->shift && !p.single ? kShiftRows : 1;
  p.status = static_cast<DeviceStatus*>(a->status);
  const dim3 grid((a->rows + p.per_cta - 1) / p.per_cta), block(row_threads(a->dim_pad));
  switch (row_vpt(a->dim_pad)) {
    case 1: launch_pdl(pre_norm_step_kernel<T, 1>, grid, block, 0, s, p); break;
    case 2: launch_pdl(pre_norm_step_kernel<T, 2>, grid, block, 0, s, p); break;
    case 4: launch_pdl(pre_norm_step_kernel<T, 4>, grid, block, 0, s, p); break;
    case 8: launch_pdl(pre_norm_step_kernel<T, 8>, grid, block, 0, s, p); break;
    default: return FB_ERR_LIMIT;
  }
  return ok_launch();
}

extern "C" int fb_pre_norm_step(const FbPreNormArgs* a, void* stream) {
  if (!a || !a->x_out || (!a->x && !a->ids) || a->rows <= 0 || a->dim <= 0 || a->dim_pad < a->dim || a->dim_pad % 8 ||
      a->ldx < a->dim_pad || a->ldx % 8)
    return FB_ERR_SHAPE;
  if (a->ids && (!a->table || a->ldt < a->dim_pad || a->ldt % 8 || a->vocab <= 0)) return FB_ERR_SHAPE;
  if ((a->y && (a->ldy < a->dim_pad || a->ldy % 8)) || (a->act && (!a->norm_w || a->lda < a->dim_pad || a->lda % 8)))
    return FB_ERR_SHAPE;
  if ((a->ffn && (a->ldf < a->dim_pad || a->ldf % 8 || a->slots < a->topk || a->topk <= 0)) ||
      (a->shared && (!a->ffn || !a->shared_gate || a->lds < a->dim_pad || a->lds % 8)))
    return FB_ERR_SHAPE;
  if (a->shift && (!a->act || !a->plane || !a->row_seq || !a->seq_start || !a->state_in || !a->state_out || a->n_states <= 0 ||
                   a->n_seqs <= 0 || a->n_seqs > a->rows || (a->n_seqs != a->rows && !a->ids && a->x == a->x_out)))
    return FB_ERR_SHAPE;
  if (!aligned16(a->x) || !aligned16(a->x_out) || !aligned16(a->table) || !aligned16(a->y) || !aligned16(a->ffn) ||
      !aligned16(a->shared) || !aligned16(a->norm_w) || !aligned16(a->act) || !aligned16(a->shift) || !aligned16(a->plane))
    return FB_ERR_ALIGN;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  return a->fp32 ? launch_pre_norm<float>(a, s) : launch_pre_norm<__nv_bfloat16>(a, s);
}

template <typename T, int VPT>
static int launch_group_rows(const void* x, long long ldx, const float* w, void* out, long long ldo, int rows, int dim, int dim_pad,
                             int groups, float eps, cudaStream_t s) {
  const int n_sums = group_sums(dim, groups);
  const size_t smem = (static_cast<size_t>(n_sums) + groups) * sizeof(float);
  if (smem > 200 * 1024) return FB_ERR_LIMIT;
  static bool attr = false;
  if (!attr) {
    if (cudaFuncSetAttribute(group_norm_rows_kernel<T, VPT>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024) != cudaSuccess)
      return FB_ERR_LAUNCH;
    attr = true;
  }
  launch_pdl(group_norm_rows_kernel<T, VPT>, dim3(rows), dim3(row_threads(dim_pad)), smem, s, static_cast<const T*>(x), ldx, w,
             static_cast<T*>(out), ldo, dim, dim_pad, groups, n_sums, eps);
  return ok_launch();
}

template <typename T>
static int run_group_rows(const void* x, long long ldx, const float* w, void* out, long long ldo, int rows, int dim, int dim_pad,
                          int groups, float eps, cudaStream_t s) {
  switch (row_vpt(dim_pad)) {
    case 1: return launch_group_rows<T, 1>(x, ldx, w, out, ldo, rows, dim, dim_pad, groups, eps, s);
    case 2: return launch_group_rows<T, 2>(x, ldx, w, out, ldo, rows, dim, dim_pad, groups, eps, s);
    case 4: return launch_group_rows<T, 4>(x, ldx, w, out, ldo, rows, dim, dim_pad, groups, eps, s);
    case 8: return launch_group_rows<T, 8>(x, ldx, w, out, ldo, rows, dim, dim_pad, groups, eps, s);
    default: return FB_ERR_LIMIT;
  }
}

extern "C" int fb_group_norm_rows(const void* x, long long ldx, const float* norm_w, void* out, long long ldo, int rows, int dim,
                                  int dim_pad, int groups, float eps, int fp32, void* stream) {
  if (!x || !norm_w || !out || rows <= 0 || dim <= 0 || dim_pad < dim || dim_pad % 8 || ldx < dim_pad || ldo < dim_pad ||
      groups <= 0 || dim % groups)
    return FB_ERR_SHAPE;
  if (ldx % 8 || ldo % 8 || !aligned16(x) || !aligned16(norm_w) || !aligned16(out)) return FB_ERR_ALIGN;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  return fp32 ? run_group_rows<float>(x, ldx, norm_w, out, ldo, rows, dim, dim_pad, groups, eps, s)
              : run_group_rows<__nv_bfloat16>(x, ldx, norm_w, out, ldo, rows, dim, dim_pad, groups, eps, s);
}
