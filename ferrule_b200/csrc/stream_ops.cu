// Row operators of output-norm and sandwich blocks (32-bit residual stream, a norm on every sublayer's output): embedding,
// learned positions, norms and residual addition, short causal convolutions over packed sequences.
//
//   fb_stream_step  x = table[id] + pos[p]  or  x += norm(y); also the new rows as activations, and in decode steps (one
//                   row per sequence) the next mixer's input h = x + conv(x) with the convolution state
//   fb_short_conv   the convolution over any mix of row counts; its state is the last taps - 1 inputs of a sequence
//   fb_norm_rows    norm of selected rows (the rows whose logits are wanted)
//   fb_sandwich_step, fb_sandwich_rows   the same for RMS norms of equal parts of a row, with the norm in front of the next
//                   sublayer and the embedding that a new pass over looped layers adds
//
// State of a convolution: buffer `state_in[seq]` is read (-1: a new sequence, zeros), buffer `state_out[seq]` written
// (-1: nothing is kept), never the same one.
#include "act_type.cuh"
#include "common.cuh"
#include "ferrule_b200.h"
#include "launch.cuh"
#include "row_norm.cuh"

namespace fb {

// mean and inverse deviation of a row held in registers: VPT vectors of 8, `dim` valid elements
template <int VPT>
__device__ __forceinline__ void row_moments(const float (&v)[VPT][8], int dim, int rms, float eps, float (*red)[32],
                                            float& mean, float& inv) {
  mean = 0.f;
  if (!rms) {
    float s = 0.f;
#pragma unroll
    for (int k = 0; k < VPT; ++k)
#pragma unroll
      for (int j = 0; j < 8; ++j) s += v[k][j];
    mean = cta_sum(s, red[0]) / dim;
  }
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < VPT; ++k) {
    const int i = (k * blockDim.x + threadIdx.x) * 8;
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const float d = i + j < dim ? v[k][j] - mean : 0.f;
      ss = fmaf(d, d, ss);
    }
  }
  inv = 1.f / sqrtf(cta_sum(ss, red[1]) / dim + eps);
}

template <typename T>
struct StreamParams {
  float* x;
  long long ldx;
  const int* ids;
  const int* positions;
  const T* table;
  const T* pos_table;
  long long ldt;
  int vocab, max_pos;
  const T* y;
  long long ldy;
  const float* norm_w;
  const float* norm_b;
  int rms;
  T* act;
  long long lda;
  const float* conv;
  float* tail;
  const int* state_in;
  const int* state_out;
  int taps, n_states;
  T* h;
  long long ldh;
  int dim, dim_pad;
  float eps;
  DeviceStatus* status;
};

template <typename T, int VPT>
__global__ void __launch_bounds__(kRowThreads)
stream_step_kernel(const StreamParams<T> p) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float red[2][32];
  const int r = blockIdx.x;
  float v[VPT][8];
  if (p.ids) {
    int id = p.ids[r], pos = p.pos_table ? p.positions[r] : 0;
    if (id < 0 || id >= p.vocab || (p.pos_table && (pos < 0 || pos >= p.max_pos))) {
      if (threadIdx.x == 0) report_status(p.status, kStatusBadIndex, 0xD00, r, id);
      id = pos = 0;
    }
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
      const int i = (k * blockDim.x + threadIdx.x) * 8;
      if (i >= p.dim_pad) continue;
      float e[8];
      act_load8(p.table + id * p.ldt + i, v[k]);
      if (p.pos_table) {
        act_load8(p.pos_table + pos * p.ldt + i, e);
#pragma unroll
        for (int j = 0; j < 8; ++j) v[k][j] += e[j];
      }
    }
  } else {
    float y[VPT][8], mean, inv;
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
      const int i = (k * blockDim.x + threadIdx.x) * 8;
      if (i < p.dim_pad) {
        act_load8(p.y + r * p.ldy + i, y[k]);
        act_load8(p.x + r * p.ldx + i, v[k]);
      } else {
#pragma unroll
        for (int j = 0; j < 8; ++j) y[k][j] = 0.f;
      }
    }
    row_moments<VPT>(y, p.dim, p.rms, p.eps, red, mean, inv);
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
      const int i = (k * blockDim.x + threadIdx.x) * 8;
      if (i >= p.dim_pad) continue;
      float w[8], b[8] = {};
      act_load8(p.norm_w + i, w);
      if (p.norm_b) act_load8(p.norm_b + i, b);
#pragma unroll
      for (int j = 0; j < 8; ++j) v[k][j] = i + j < p.dim ? v[k][j] + fmaf((y[k][j] - mean) * inv, w[j], b[j]) : 0.f;
    }
  }
  int sin = -1, sout = -1;
  if (p.conv) {
    sin = p.state_in[r];
    sout = p.state_out[r];
    if (sin >= p.n_states || sout >= p.n_states || (sin >= 0 && sin == sout)) {
      if (threadIdx.x == 0) report_status(p.status, kStatusBadIndex, 0xD01, r, sout);
      sin = sout = -1;
    }
  }
  const int keep = p.taps - 1;
#pragma unroll
  for (int k = 0; k < VPT; ++k) {
    const int i = (k * blockDim.x + threadIdx.x) * 8;
    if (i >= p.dim_pad) continue;
    act_store8(p.x + r * p.ldx + i, v[k]);
    if (p.act) act_store8(p.act + r * p.lda + i, v[k]);
    if (!p.conv) continue;
    float h[8], w[8], o[8];
    act_load8(p.conv + static_cast<long long>(keep) * p.dim_pad + i, w);
#pragma unroll
    for (int j = 0; j < 8; ++j) h[j] = fmaf(w[j], v[k][j], v[k][j]);
    for (int t = 0; t < keep; ++t) {
#pragma unroll
      for (int j = 0; j < 8; ++j) o[j] = 0.f;
      if (sin >= 0) {
        act_load8(p.tail + (static_cast<long long>(sin) * keep + t) * p.dim_pad + i, o);
        act_load8(p.conv + static_cast<long long>(t) * p.dim_pad + i, w);
#pragma unroll
        for (int j = 0; j < 8; ++j) h[j] = fmaf(w[j], o[j], h[j]);
      }
      if (sout >= 0 && t > 0) act_store8(p.tail + (static_cast<long long>(sout) * keep + t - 1) * p.dim_pad + i, o);
    }
    if (sout >= 0 && keep > 0) act_store8(p.tail + (static_cast<long long>(sout) * keep + keep - 1) * p.dim_pad + i, v[k]);
    act_store8(p.h + r * p.ldh + i, h);
  }
}

template <typename T, int VPT>
__global__ void __launch_bounds__(kRowThreads)
norm_rows_kernel(const float* __restrict__ x, long long ldx, int x_rows, const int* __restrict__ rows_idx,
                 const float* __restrict__ norm_w, const float* __restrict__ norm_b, int rms, T* __restrict__ out,
                 long long ldo, int dim, int dim_pad, float eps, DeviceStatus* st) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float red[2][32];
  int r = rows_idx[blockIdx.x];
  if (r < 0 || r >= x_rows) {
    if (threadIdx.x == 0) report_status(st, kStatusBadIndex, 0xD10, blockIdx.x, r);
    r = 0;
  }
  float v[VPT][8], mean, inv;
#pragma unroll
  for (int k = 0; k < VPT; ++k) {
    const int i = (k * blockDim.x + threadIdx.x) * 8;
#pragma unroll
    for (int j = 0; j < 8; ++j) v[k][j] = 0.f;
    if (i < dim_pad) act_load8(x + r * ldx + i, v[k]);
  }
  row_moments<VPT>(v, dim, rms, eps, red, mean, inv);
#pragma unroll
  for (int k = 0; k < VPT; ++k) {
    const int i = (k * blockDim.x + threadIdx.x) * 8;
    if (i >= dim_pad) continue;
    float w[8], b[8] = {}, o[8];
    act_load8(norm_w + i, w);
    if (norm_b) act_load8(norm_b + i, b);
#pragma unroll
    for (int j = 0; j < 8; ++j) o[j] = i + j < dim ? fmaf((v[k][j] - mean) * inv, w[j], b[j]) : 0.f;
    act_store8(out + blockIdx.x * ldo + i, o);
  }
}

template <typename T>
struct SandwichParams {
  float* x;
  long long ldx;
  const T* y;
  long long ldy;
  const float* y_bias;
  const float* out_w;
  const int* ids;
  const T* table;
  long long ldt;
  int vocab, fresh;
  const float* in_w;
  T* act;
  long long lda;
  int dim, dim_pad, groups, n_sums;
  float eps;
  DeviceStatus* status;
};

template <typename T, int VPT>
__global__ void __launch_bounds__(kRowThreads)
sandwich_step_kernel(const SandwichParams<T> p) {
  pdl_launch_dependents();
  extern __shared__ float group_sm[];
  __shared__ float red[2][64];
  const GroupScratch g{group_sm, group_sm + p.n_sums, red};
  const int r = blockIdx.x;
  pdl_wait();
  float v[VPT][8], y[VPT][8];
#pragma unroll
  for (int k = 0; k < VPT; ++k) {
    const int i = (k * blockDim.x + threadIdx.x) * 8;
#pragma unroll
    for (int j = 0; j < 8; ++j) v[k][j] = y[k][j] = 0.f;
    if (i >= p.dim_pad) continue;
    if (!p.fresh) act_load8(p.x + r * p.ldx + i, v[k]);
    if (p.y) act_load8(p.y + r * p.ldy + i, y[k]);
  }
  if (p.y) {
    if (p.y_bias) {
#pragma unroll
      for (int k = 0; k < VPT; ++k) {
        const int i = (k * blockDim.x + threadIdx.x) * 8;
        if (i >= p.dim_pad) continue;
        float b[8];
        act_load8(p.y_bias + i, b);
#pragma unroll
        for (int j = 0; j < 8; ++j) y[k][j] += b[j];
      }
    }
    group_norm<VPT>(y, p.dim, p.groups, p.eps, g, 0, y);
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
      const int i = (k * blockDim.x + threadIdx.x) * 8;
      if (i >= p.dim_pad) continue;
      float w[8];
      act_load8(p.out_w + i, w);
#pragma unroll
      for (int j = 0; j < 8; ++j) v[k][j] = fmaf(y[k][j], w[j], v[k][j]);
    }
  }
  if (p.ids) {
    int id = p.ids[r];
    if (id < 0 || id >= p.vocab) {
      if (threadIdx.x == 0) report_status(p.status, kStatusBadIndex, 0xD30, r, id);
      id = 0;
    }
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
      const int i = (k * blockDim.x + threadIdx.x) * 8;
      if (i >= p.dim_pad) continue;
      float e[8];
      act_load8(p.table + id * p.ldt + i, e);
#pragma unroll
      for (int j = 0; j < 8; ++j) v[k][j] += e[j];
    }
  }
  if (p.y || p.ids) {
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
      const int i = (k * blockDim.x + threadIdx.x) * 8;
      if (i < p.dim_pad) act_store8(p.x + r * p.ldx + i, v[k]);
    }
  }
  if (!p.act) return;
  group_norm<VPT>(v, p.dim, p.groups, p.eps, g, 1, v);
#pragma unroll
  for (int k = 0; k < VPT; ++k) {
    const int i = (k * blockDim.x + threadIdx.x) * 8;
    if (i >= p.dim_pad) continue;
    float w[8];
    act_load8(p.in_w + i, w);
#pragma unroll
    for (int j = 0; j < 8; ++j) v[k][j] *= w[j];
    act_store8(p.act + r * p.lda + i, v[k]);
  }
}

template <typename T, int VPT>
__global__ void __launch_bounds__(kRowThreads)
sandwich_rows_kernel(const float* __restrict__ x, long long ldx, int x_rows, const int* __restrict__ rows_idx,
                     const float* __restrict__ w_in, T* __restrict__ out, long long ldo, int dim, int dim_pad, int groups,
                     int n_sums, float eps, DeviceStatus* st) {
  pdl_launch_dependents();
  extern __shared__ float group_sm[];
  __shared__ float red[2][64];
  const GroupScratch g{group_sm, group_sm + n_sums, red};
  pdl_wait();
  int r = rows_idx[blockIdx.x];
  if (r < 0 || r >= x_rows) {
    if (threadIdx.x == 0) report_status(st, kStatusBadIndex, 0xD31, blockIdx.x, r);
    r = 0;
  }
  float v[VPT][8];
#pragma unroll
  for (int k = 0; k < VPT; ++k) {
    const int i = (k * blockDim.x + threadIdx.x) * 8;
#pragma unroll
    for (int j = 0; j < 8; ++j) v[k][j] = 0.f;
    if (i < dim_pad) act_load8(x + r * ldx + i, v[k]);
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
    act_store8(out + blockIdx.x * ldo + i, v[k]);
  }
}

// ---------------------------------------------------------------------------------
// short causal convolution
// ---------------------------------------------------------------------------------
template <typename TI, typename TO>
struct ConvParams {
  const TI* x;
  long long ldx;
  const float* w;
  const float* bias;
  TI* tail;
  TO* out;
  long long ldo;
  const int* row_seq;
  const int* seq_start;
  const int* state_in;
  const int* state_out;
  int rows, channels, taps, n_states, n_seqs;
  DeviceStatus* status;
};

template <typename T>
__device__ __forceinline__ void zero8(float (&v)[8]) {
#pragma unroll
  for (int j = 0; j < 8; ++j) v[j] = 0.f;
}

template <bool RESIDUAL, bool SILU, bool EXACT, typename TO>
__device__ __forceinline__ void conv_finish(const float (&x)[8], float (&acc)[8], TO* out) {
#pragma unroll
  for (int j = 0; j < 8; ++j) {
    if (RESIDUAL) acc[j] += x[j];
    if (SILU) acc[j] = EXACT ? acc[j] / (1.f + expf(-acc[j])) : __fdividef(acc[j], 1.f + __expf(-acc[j]));
  }
  act_store8(out, acc);
}

// The inputs the next step needs: entry j of a tail is the input `keep - j` tokens before the sequence's end.  Row i of n
// keeps its own input; row 0 also moves the entries that still come from the old tail.
template <typename TI>
__device__ __forceinline__ void conv_tail(TI* tail, int channels, int keep, int c, int i, int n, int sin, int sout,
                                          const float (&x)[8]) {
  if (sout < 0 || keep <= 0) return;
  TI* dst = tail + static_cast<long long>(sout) * keep * channels + c;
  const int j = i - (n - keep);
  if (j >= 0) act_store8(dst + static_cast<long long>(j) * channels, x);
  if (i == 0) {
    for (int q = 0; q < keep - n; ++q) {
      float o[8];
      zero8<float>(o);
      if (sin >= 0) act_load8(tail + (static_cast<long long>(sin) * keep + q + n) * channels + c, o);
      act_store8(dst + static_cast<long long>(q) * channels, o);
    }
  }
}

template <typename TI, typename TO>
__device__ __forceinline__ bool conv_row(const ConvParams<TI, TO>& p, int r, int& i, int& n, int& sin, int& sout) {
  const int seq = p.row_seq[r];
  if (seq < 0 || seq >= p.n_seqs) {
    report_status(p.status, kStatusBadIndex, 0xD20, r, seq);
    return false;
  }
  const int r0 = p.seq_start[seq];
  n = p.seq_start[seq + 1] - r0;
  i = r - r0;
  sin = p.state_in[seq];
  sout = p.state_out[seq];
  if (r0 < 0 || i < 0 || i >= n || r0 + n > p.rows || sin >= p.n_states || sout >= p.n_states || (sin >= 0 && sin == sout)) {
    report_status(p.status, kStatusBadIndex, 0xD21, r, seq);
    return false;
  }
  return true;
}

// ROWS consecutive rows x 8 channels per thread; KEEP = taps - 1 when it is at most 3 (the inputs of all rows are
// requested together), -1: any number of taps
template <typename TI, typename TO, int KEEP, int ROWS, bool RESIDUAL, bool SILU>
__global__ void __launch_bounds__(128)
short_conv_kernel(const ConvParams<TI, TO> p) {
  pdl_launch_dependents();
  const int c = (blockIdx.x * blockDim.x + threadIdx.x) * 8;
  const int rb = blockIdx.y * ROWS;
  constexpr bool kExact = sizeof(TO) == 4;
  const int keep = KEEP >= 0 ? KEEP : p.taps - 1;
  if (c >= p.channels) {
    pdl_wait();
    return;
  }
  if constexpr (KEEP >= 0) {
    float w[KEEP + 1][8], b[8];
#pragma unroll
    for (int t = 0; t <= KEEP; ++t) act_load8(p.w + static_cast<long long>(t) * p.channels + c, w[t]);
    zero8<float>(b);
    if (p.bias) act_load8(p.bias + c, b);
    pdl_wait();
    // the inputs of all rows and the row tables are requested before anything is waited for (addresses clamped)
    Raw8<TI> win[ROWS + KEEP];
#pragma unroll
    for (int t = 0; t < ROWS + KEEP; ++t) win[t].load(p.x + min(max(rb - KEEP + t, 0), p.rows - 1) * p.ldx + c);
    int i_[ROWS], n_[ROWS], in_[ROWS], out_[ROWS], seq_[ROWS];
    bool ok_[ROWS];
#pragma unroll
    for (int k = 0; k < ROWS; ++k) seq_[k] = p.row_seq[min(rb + k, p.rows - 1)];
#pragma unroll
    for (int k = 0; k < ROWS; ++k) {
      const int seq = min(max(seq_[k], 0), p.n_seqs - 1), r0 = p.seq_start[seq];
      n_[k] = p.seq_start[seq + 1] - r0;
      i_[k] = rb + k - r0;
      in_[k] = p.state_in[seq];
      out_[k] = p.state_out[seq];
      ok_[k] = rb + k < p.rows;
    }
#pragma unroll
    for (int k = 0; k < ROWS; ++k) {
      if (!ok_[k]) continue;
      const int r0 = rb + k - i_[k];
      ok_[k] = seq_[k] >= 0 && seq_[k] < p.n_seqs && r0 >= 0 && i_[k] >= 0 && i_[k] < n_[k] && r0 + n_[k] <= p.rows &&
               in_[k] < p.n_states && out_[k] < p.n_states && !(in_[k] >= 0 && in_[k] == out_[k]);
      if (!ok_[k]) report_status(p.status, kStatusBadIndex, 0xD20, rb + k, seq_[k]);
    }
#pragma unroll
    for (int k = 0; k < ROWS; ++k) {
      if (!ok_[k]) continue;
      const int r = rb + k, i = i_[k], n = n_[k], sin = in_[k], sout = out_[k];
      float acc[8];
#pragma unroll
      for (int j = 0; j < 8; ++j) acc[j] = b[j];
#pragma unroll
      for (int t = 0; t <= KEEP; ++t) {
        const int back = KEEP - t;
        if (back <= i) {
          float x[8];
          win[k + t].get(x);
#pragma unroll
          for (int j = 0; j < 8; ++j) acc[j] = fmaf(w[t][j], x[j], acc[j]);
        } else if (sin >= 0) {
          float o[8];
          act_load8(p.tail + (static_cast<long long>(sin) * KEEP + i + t) * p.channels + c, o);
#pragma unroll
          for (int j = 0; j < 8; ++j) acc[j] = fmaf(w[t][j], o[j], acc[j]);
        }
      }
      float x[8];
      win[k + KEEP].get(x);
      if (i == 0 || i >= n - KEEP) conv_tail(p.tail, p.channels, KEEP, c, i, n, sin, sout, x);
      conv_finish<RESIDUAL, SILU, kExact>(x, acc, p.out + r * p.ldo + c);
    }
  } else {
    pdl_wait();
    for (int k = 0; k < ROWS; ++k) {
      const int r = rb + k;
      int i, n, sin, sout;
      if (r >= p.rows || !conv_row(p, r, i, n, sin, sout)) continue;
      float acc[8], x[8], w[8];
      zero8<float>(acc);
      if (p.bias) act_load8(p.bias + c, acc);
      for (int t = 0; t <= keep; ++t) {
        const int back = keep - t;
        zero8<float>(x);
        if (back <= i) act_load8(p.x + (r - back) * p.ldx + c, x);
        else if (sin >= 0) act_load8(p.tail + (static_cast<long long>(sin) * keep + i + t) * p.channels + c, x);
        act_load8(p.w + static_cast<long long>(t) * p.channels + c, w);
#pragma unroll
        for (int j = 0; j < 8; ++j) acc[j] = fmaf(w[j], x[j], acc[j]);
      }
      if (i == 0 || i >= n - keep) conv_tail(p.tail, p.channels, keep, c, i, n, sin, sout, x);
      conv_finish<RESIDUAL, SILU, kExact>(x, acc, p.out + r * p.ldo + c);
    }
  }
}

}  // namespace fb

using namespace fb;

static int ok_launch() { return cudaGetLastError() == cudaSuccess ? FB_OK : FB_ERR_LAUNCH; }
static bool aligned16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

template <typename T>
static int launch_stream(const FbStreamArgs* a, cudaStream_t s) {
  StreamParams<T> p{};
  p.x = a->x; p.ldx = a->ldx;
  p.ids = a->ids; p.positions = a->positions;
  p.table = static_cast<const T*>(a->table); p.pos_table = static_cast<const T*>(a->pos_table); p.ldt = a->ldt;
  p.vocab = a->vocab; p.max_pos = a->max_pos;
  p.y = static_cast<const T*>(a->y); p.ldy = a->ldy;
  p.norm_w = a->norm_w; p.norm_b = a->norm_b; p.rms = a->rms;
  p.act = static_cast<T*>(a->act); p.lda = a->lda;
  p.conv = a->conv; p.tail = a->tail; p.state_in = a->state_in; p.state_out = a->state_out;
  p.taps = a->taps; p.n_states = a->n_states;
  p.h = static_cast<T*>(a->h); p.ldh = a->ldh;
  p.dim = a->dim; p.dim_pad = a->dim_pad; p.eps = a->eps;
  p.status = static_cast<DeviceStatus*>(a->status);
  const dim3 grid(a->rows), block(row_threads(a->dim_pad));
  switch (row_vpt(a->dim_pad)) {
    case 1: launch_pdl(stream_step_kernel<T, 1>, grid, block, 0, s, p); break;
    case 2: launch_pdl(stream_step_kernel<T, 2>, grid, block, 0, s, p); break;
    case 4: launch_pdl(stream_step_kernel<T, 4>, grid, block, 0, s, p); break;
    case 8: launch_pdl(stream_step_kernel<T, 8>, grid, block, 0, s, p); break;
    default: return FB_ERR_LIMIT;
  }
  return ok_launch();
}

extern "C" int fb_stream_step(const FbStreamArgs* a, void* stream) {
  if (!a || !a->x || a->rows <= 0 || a->dim <= 0 || a->dim_pad < a->dim || a->dim_pad % 8 || a->ldx < a->dim_pad || a->ldx % 8)
    return FB_ERR_SHAPE;
  if (!a->ids == !a->y) return FB_ERR_SHAPE;
  if (a->ids && (!a->table || a->ldt < a->dim_pad || a->ldt % 8 || a->vocab <= 0 || (a->pos_table && (!a->positions || a->max_pos <= 0))))
    return FB_ERR_SHAPE;
  if (a->y && (!a->norm_w || a->ldy < a->dim_pad || a->ldy % 8)) return FB_ERR_SHAPE;
  if (a->act && (a->lda < a->dim_pad || a->lda % 8)) return FB_ERR_SHAPE;
  if (a->conv && (!a->h || !a->state_in || !a->state_out || a->taps <= 0 || a->n_states <= 0 || a->ldh < a->dim_pad ||
                  a->ldh % 8 || (a->taps > 1 && !a->tail)))
    return FB_ERR_SHAPE;
  if (!aligned16(a->x) || !aligned16(a->table) || !aligned16(a->pos_table) || !aligned16(a->y) || !aligned16(a->act) ||
      !aligned16(a->h) || !aligned16(a->norm_w) || !aligned16(a->norm_b) || !aligned16(a->conv) || !aligned16(a->tail))
    return FB_ERR_ALIGN;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  return a->fp32 ? launch_stream<float>(a, s) : launch_stream<__nv_bfloat16>(a, s);
}

template <typename T>
static int launch_norm_rows(const float* x, long long ldx, int x_rows, const int* idx, int n, const float* w, const float* b,
                            int rms, void* out, long long ldo, int dim, int dim_pad, float eps, void* status, cudaStream_t s) {
  const dim3 grid(n), block(row_threads(dim_pad));
  T* o = static_cast<T*>(out);
  DeviceStatus* st = static_cast<DeviceStatus*>(status);
  switch (row_vpt(dim_pad)) {
    case 1: launch_pdl(norm_rows_kernel<T, 1>, grid, block, 0, s, x, ldx, x_rows, idx, w, b, rms, o, ldo, dim, dim_pad, eps, st); break;
    case 2: launch_pdl(norm_rows_kernel<T, 2>, grid, block, 0, s, x, ldx, x_rows, idx, w, b, rms, o, ldo, dim, dim_pad, eps, st); break;
    case 4: launch_pdl(norm_rows_kernel<T, 4>, grid, block, 0, s, x, ldx, x_rows, idx, w, b, rms, o, ldo, dim, dim_pad, eps, st); break;
    case 8: launch_pdl(norm_rows_kernel<T, 8>, grid, block, 0, s, x, ldx, x_rows, idx, w, b, rms, o, ldo, dim, dim_pad, eps, st); break;
    default: return FB_ERR_LIMIT;
  }
  return ok_launch();
}

extern "C" int fb_norm_rows(const float* x, long long ldx, int x_rows, const int* rows_idx, int n, const float* norm_w,
                            const float* norm_b, int rms, void* out, long long ldo, int dim, int dim_pad, float eps,
                            int fp32, void* status, void* stream) {
  if (!x || !rows_idx || !norm_w || !out || n <= 0 || x_rows <= 0 || dim <= 0 || dim_pad < dim || dim_pad % 8 ||
      ldx < dim_pad || ldo < dim_pad || ldx % 8 || ldo % 8)
    return FB_ERR_SHAPE;
  if (!aligned16(x) || !aligned16(norm_w) || !aligned16(norm_b) || !aligned16(out)) return FB_ERR_ALIGN;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  return fp32 ? launch_norm_rows<float>(x, ldx, x_rows, rows_idx, n, norm_w, norm_b, rms, out, ldo, dim, dim_pad, eps, status, s)
              : launch_norm_rows<__nv_bfloat16>(x, ldx, x_rows, rows_idx, n, norm_w, norm_b, rms, out, ldo, dim, dim_pad, eps,
                                                status, s);
}

template <typename T, int VPT>
static int launch_sandwich(const SandwichParams<T>& p, int rows, cudaStream_t s) {
  const size_t smem = (p.n_sums + p.groups) * sizeof(float);
  if (smem > 160 * 1024) return FB_ERR_LIMIT;
  static bool attr = false;
  if (smem > 40 * 1024 && !attr) {
    if (cudaFuncSetAttribute(sandwich_step_kernel<T, VPT>, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024) != cudaSuccess)
      return FB_ERR_LAUNCH;
    attr = true;
  }
  launch_pdl(sandwich_step_kernel<T, VPT>, dim3(rows), dim3(row_threads(p.dim_pad)), smem, s, p);
  return ok_launch();
}

template <typename T>
static int run_sandwich(const FbSandwichArgs* a, cudaStream_t s) {
  SandwichParams<T> p{};
  p.x = a->x; p.ldx = a->ldx;
  p.y = static_cast<const T*>(a->y); p.ldy = a->ldy; p.y_bias = a->y_bias; p.out_w = a->out_w;
  p.ids = a->ids; p.table = static_cast<const T*>(a->table); p.ldt = a->ldt; p.vocab = a->vocab; p.fresh = a->fresh;
  p.in_w = a->in_w; p.act = static_cast<T*>(a->act); p.lda = a->lda;
  p.dim = a->dim; p.dim_pad = a->dim_pad; p.groups = a->groups; p.n_sums = group_sums(a->dim, a->groups); p.eps = a->eps;
  p.status = static_cast<DeviceStatus*>(a->status);
  switch (row_vpt(a->dim_pad)) {
    case 1: return launch_sandwich<T, 1>(p, a->rows, s);
    case 2: return launch_sandwich<T, 2>(p, a->rows, s);
    case 4: return launch_sandwich<T, 4>(p, a->rows, s);
    case 8: return launch_sandwich<T, 8>(p, a->rows, s);
    default: return FB_ERR_LIMIT;
  }
}

extern "C" int fb_sandwich_step(const FbSandwichArgs* a, void* stream) {
  if (!a || !a->x || a->rows <= 0 || a->dim <= 0 || a->dim_pad < a->dim || a->dim_pad % 8 || a->ldx < a->dim_pad || a->ldx % 8 ||
      a->groups <= 0 || a->dim % a->groups)
    return FB_ERR_SHAPE;
  if (a->y && (!a->out_w || a->ldy < a->dim_pad || a->ldy % 8)) return FB_ERR_SHAPE;
  if (a->ids && (!a->table || a->ldt < a->dim_pad || a->ldt % 8 || a->vocab <= 0)) return FB_ERR_SHAPE;
  if (!a->act != !a->in_w || (a->act && (a->lda < a->dim_pad || a->lda % 8))) return FB_ERR_SHAPE;
  if (!aligned16(a->x) || !aligned16(a->y) || !aligned16(a->y_bias) || !aligned16(a->out_w) || !aligned16(a->table) ||
      !aligned16(a->in_w) || !aligned16(a->act))
    return FB_ERR_ALIGN;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  return a->fp32 ? run_sandwich<float>(a, s) : run_sandwich<__nv_bfloat16>(a, s);
}

template <typename T, int VPT>
static int launch_sandwich_rows(const float* x, long long ldx, int x_rows, const int* idx, int n, const float* w, void* out,
                                long long ldo, int dim, int dim_pad, int groups, float eps, void* status, cudaStream_t s) {
  const int n_sums = group_sums(dim, groups);
  const size_t smem = (n_sums + groups) * sizeof(float);
  if (smem > 160 * 1024) return FB_ERR_LIMIT;
  static bool attr = false;
  if (smem > 40 * 1024 && !attr) {
    if (cudaFuncSetAttribute(sandwich_rows_kernel<T, VPT>, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024) != cudaSuccess)
      return FB_ERR_LAUNCH;
    attr = true;
  }
  launch_pdl(sandwich_rows_kernel<T, VPT>, dim3(n), dim3(row_threads(dim_pad)), smem, s, x, ldx, x_rows, idx, w,
             static_cast<T*>(out), ldo, dim, dim_pad, groups, n_sums, eps, static_cast<DeviceStatus*>(status));
  return ok_launch();
}

template <typename T>
static int run_sandwich_rows(const float* x, long long ldx, int x_rows, const int* idx, int n, const float* w, void* out,
                             long long ldo, int dim, int dim_pad, int groups, float eps, void* status, cudaStream_t s) {
  switch (row_vpt(dim_pad)) {
    case 1: return launch_sandwich_rows<T, 1>(x, ldx, x_rows, idx, n, w, out, ldo, dim, dim_pad, groups, eps, status, s);
    case 2: return launch_sandwich_rows<T, 2>(x, ldx, x_rows, idx, n, w, out, ldo, dim, dim_pad, groups, eps, status, s);
    case 4: return launch_sandwich_rows<T, 4>(x, ldx, x_rows, idx, n, w, out, ldo, dim, dim_pad, groups, eps, status, s);
    case 8: return launch_sandwich_rows<T, 8>(x, ldx, x_rows, idx, n, w, out, ldo, dim, dim_pad, groups, eps, status, s);
    default: return FB_ERR_LIMIT;
  }
}

extern "C" int fb_sandwich_rows(const float* x, long long ldx, int x_rows, const int* rows_idx, int n, const float* w, void* out,
                                long long ldo, int dim, int dim_pad, int groups, float eps, int fp32, void* status, void* stream) {
  if (!x || !rows_idx || !w || !out || n <= 0 || x_rows <= 0 || dim <= 0 || dim_pad < dim || dim_pad % 8 || ldx < dim_pad ||
      ldo < dim_pad || ldx % 8 || ldo % 8 || groups <= 0 || dim % groups)
    return FB_ERR_SHAPE;
  if (!aligned16(x) || !aligned16(w) || !aligned16(out)) return FB_ERR_ALIGN;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  return fp32 ? run_sandwich_rows<float>(x, ldx, x_rows, rows_idx, n, w, out, ldo, dim, dim_pad, groups, eps, status, s)
              : run_sandwich_rows<__nv_bfloat16>(x, ldx, x_rows, rows_idx, n, w, out, ldo, dim, dim_pad, groups, eps, status, s);
}

template <typename TI, typename TO, int KEEP, int ROWS>
static int launch_conv_rows(const ConvParams<TI, TO>& p, bool residual, bool silu, cudaStream_t s) {
  const dim3 grid((p.channels / 8 + 127) / 128, (p.rows + ROWS - 1) / ROWS);
  if (grid.y > 65535) return FB_ERR_LIMIT;
  if (residual && silu) return FB_ERR_SHAPE;
  if (residual) launch_pdl(short_conv_kernel<TI, TO, KEEP, ROWS, true, false>, grid, dim3(128), 0, s, p);
  else if (silu) launch_pdl(short_conv_kernel<TI, TO, KEEP, ROWS, false, true>, grid, dim3(128), 0, s, p);
  else launch_pdl(short_conv_kernel<TI, TO, KEEP, ROWS, false, false>, grid, dim3(128), 0, s, p);
  return ok_launch();
}

template <typename TI, typename TO>
static int launch_conv(const FbConvArgs* a, cudaStream_t s) {
  ConvParams<TI, TO> p{};
  p.x = static_cast<const TI*>(a->x); p.ldx = a->ldx; p.w = a->w; p.bias = a->bias; p.tail = static_cast<TI*>(a->tail);
  p.out = static_cast<TO*>(a->out); p.ldo = a->ldo;
  p.row_seq = a->row_seq; p.seq_start = a->seq_start; p.state_in = a->state_in; p.state_out = a->state_out;
  p.rows = a->rows; p.channels = a->channels; p.taps = a->taps; p.n_states = a->n_states; p.n_seqs = a->n_seqs;
  p.status = static_cast<DeviceStatus*>(a->status);
  const bool res = a->residual != 0, silu = a->silu != 0, one = a->n_seqs == a->rows;
  if (a->taps == 4)
    return one ? launch_conv_rows<TI, TO, 3, 1>(p, res, silu, s) : launch_conv_rows<TI, TO, 3, 4>(p, res, silu, s);
  if (a->taps == 3) return launch_conv_rows<TI, TO, 2, 4>(p, res, silu, s);
  if (a->taps == 2) return launch_conv_rows<TI, TO, 1, 4>(p, res, silu, s);
  return launch_conv_rows<TI, TO, -1, 4>(p, res, silu, s);
}

extern "C" int fb_short_conv(const FbConvArgs* a, void* stream) {
  if (!a || !a->x || !a->w || !a->out || !a->row_seq || !a->seq_start || !a->state_in || !a->state_out || a->rows <= 0 ||
      a->channels <= 0 || a->channels % 8 || a->taps <= 0 || a->n_states <= 0 || a->n_seqs <= 0 || (a->taps > 1 && !a->tail))
    return FB_ERR_SHAPE;
  if (a->ldx < a->channels || a->ldo < a->channels || a->ldx % 8 || a->ldo % 8) return FB_ERR_SHAPE;
  if (!aligned16(a->x) || !aligned16(a->w) || !aligned16(a->bias) || !aligned16(a->tail) || !aligned16(a->out))
    return FB_ERR_ALIGN;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (a->x_fp32) return a->out_fp32 ? launch_conv<float, float>(a, s) : launch_conv<float, __nv_bfloat16>(a, s);
  if (a->out_fp32) return FB_ERR_SHAPE;
  return launch_conv<__nv_bfloat16, __nv_bfloat16>(a, s);
}
