// Gated delta rule with one decay per key channel or per head, short causal convolutions in front, gated per-head output
// norm (sigmoid or SiLU gate).
//
// Per head, S [dim, vdim] in fp32, rows of key channels (g_t one number with a decay per head):
//     S <- diag(g_t) S;   u = beta_t (v_t - S^T k_t);   S <- S + k_t u^T;   o_t = S^T q_t
// with q, k the unit vectors (q also times dim^-1/2) of silu(conv(W x)), v = silu(conv(W_v x)),
// g = exp(a_neg * softplus(decay + dt_bias)), beta = sigmoid(b).
//
// State of a sequence: one S per head and the last taps - 1 projected inputs of every convolved channel.  A slot of
// the state pool has several buffers; a step reads buffer `state_in[seq]` (-1: a new sequence, all zeros) and writes
// buffer `state_out[seq]` (-1: nothing is kept), so a step that is rolled back leaves the committed state untouched.
//
//   fb_delta_decode   one row per sequence, everything in one launch: one CTA per (sequence, head), the state slice in
//                     registers (16 bytes per thread and row)
//   fb_delta_prefill  any mix of row counts: prepare (convolutions, unit norms, decays; one CTA per row) -> scan (the
//                     recurrence, state in registers, eight lanes per value column) -> output norm and gate
//
// S^T q after the write equals S^T q before it plus (q . k) u, so both dot products of a token are taken in one pass
// over the decayed state.
#include "act_type.cuh"
#include "common.cuh"
#include "f32x2.cuh"
#include "ferrule_b200.h"
#include "launch.cuh"

namespace fb {

template <typename T>
struct DeltaParams {
  const T* proj;              // [rows, ldp]: pre-convolution q | k | v at off_q / off_k / off_v, beta logits at off_b
  long long ldp;
  int off_q, off_k, off_v, off_b;
  const float* ag;            // [rows, ldag]: decay pre-activation at 0, output gate pre-activation at off_gate
  long long ldag;
  int off_gate;
  int off_a;                  // >= 0: one decay per head, its pre-activation in column off_a + h of a projected row
  int off_g;                  // >= 0: output gate pre-activation in columns off_g .. of a projected row instead of `ag`
  int gate_silu;
  const float* conv;          // [taps, channels], channels = q | k | v
  const float* a_neg;         // [heads]
  const float* dt_bias;       // [heads * dim], one decay per head: [heads]
  const float* norm_w;        // [vdim]
  float eps;
  float* state;               // [n_states, heads, dim, vdim]
  T* tail;                    // [n_states, taps - 1, channels]
  int n_states;
  const int* row_seq;
  const int* seq_start;       // [n_seqs + 1]
  const int* state_in;
  const int* state_out;
  int rows, n_seqs, heads, kv_heads, dim, vdim, taps, long_seqs;
  float *qn, *kn, *v, *decay, *beta, *qk, *o;      // scratch of the prefill form
  T* out;                     // [rows, ldo]
  long long ldo;
  DeviceStatus* status;
  __device__ int channels() const { return 2 * kv_heads * dim + heads * vdim; }
  // column of channel c in a projected row
  __device__ int col(int c) const {
    const int nk = kv_heads * dim;
    return c < nk ? off_q + c : (c < 2 * nk ? off_k + c - nk : off_v + c - 2 * nk);
  }
};

// silu(conv) of channel c at local row i of the sequence whose rows start at r0
template <typename T>
__device__ __forceinline__ float conv_silu(const DeltaParams<T>& p, int c, int r0, int i, int sin, int channels) {
  const int col = p.col(c), taps = p.taps;
  float acc = 0.f;
  for (int j = 0; j < taps; ++j) {
    const int idx = i - (taps - 1) + j;
    float x = 0.f;
    if (idx >= 0) x = act_load(p.proj + (r0 + idx) * p.ldp + col);
    else if (sin >= 0) x = act_load(p.tail + (static_cast<long long>(sin) * (taps - 1) + idx + taps - 1) * channels + c);
    acc = fmaf(p.conv[static_cast<long long>(j) * channels + c], x, acc);
  }
  return acc / (1.f + expf(-acc));
}

// The convolution inputs the next step needs: entry j of the tail is the input `taps - 1 - j` tokens before the end.
// Called for local row i of n: that row's own entry, and by row 0 the entries that still come from the old tail.
template <typename T>
__device__ __forceinline__ void store_tail(const DeltaParams<T>& p, int c, int r0, int i, int n, int sin, int sout,
                                           int channels) {
  const int keep = p.taps - 1;
  if (sout < 0 || keep <= 0) return;
  T* dst = p.tail + static_cast<long long>(sout) * keep * channels + c;
  const int j = i - (n - keep);
  if (j >= 0) dst[static_cast<long long>(j) * channels] = p.proj[(r0 + i) * p.ldp + p.col(c)];
  if (i == 0) {
    for (int q = 0; q < keep - n; ++q) {
      T x{};
      if (sin >= 0) x = p.tail[(static_cast<long long>(sin) * keep + q + n) * channels + c];
      else act_store(&x, 0.f);
      dst[static_cast<long long>(q) * channels] = x;
    }
  }
}

template <typename T>
__device__ __forceinline__ bool seq_states(const DeltaParams<T>& p, int seq, int& sin, int& sout) {
  sin = p.state_in[seq];
  sout = p.state_out[seq];
  if (sin >= p.n_states || sout >= p.n_states || (sin >= 0 && sin == sout)) {
    if (threadIdx.x == 0) report_status(p.status, kStatusBadIndex, 0xC00, seq, sout);
    return false;
  }
  return true;
}

// exp(a * softplus(z)) and silu(z).  bf16 models take the hardware exponential and logarithm (a few 1e-7 relative, far
// below the rounding of z itself), fp32 models the full-precision functions.
template <typename T>
__device__ __forceinline__ float decay_of(float a, float z) {
  if constexpr (sizeof(T) == 4) return expf(a * softplus_f(z));
  const float e = __expf(-fabsf(z)), w = 1.f + e;
  // log1p(e) = log(w) * e / (w - 1): the quotient restores what rounding w lost
  const float l = w == 1.f ? e : __logf(w) * __fdividef(e, w - 1.f);
  return __expf(a * (fmaxf(z, 0.f) + l));
}
template <typename T>
__device__ __forceinline__ float silu_of(float z) {
  if constexpr (sizeof(T) == 4) return z / (1.f + expf(-z));
  return __fdividef(z, 1.f + __expf(-z));
}

template <typename T>
__device__ __forceinline__ float output_gate(const DeltaParams<T>& p, float z) {
  return p.gate_silu ? silu_of<T>(z) : sigmoid_f(z);
}
// pre-activation of the output gate of value column i (head * vdim + column) of row r
template <typename T>
__device__ __forceinline__ float gate_pre(const DeltaParams<T>& p, long long r, int i) {
  return p.off_g >= 0 ? act_load(p.proj + r * p.ldp + p.off_g + i) : p.ag[r * p.ldag + p.off_gate + i];
}

// ---------------------------------------------------------------------------------
// prepare: one CTA per row.  VEC consecutive channels per thread (4 when every block of channels is a multiple of 4)
// ---------------------------------------------------------------------------------
// (reads of memory the kernel never writes: independent iterations may then be in flight together)
__device__ __forceinline__ void load_vec(const __nv_bfloat16* p, float (&v)[4]) {
  const uint2 a = __ldg(reinterpret_cast<const uint2*>(p));
  const __nv_bfloat16* e = reinterpret_cast<const __nv_bfloat16*>(&a);
#pragma unroll
  for (int j = 0; j < 4; ++j) v[j] = __bfloat162float(e[j]);
}
__device__ __forceinline__ void load_vec(const float* p, float (&v)[4]) {
  const float4 a = __ldg(reinterpret_cast<const float4*>(p));
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
}
__device__ __forceinline__ void load_vec(const __nv_bfloat16* p, float (&v)[1]) { v[0] = __bfloat162float(__ldg(p)); }
__device__ __forceinline__ void load_vec(const float* p, float (&v)[1]) { v[0] = __ldg(p); }
__device__ __forceinline__ void store_vec(float* p, const float (&v)[4]) {
  *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
}
__device__ __forceinline__ void store_vec(float* p, const float (&v)[1]) { p[0] = v[0]; }

// convolution and silu of channels [c0, c0 + n) of one row into `dst`, whose inputs start at column `col0`
template <int VEC, typename T>
__device__ __forceinline__ void conv_block(const DeltaParams<T>& p, int c0, int n, int col0, int r, int i, int sin,
                                           int channels, float* dst) {
  const int keep = p.taps - 1;
  const T* tail = p.tail + static_cast<long long>(max(sin, 0)) * keep * channels;
#pragma unroll 2
  for (int c = threadIdx.x * VEC; c < n; c += blockDim.x * VEC) {
    float acc[VEC], x[VEC], w[VEC];
#pragma unroll
    for (int e = 0; e < VEC; ++e) acc[e] = 0.f;
    const T* in = p.proj + r * p.ldp + col0 + c;
    if (keep <= 3 && i >= keep) {
      // every tap lies in this batch: all loads go out together
      float xs[4][VEC], wf[4][VEC];
#pragma unroll
      for (int b = 0; b < 4; ++b) {
        if (b <= keep) {
          load_vec(in - b * p.ldp, xs[b]);
          load_vec(p.conv + static_cast<long long>(keep - b) * channels + c0 + c, wf[b]);
        }
      }
#pragma unroll
      for (int b = 3; b >= 0; --b)
        if (b <= keep) {
#pragma unroll
          for (int e = 0; e < VEC; ++e) acc[e] = fmaf(wf[b][e], xs[b][e], acc[e]);
        }
    } else
    for (int j = 0; j <= keep; ++j) {
      const int back = keep - j;                          // tokens before this one
      load_vec(p.conv + static_cast<long long>(j) * channels + c0 + c, w);
      if (back <= i) {
        load_vec(in - back * p.ldp, x);
      } else {
        // (the tails are written by this launch: plain loads)
#pragma unroll
        for (int e = 0; e < VEC; ++e)
          x[e] = sin >= 0 ? act_load(tail + static_cast<long long>(i + j) * channels + c0 + c + e) : 0.f;
      }
#pragma unroll
      for (int e = 0; e < VEC; ++e) acc[e] = fmaf(w[e], x[e], acc[e]);
    }
#pragma unroll
    for (int e = 0; e < VEC; ++e) acc[e] = silu_of<T>(acc[e]);
    store_vec(dst + c, acc);
  }
}

template <typename T, int VEC>
__global__ void __launch_bounds__(256)
delta_prepare_kernel(const DeltaParams<T> p) {
  // no early release: the scan's CTAs would be packed onto the first SMs with room instead of spreading over all
  pdl_wait();
  extern __shared__ __align__(16) float qk_s[];   // [2 * kv_heads * dim]
  const int r = blockIdx.x;
  const int seq = p.row_seq[r];
  if (seq < 0 || seq >= p.n_seqs) {
    if (threadIdx.x == 0) report_status(p.status, kStatusBadIndex, 0xC01, r, seq);
    return;
  }
  const int r0 = p.seq_start[seq], n = p.seq_start[seq + 1] - r0, i = r - r0;
  if (r0 < 0 || i < 0 || i >= n || r0 + n > p.rows) {
    if (threadIdx.x == 0) report_status(p.status, kStatusBadIndex, 0xC02, r, r0);
    return;
  }
  int sin, sout;
  if (!seq_states(p, seq, sin, sout)) return;
  const int nk = p.kv_heads * p.dim, nv = p.heads * p.vdim, channels = p.channels();
  conv_block<VEC>(p, 0, nk, p.off_q, r, i, sin, channels, qk_s);
  conv_block<VEC>(p, nk, nk, p.off_k, r, i, sin, channels, qk_s + nk);
  conv_block<VEC>(p, 2 * nk, nv, p.off_v, r, i, sin, channels, p.v + static_cast<long long>(r) * nv);
  if (i == 0 || i > n - p.taps)
    for (int c = threadIdx.x; c < channels; c += blockDim.x) store_tail(p, c, r0, i, n, sin, sout, channels);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  if (p.off_a >= 0) {
    for (int h = threadIdx.x; h < p.heads; h += blockDim.x)
      p.decay[static_cast<long long>(r) * p.heads + h] =
          decay_of<T>(p.a_neg[h], act_load(p.proj + r * p.ldp + p.off_a + h) + p.dt_bias[h]);
  } else
  for (int h = warp; h < p.heads; h += nw) {
    const float a = p.a_neg[h];
    const float* pre = p.ag + r * p.ldag + h * p.dim;
    const float* bias = p.dt_bias + h * p.dim;
    float* dst = p.decay + (static_cast<long long>(r) * p.heads + h) * p.dim;
#pragma unroll 4
    for (int d = lane; d < p.dim; d += 32) dst[d] = decay_of<T>(a, __ldg(pre + d) + __ldg(bias + d));
  }
  for (int h = threadIdx.x; h < p.heads; h += blockDim.x)
    p.beta[static_cast<long long>(r) * p.heads + h] = sigmoid_f(act_load(p.proj + r * p.ldp + p.off_b + h));
  __syncthreads();
  for (int h = warp; h < p.kv_heads; h += nw) {
    const float* q = qk_s + h * p.dim;
    const float* k = qk_s + nk + h * p.dim;
    float sq = 0.f, sk = 0.f, dot = 0.f;
    for (int d = lane; d < p.dim; d += 32) {
      sq = fmaf(q[d], q[d], sq);
      sk = fmaf(k[d], k[d], sk);
      dot = fmaf(q[d], k[d], dot);
    }
    sq = warp_sum(sq);
    sk = warp_sum(sk);
    dot = warp_sum(dot);
    const float fq = 1.f / sqrtf(sq + 1e-6f) / sqrtf(static_cast<float>(p.dim)), fk = 1.f / sqrtf(sk + 1e-6f);
    const long long base = static_cast<long long>(r) * nk + h * p.dim;
    for (int d = lane; d < p.dim; d += 32) {
      p.qn[base + d] = q[d] * fq;
      p.kn[base + d] = k[d] * fk;
    }
    if (lane == 0) p.qk[static_cast<long long>(r) * p.kv_heads + h] = dot * fq * fk;
  }
}

__device__ __forceinline__ void cp_async4(float* dst, const float* src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async16(float* dst, const float* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
}

// ---------------------------------------------------------------------------------
// scan: CTA = (head, 16 * COLS value columns) x sequence; eight lanes share COLS columns, lane l holds the key channels
// 32 * (j / 4) + 4 * l + j % 4.  Tokens are staged sixteen at a time, double buffered.  More columns per lane mean
// fewer shared-memory reads of k, q and g per column; the launcher takes as many as still fill the GPU.
// ---------------------------------------------------------------------------------
constexpr int kScanStep = 16;

// HEADG: one decay per head.  The dot products are then taken over the state before the decay and scaled, so that the
// decay of the state runs beside them instead of ahead of them.
template <typename T, int RPT, int COLS, bool HEADG>
constexpr int scan_buf() { return kScanStep * ((HEADG ? 2 : 3) * RPT * 8 + 16 * COLS + 2 + (HEADG ? 1 : 0)); }

template <typename T, int RPT, int COLS, bool HEADG>
__global__ void __launch_bounds__(128)
delta_scan_kernel(const DeltaParams<T> p) {
  // the dependents are released at the end: their CTAs would only wait, on the SMs this long kernel needs
  pdl_wait();
  constexpr int DP = RPT * 8;                                   // padded key dimension
  constexpr int kCols = 16 * COLS;
  extern __shared__ __align__(16) float sm[];
  // per buffer: k, q, g [kScanStep][DP], v [kScanStep][kCols], beta, qk [kScanStep]; one decay per head: no g rows,
  // g [kScanStep] at the end
  constexpr int kBuf = scan_buf<T, RPT, COLS, HEADG>();
  constexpr int kV = (HEADG ? 2 : 3) * kScanStep * DP;          // first float of v
  // (a mixed batch lists its decode rows first: the long sequences' CTAs start first and spread over all SMs)
  const int seq = gridDim.y - 1 - blockIdx.y;
  const int vtiles = (p.vdim + kCols - 1) / kCols;
  const int h = blockIdx.x / vtiles, v0 = (blockIdx.x - h * vtiles) * kCols;
  const int hk = h / (p.heads / p.kv_heads);
  const int r0 = p.seq_start[seq], n = p.seq_start[seq + 1] - r0;
  if (r0 < 0 || n <= 0 || r0 + n > p.rows) return;              // reported by the prepare kernel
  int sin, sout;
  if (!seq_states(p, seq, sin, sout)) return;
  const int tid = threadIdx.x, l8 = tid & 7;
  const int vc = (tid >> 3) * COLS;                             // first column of this lane inside the tile
  for (int i = tid; i < 2 * kBuf; i += 128) sm[i] = 0.f;        // padding channels stay zero

  uint64_t S[COLS][RPT / 2];                                    // pairs of neighbouring key channels
  const long long per_state = static_cast<long long>(p.heads) * p.dim * p.vdim;
  const long long sbase = static_cast<long long>(h) * p.dim * p.vdim + v0 + vc;
#pragma unroll
  for (int j = 0; j < RPT; j += 2) {
    const int d = (j / 4) * 32 + l8 * 4 + (j & 3);
    const float* src = p.state + max(sin, 0) * per_state + sbase + static_cast<long long>(d) * p.vdim;
#pragma unroll
    for (int c = 0; c < COLS; ++c) {
      const bool in = sin >= 0 && v0 + vc + c < p.vdim;
      S[c][j / 2] = pack2(in && d < p.dim ? src[c] : 0.f, in && d + 1 < p.dim ? src[p.vdim + c] : 0.f);
    }
  }
  __syncthreads();
  const long long ldk = static_cast<long long>(p.kv_heads) * p.dim, ldg = static_cast<long long>(p.heads) * p.dim,
                  ldv = static_cast<long long>(p.heads) * p.vdim;
  auto stage = [&](int t0, int b) {
    float* base = sm + b * kBuf;
    const int cnt = min(kScanStep, n - t0);
    if ((p.dim & 3) == 0) {
      const int q4 = p.dim >> 2;
      for (int i = tid; i < cnt * q4; i += 128) {
        const int t = i / q4, d = (i - t * q4) * 4;
        const long long r = r0 + t0 + t;
        cp_async16(base + t * DP + d, p.kn + r * ldk + hk * p.dim + d);
        cp_async16(base + kScanStep * DP + t * DP + d, p.qn + r * ldk + hk * p.dim + d);
        if (!HEADG) cp_async16(base + 2 * kScanStep * DP + t * DP + d, p.decay + r * ldg + h * p.dim + d);
      }
    } else {
      for (int i = tid; i < cnt * p.dim; i += 128) {
        const int t = i / p.dim, d = i - t * p.dim;
        const long long r = r0 + t0 + t;
        cp_async4(base + t * DP + d, p.kn + r * ldk + hk * p.dim + d);
        cp_async4(base + kScanStep * DP + t * DP + d, p.qn + r * ldk + hk * p.dim + d);
        if (!HEADG) cp_async4(base + 2 * kScanStep * DP + t * DP + d, p.decay + r * ldg + h * p.dim + d);
      }
    }
    float* vb = base + kV;
    for (int i = tid; i < cnt * kCols; i += 128) {
      const int t = i / kCols, c = i - t * kCols;
      if (v0 + c < p.vdim) cp_async4(vb + i, p.v + (r0 + t0 + t) * ldv + h * p.vdim + v0 + c);
    }
    if (tid < cnt) {
      cp_async4(vb + kScanStep * kCols + tid, p.beta + static_cast<long long>(r0 + t0 + tid) * p.heads + h);
      cp_async4(vb + kScanStep * kCols + kScanStep + tid, p.qk + static_cast<long long>(r0 + t0 + tid) * p.kv_heads + hk);
      if (HEADG)
        cp_async4(vb + kScanStep * kCols + 2 * kScanStep + tid, p.decay + static_cast<long long>(r0 + t0 + tid) * p.heads + h);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  stage(0, 0);
  int b = 0;
  for (int t0 = 0; t0 < n; t0 += kScanStep, b ^= 1) {
    if (t0 + kScanStep < n) {
      stage(t0 + kScanStep, b ^ 1);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    const float* base = sm + b * kBuf;
    const float* vb = base + kV;
    const int cnt = min(kScanStep, n - t0);
    uint64_t k[RPT / 2], q[RPT / 2], g[RPT / 2];
    auto fetch = [&](int t) {
#pragma unroll
      for (int j = 0; j < RPT / 4; ++j) {
        const float* row = base + t * DP + j * 32 + l8 * 4;
        const ulonglong2 a = *reinterpret_cast<const ulonglong2*>(row);
        const ulonglong2 c = *reinterpret_cast<const ulonglong2*>(row + kScanStep * DP);
        k[2 * j] = a.x; k[2 * j + 1] = a.y;
        q[2 * j] = c.x; q[2 * j + 1] = c.y;
        if (!HEADG) {
          const ulonglong2 e = *reinterpret_cast<const ulonglong2*>(row + 2 * kScanStep * DP);
          g[2 * j] = e.x; g[2 * j + 1] = e.y;
        }
      }
    };
    fetch(0);
    float* o = p.o + (r0 + t0) * ldv + h * p.vdim + v0 + vc + l8;
    const bool writer = l8 < COLS && v0 + vc + l8 < p.vdim;
    for (int t = 0; t < cnt; ++t, o += ldv) {
      const float beta = vb[kScanStep * kCols + t], qk = vb[kScanStep * kCols + kScanStep + t];
      float sk[COLS], sq[COLS], vt[COLS], out = 0.f;
      const float gh = HEADG ? vb[kScanStep * kCols + 2 * kScanStep + t] : 1.f;
      const uint64_t gh2 = pack2(gh, gh);
#pragma unroll
      for (int c = 0; c < COLS; ++c) vt[c] = vb[t * kCols + vc + c];
#pragma unroll
      for (int c = 0; c < COLS; ++c) {
        uint64_t ka = 0, kb = 0, qa = 0, qb = 0;          // two chains each
#pragma unroll
        for (int j = 0; j < RPT / 2; j += 2) {
          if (!HEADG) {
            S[c][j] = mul2(S[c][j], g[j]);
            S[c][j + 1] = mul2(S[c][j + 1], g[j + 1]);
          }
          ka = fma2(S[c][j], k[j], ka);
          kb = fma2(S[c][j + 1], k[j + 1], kb);
          qa = fma2(S[c][j], q[j], qa);
          qb = fma2(S[c][j + 1], q[j + 1], qb);
        }
        float a0, a1, b0, b1;
        unpack2(ka, a0, a1);
        unpack2(kb, b0, b1);
        sk[c] = (a0 + b0) + (a1 + b1);
        unpack2(qa, a0, a1);
        unpack2(qb, b0, b1);
        sq[c] = (a0 + b0) + (a1 + b1);
        if (HEADG) {
#pragma unroll
          for (int j = 0; j < RPT / 2; ++j) S[c][j] = mul2(S[c][j], gh2);
        }
      }
#pragma unroll
      for (int x = 1; x < 8; x <<= 1)
#pragma unroll
        for (int c = 0; c < COLS; ++c) {
          sk[c] += __shfl_xor_sync(0xffffffffu, sk[c], x);
          sq[c] += __shfl_xor_sync(0xffffffffu, sq[c], x);
        }
#pragma unroll
      for (int c = 0; c < COLS; ++c) {
        const float u = beta * (HEADG ? fmaf(-gh, sk[c], vt[c]) : vt[c] - sk[c]);
        if (l8 == c) out = fmaf(qk, u, HEADG ? gh * sq[c] : sq[c]);
        const uint64_t u2 = pack2(u, u);
#pragma unroll
        for (int j = 0; j < RPT / 2; ++j) S[c][j] = fma2(k[j], u2, S[c][j]);
      }
      fetch(min(t + 1, kScanStep - 1));
      if (writer) *o = out;
    }
    __syncthreads();
  }
  pdl_launch_dependents();
  if (sout >= 0) {
#pragma unroll
    for (int j = 0; j < RPT; j += 2) {
      const int d = (j / 4) * 32 + l8 * 4 + (j & 3);
      float* dst = p.state + sout * per_state + sbase + static_cast<long long>(d) * p.vdim;
#pragma unroll
      for (int c = 0; c < COLS; ++c) {
        if (v0 + vc + c >= p.vdim) continue;
        float a0, a1;
        unpack2(S[c][j / 2], a0, a1);
        if (d < p.dim) dst[c] = a0;
        if (d + 1 < p.dim) dst[p.vdim + c] = a1;
      }
    }
  }
}

// output norm and gate: one warp per (row, head)
template <typename T>
__global__ void __launch_bounds__(128)
delta_output_kernel(const DeltaParams<T> p) {
  pdl_launch_dependents();
  pdl_wait();
  const long long i = static_cast<long long>(blockIdx.x) * 4 + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  if (i >= static_cast<long long>(p.rows) * p.heads) return;
  const long long r = i / p.heads;
  const int h = static_cast<int>(i - r * p.heads);
  const float* o = p.o + i * p.vdim;
  const bool gate_vec = p.off_g >= 0 ? (p.off_g & 3) == 0 && (p.ldp & 3) == 0 : (p.ldag & 3) == 0 && (p.off_gate & 3) == 0;
  if (p.vdim <= 128 && (p.vdim & 3) == 0 && gate_vec) {
    // four columns per lane, everything requested up front
    const int v = lane * 4;
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f), w = a;
    float g[4] = {};
    if (v < p.vdim) {
      a = *reinterpret_cast<const float4*>(o + v);
      if (p.off_g >= 0) load_vec(p.proj + r * p.ldp + p.off_g + h * p.vdim + v, g);
      else load_vec(p.ag + r * p.ldag + p.off_gate + h * p.vdim + v, g);
      w = *reinterpret_cast<const float4*>(p.norm_w + v);
    }
    const float inv = 1.f / sqrtf(warp_sum(a.x * a.x + a.y * a.y + a.z * a.z + a.w * a.w) / p.vdim + p.eps);
    if (v < p.vdim) {
      T* dst = p.out + r * p.ldo + h * p.vdim + v;
      act_store(dst, a.x * inv * w.x * output_gate(p, g[0]));
      act_store(dst + 1, a.y * inv * w.y * output_gate(p, g[1]));
      act_store(dst + 2, a.z * inv * w.z * output_gate(p, g[2]));
      act_store(dst + 3, a.w * inv * w.w * output_gate(p, g[3]));
    }
    return;
  }
  float ss = 0.f;
  for (int v = lane; v < p.vdim; v += 32) ss = fmaf(o[v], o[v], ss);
  ss = warp_sum(ss);
  const float inv = 1.f / sqrtf(ss / p.vdim + p.eps);
  for (int v = lane; v < p.vdim; v += 32)
    act_store(p.out + r * p.ldo + h * p.vdim + v,
              o[v] * inv * p.norm_w[v] * output_gate(p, gate_pre(p, r, h * p.vdim + v)));
}

// ---------------------------------------------------------------------------------
// decode: CTA = (sequence, head), 8 warps; lane l holds the value columns 4l .. 4l + 3, warp w the key channels
// w, w + 8, ...  Needs vdim <= 128, vdim % 4 == 0, dim <= 8 * RW.
// ---------------------------------------------------------------------------------
// convolution and silu of channel c for the only row of its sequence; with `keep_inputs` also the tail for the next step
template <typename T>
__device__ __forceinline__ float conv_step(const DeltaParams<T>& p, int c, int r, int sin, int sout, int channels,
                                           bool keep_inputs) {
  const int keep = p.taps - 1;
  if (keep > 3) {
    if (keep_inputs) store_tail(p, c, r, 0, 1, sin, sout, channels);
    return conv_silu(p, c, r, 0, sin, channels);
  }
  // inputs and taps are requested together; x[keep] is the current token's input
  float x[4], w[4], acc = 0.f;
  const T* old = p.tail + static_cast<long long>(max(sin, 0)) * keep * channels + c;
#pragma unroll
  for (int b = 0; b < 4; ++b) {
    x[b] = w[b] = 0.f;
    if (b < keep && sin >= 0) x[b] = act_load(old + static_cast<long long>(b) * channels);
    if (b <= keep) w[b] = p.conv[static_cast<long long>(b) * channels + c];
  }
  const float cur = act_load(p.proj + r * p.ldp + p.col(c));
#pragma unroll
  for (int b = 0; b < 4; ++b) {
    if (b == keep) x[b] = cur;
    if (b <= keep) acc = fmaf(w[b], x[b], acc);
  }
  if (keep_inputs && sout >= 0) {
    T* dst = p.tail + static_cast<long long>(sout) * keep * channels + c;
#pragma unroll
    for (int b = 0; b < 3; ++b)
      if (b < keep) act_store(dst + static_cast<long long>(b) * channels, x[b + 1]);
  }
  return silu_of<T>(acc);
}

template <typename T, int RW>
__global__ void __launch_bounds__(256)
delta_decode_kernel(const DeltaParams<T> p) {
  pdl_launch_dependents();
  __shared__ float s_q[8 * RW], s_k[8 * RW], s_g[8 * RW], s_v[128], s_red[2][8][128];
  const int seq = blockIdx.x, h = blockIdx.y;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int hk = h / (p.heads / p.kv_heads);
  // the state binding and the sequence's state precede the running step: their loads go out before the dependency wait
  int sin, sout;
  const bool ok = seq_states(p, seq, sin, sout);
  const long long per_state = static_cast<long long>(p.heads) * p.dim * p.vdim;
  const int vcol = lane * 4;
  const bool vok = vcol < p.vdim;
  float4 S[RW];
#pragma unroll
  for (int j = 0; j < RW; ++j) {
    const int d = warp + 8 * j;
    S[j] = (ok && sin >= 0 && vok && d < p.dim)
               ? *reinterpret_cast<const float4*>(p.state + sin * per_state +
                                                  (static_cast<long long>(h) * p.dim + d) * p.vdim + vcol)
               : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  pdl_wait();
  if (!ok) return;
  const int r = p.seq_start[seq];
  if (r < 0 || r >= p.rows || p.seq_start[seq + 1] != r + 1) {
    if (tid == 0) report_status(p.status, kStatusBadIndex, 0xC03, seq, r);
    return;
  }
  const int nk = p.kv_heads * p.dim, channels = p.channels();
  const int first = h % (p.heads / p.kv_heads) == 0;         // this CTA also keeps the shared q / k inputs
  // channels of this head: q (8 RW entries, zero past dim) | k | v, then the decays
  for (int i = tid; i < 16 * RW + 128; i += 256) {
    const int part = i < 8 * RW ? 0 : (i < 16 * RW ? 1 : 2), d = part == 2 ? i - 16 * RW : i - part * 8 * RW;
    float y = 0.f;
    if (d < (part == 2 ? p.vdim : p.dim)) {
      const int c = part == 2 ? 2 * nk + h * p.vdim + d : part * nk + hk * p.dim + d;
      y = conv_step(p, c, r, sin, sout, channels, part == 2 || first);
    }
    (part == 0 ? s_q : part == 1 ? s_k : s_v)[d] = y;
  }
  const float gh = p.off_a >= 0 ? decay_of<T>(p.a_neg[h], act_load(p.proj + r * p.ldp + p.off_a + h) + p.dt_bias[h]) : 0.f;
  for (int d = tid; d < 8 * RW; d += 256) {
    const int c = h * p.dim + d;
    if (p.off_a >= 0) s_g[d] = d < p.dim ? gh : 0.f;
    else s_g[d] = d < p.dim ? decay_of<T>(p.a_neg[h], p.ag[r * p.ldag + c] + p.dt_bias[c]) : 0.f;
  }
  __syncthreads();
  // norms of q and k, their product: every warp computes them for itself
  float nq = 0.f, nkk = 0.f, dot = 0.f;
#pragma unroll
  for (int d = lane; d < 8 * RW; d += 32) {
    nq = fmaf(s_q[d], s_q[d], nq);
    nkk = fmaf(s_k[d], s_k[d], nkk);
    dot = fmaf(s_q[d], s_k[d], dot);
  }
  nq = warp_sum(nq);
  nkk = warp_sum(nkk);
  dot = warp_sum(dot);
  const float fq = 1.f / sqrtf(nq + 1e-6f) / sqrtf(static_cast<float>(p.dim)), fk = 1.f / sqrtf(nkk + 1e-6f);
  float4 ak = make_float4(0.f, 0.f, 0.f, 0.f), aq = ak;
#pragma unroll
  for (int j = 0; j < RW; ++j) {
    const int d = warp + 8 * j;
    const float g = s_g[d], k = s_k[d] * fk, q = s_q[d] * fq;
    S[j].x *= g; S[j].y *= g; S[j].z *= g; S[j].w *= g;
    ak.x = fmaf(S[j].x, k, ak.x); ak.y = fmaf(S[j].y, k, ak.y); ak.z = fmaf(S[j].z, k, ak.z); ak.w = fmaf(S[j].w, k, ak.w);
    aq.x = fmaf(S[j].x, q, aq.x); aq.y = fmaf(S[j].y, q, aq.y); aq.z = fmaf(S[j].z, q, aq.z); aq.w = fmaf(S[j].w, q, aq.w);
  }
  *reinterpret_cast<float4*>(&s_red[0][warp][vcol]) = ak;
  *reinterpret_cast<float4*>(&s_red[1][warp][vcol]) = aq;
  __syncthreads();
  float sk[4] = {}, sq[4] = {};
#pragma unroll
  for (int w = 0; w < 8; ++w) {
    const float4 a = *reinterpret_cast<const float4*>(&s_red[0][w][vcol]);
    const float4 c = *reinterpret_cast<const float4*>(&s_red[1][w][vcol]);
    sk[0] += a.x; sk[1] += a.y; sk[2] += a.z; sk[3] += a.w;
    sq[0] += c.x; sq[1] += c.y; sq[2] += c.z; sq[3] += c.w;
  }
  const float beta = sigmoid_f(act_load(p.proj + r * p.ldp + p.off_b + h));
  const float qk = dot * fq * fk;
  float u[4], o[4], ss = 0.f;
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    u[e] = vok ? beta * (s_v[vcol + e] - sk[e]) : 0.f;
    o[e] = vok ? fmaf(qk, u[e], sq[e]) : 0.f;
    ss = fmaf(o[e], o[e], ss);
  }
  if (sout >= 0 && vok) {
#pragma unroll
    for (int j = 0; j < RW; ++j) {
      const int d = warp + 8 * j;
      if (d < p.dim) {
        const float k = s_k[d] * fk;
        *reinterpret_cast<float4*>(p.state + sout * per_state + (static_cast<long long>(h) * p.dim + d) * p.vdim + vcol) =
            make_float4(fmaf(k, u[0], S[j].x), fmaf(k, u[1], S[j].y), fmaf(k, u[2], S[j].z), fmaf(k, u[3], S[j].w));
      }
    }
  }
  if (warp == 0) {
    ss = warp_sum(ss);
    const float inv = 1.f / sqrtf(ss / p.vdim + p.eps);
    if (vok) {
#pragma unroll
      for (int e = 0; e < 4; ++e)
        act_store(p.out + r * p.ldo + h * p.vdim + vcol + e,
                  o[e] * inv * p.norm_w[vcol + e] * output_gate(p, gate_pre(p, r, h * p.vdim + vcol + e)));
    }
  }
}

template <typename T>
static int fill(const FbDeltaArgs* a, DeltaParams<T>& p) {
  if (!a || !a->proj || (!a->ag && (a->off_a < 0 || a->off_g < 0)) || !a->conv || !a->a_neg || !a->dt_bias || !a->norm_w || !a->state || !a->seq_start ||
      !a->state_in || !a->state_out || !a->out)
    return FB_ERR_SHAPE;
  if (a->rows <= 0 || a->n_seqs <= 0 || a->heads <= 0 || a->kv_heads <= 0 || a->heads % a->kv_heads || a->dim <= 0 ||
      a->vdim <= 0 || a->taps <= 0 || a->n_states <= 0 || (a->taps > 1 && !a->tail))
    return FB_ERR_SHAPE;
  if (a->ldo < static_cast<long long>(a->heads) * a->vdim) return FB_ERR_SHAPE;
  p.proj = static_cast<const T*>(a->proj); p.ldp = a->ldp;
  p.off_q = a->off_q; p.off_k = a->off_k; p.off_v = a->off_v; p.off_b = a->off_b;
  p.ag = a->ag; p.ldag = a->ldag; p.off_gate = a->off_gate;
  p.off_a = a->off_a; p.off_g = a->off_g; p.gate_silu = a->gate_silu;
  p.conv = a->conv; p.a_neg = a->a_neg; p.dt_bias = a->dt_bias; p.norm_w = a->norm_w; p.eps = a->eps;
  p.state = a->state; p.tail = static_cast<T*>(a->tail); p.n_states = a->n_states;
  p.row_seq = a->row_seq; p.seq_start = a->seq_start; p.state_in = a->state_in; p.state_out = a->state_out;
  p.rows = a->rows; p.n_seqs = a->n_seqs; p.heads = a->heads; p.kv_heads = a->kv_heads; p.dim = a->dim; p.vdim = a->vdim;
  p.taps = a->taps;
  p.long_seqs = a->long_seqs;
  p.qn = a->qn; p.kn = a->kn; p.v = a->v; p.decay = a->decay; p.beta = a->beta; p.qk = a->qk; p.o = a->o;
  p.out = static_cast<T*>(a->out); p.ldo = a->ldo;
  p.status = static_cast<DeviceStatus*>(a->status);
  return FB_OK;
}

static int launched() { return cudaGetLastError() == cudaSuccess ? FB_OK : FB_ERR_LAUNCH; }

template <typename T>
static int run_decode(const FbDeltaArgs* a, cudaStream_t s) {
  DeltaParams<T> p{};
  const int rc = fill<T>(a, p);
  if (rc != FB_OK) return rc;
  if (p.vdim > 128 || p.vdim % 4 || p.dim > 128 || p.heads > 65535) return FB_ERR_SHAPE;
  const dim3 grid(p.n_seqs, p.heads);
  if (p.dim <= 64) launch_pdl(delta_decode_kernel<T, 8>, grid, dim3(256), 0, s, p);
  else launch_pdl(delta_decode_kernel<T, 16>, grid, dim3(256), 0, s, p);
  return launched();
}

template <typename T, int RPT, int COLS, bool HEADG>
static int launch_scan_cols(const DeltaParams<T>& p, cudaStream_t s) {
  constexpr int need = 2 * scan_buf<T, RPT, COLS, HEADG>() * static_cast<int>(sizeof(float));
  constexpr int whole_sm = 120 * 1024;                 // more than half of an SM's shared memory
  static bool attr = false;
  if (!attr) {
    if (cudaFuncSetAttribute(delta_scan_kernel<T, RPT, COLS, HEADG>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                             need > whole_sm ? need : whole_sm) != cudaSuccess)
      return FB_ERR_LAUNCH;
    attr = true;
  }
  // A mixed batch: few long sequences among decode rows.  The long ones' CTAs are bound by the latency of a token's chain
  // and must not share an SM with each other while there are SMs for all of them.
  const long long tiles = static_cast<long long>(p.heads) * ((p.vdim + 16 * COLS - 1) / (16 * COLS));
  const bool spread = p.long_seqs > 0 && p.long_seqs < p.n_seqs && p.long_seqs * tiles <= 148;
  const int smem = spread && need < whole_sm ? whole_sm : need;
  const dim3 grid(p.heads * ((p.vdim + 16 * COLS - 1) / (16 * COLS)), p.n_seqs);
  launch_pdl(delta_scan_kernel<T, RPT, COLS, HEADG>, grid, dim3(128), smem, s, p);
  return launched();
}

template <typename T, int RPT, bool HEADG>
static int launch_scan_form(const DeltaParams<T>& p, cudaStream_t s) {
  const long long per_col = static_cast<long long>(p.heads) * (p.long_seqs > 0 ? p.long_seqs : p.n_seqs);
  auto ctas = [&](int cols) { return per_col * ((p.vdim + 16 * cols - 1) / (16 * cols)); };
  if constexpr (RPT <= 16) {
    if (ctas(4) >= 120 && p.vdim > 32) return launch_scan_cols<T, RPT, 4, HEADG>(p, s);
  }
  if (ctas(2) >= 120 && p.vdim > 16) return launch_scan_cols<T, RPT, 2, HEADG>(p, s);
  return launch_scan_cols<T, RPT, 1, HEADG>(p, s);
}

template <typename T, int RPT>
static int launch_scan(const DeltaParams<T>& p, cudaStream_t s) {
  return p.off_a >= 0 ? launch_scan_form<T, RPT, true>(p, s) : launch_scan_form<T, RPT, false>(p, s);
}

template <typename T>
static int run_prefill(const FbDeltaArgs* a, cudaStream_t s) {
  DeltaParams<T> p{};
  int rc = fill<T>(a, p);
  if (rc != FB_OK) return rc;
  if (!p.row_seq || !p.qn || !p.kn || !p.v || !p.decay || !p.beta || !p.qk || !p.o) return FB_ERR_SHAPE;
  if (p.dim > 256 || p.n_seqs > 65535) return FB_ERR_SHAPE;
  const size_t smem = 2ull * p.kv_heads * p.dim * sizeof(float);
  if (smem > 200 * 1024) return FB_ERR_LIMIT;
  const bool vec = (p.kv_heads * p.dim) % 4 == 0 && (p.heads * p.vdim) % 4 == 0 && p.ldp % 4 == 0 && p.off_q % 4 == 0 &&
                   p.off_k % 4 == 0 && p.off_v % 4 == 0 && (reinterpret_cast<uintptr_t>(p.proj) & 15) == 0 &&
                   (reinterpret_cast<uintptr_t>(p.tail) & 15) == 0;
  auto prepare = vec ? delta_prepare_kernel<T, 4> : delta_prepare_kernel<T, 1>;
  static bool attr[2] = {false, false};
  if (!attr[vec]) {
    if (cudaFuncSetAttribute(prepare, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024) != cudaSuccess)
      return FB_ERR_LAUNCH;
    attr[vec] = true;
  }
  launch_pdl(prepare, dim3(p.rows), dim3(256), smem, s, p);
  if ((rc = launched()) != FB_OK) return rc;
  if (p.dim <= 32) rc = launch_scan<T, 4>(p, s);
  else if (p.dim <= 64) rc = launch_scan<T, 8>(p, s);
  else if (p.dim <= 128) rc = launch_scan<T, 16>(p, s);
  else rc = launch_scan<T, 32>(p, s);
  if (rc != FB_OK) return rc;
  const long long items = static_cast<long long>(p.rows) * p.heads;
  launch_pdl(delta_output_kernel<T>, dim3(static_cast<unsigned>((items + 3) / 4)), dim3(128), 0, s, p);
  return launched();
}

}  // namespace fb

using namespace fb;

extern "C" int fb_delta_decode(const FbDeltaArgs* a, void* stream) {
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (!a) return FB_ERR_SHAPE;
  return a->fp32 ? run_decode<float>(a, s) : run_decode<__nv_bfloat16>(a, s);
}

extern "C" int fb_delta_prefill(const FbDeltaArgs* a, void* stream) {
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (!a) return FB_ERR_SHAPE;
  return a->fp32 ? run_prefill<float>(a, s) : run_prefill<__nv_bfloat16>(a, s);
}
