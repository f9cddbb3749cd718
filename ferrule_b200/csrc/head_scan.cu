// Scan with one decay per head and a matrix state: for head h of group g, with d = softplus(dt_h + bias_h),
//
//     S <- exp(a_h d) S + d B_g x_h^T  (S is [state, vdim]);   y_h = S^T C_g + D_h x_h;   out_h = y_h * silu(z_h)
//
// B, C and x have passed the short convolution.  Step sizes, decays, state and sums are fp32.
//
// Prompts of bf16 models take the chunked form (head_scan_chunk.cu) where the sizes allow it.  Token by token, any mix of row
// counts: CTA = (columns of a head, head, sequence).  LPC lanes share VPL columns and hold SPL state rows of each in
// registers; sixteen tokens are staged at a time and the next ones requested before the staged ones are worked on.
// Sequences with one row (decode steps, and the single rows beside chunked prompts): CTA = (head, sequence), the
// state streams through registers once; its first part is requested before the dependency wait.
//
// State of a sequence: fp32 [heads, state, vdim].  Buffer `state_in[seq]` is read (-1: a new sequence, zeros), buffer
// `state_out[seq]` written (-1: nothing is kept), never the same one.
#include "act_type.cuh"
#include "common.cuh"
#include "f32x2.cuh"
#include "ferrule_b200.h"
#include "head_scan.cuh"
#include "launch.cuh"
#include "scan_math.cuh"

namespace fb {

constexpr int kHsThreads = 128;
constexpr int kHsTokens = 16;
constexpr int kHsRows = 8, kHsCols = 4;       // state rows and columns of a lane

template <typename T, int LPC>
__global__ void __launch_bounds__(kHsThreads)
head_scan_kernel(const HeadScanParams<T> p) {
  constexpr int CB = kHsThreads / LPC * kHsCols, NP = LPC * kHsRows, TS = kHsTokens, R = kHsRows, V = kHsCols;
  constexpr int kPx = TS * CB / kHsThreads, kBc = 2 * TS * NP / kHsThreads;
  __shared__ __align__(16) float s_b[TS][NP], s_c[TS][NP], s_u[TS][CB];
  __shared__ float s_x[TS][CB], s_y[TS][CB], s_a[TS], s_d[TS];
  const int tid = threadIdx.x, l = tid % LPC, cg = tid / LPC;
  // (a mixed batch lists its decode rows first: the long sequences' CTAs start first and spread over all SMs)
  const int seq = gridDim.z - 1 - blockIdx.z, h = blockIdx.y, c0 = blockIdx.x * CB, group = h / (p.heads / p.groups);
  int sin, sout;
  const bool ok = scan_bind(p, seq, sin, sout);
  const long long plane = static_cast<long long>(p.state) * p.vdim;
  const float* old = p.states + (static_cast<long long>(max(ok ? sin : 0, 0)) * p.heads + h) * plane;
  uint64_t S[V][R / 2];
#pragma unroll
  for (int v = 0; v < V; ++v)
#pragma unroll
    for (int j = 0; j < R / 2; ++j) {
      float s[2];
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int n = l * R + 2 * j + e, c = c0 + cg * V + v;
        s[e] = ok && sin >= 0 && n < p.state && c < p.vdim ? old[static_cast<long long>(n) * p.vdim + c] : 0.f;
      }
      S[v][j] = pack2(s[0], s[1]);
    }
  const float bias = p.dt_bias[h], rate = p.a_neg[h] * 1.4426950408889634f, skip = p.d_skip[h];
  pdl_wait();
  if (!ok) {
    if (tid == 0) report_status(p.status, kStatusBadIndex, 0xE50, seq, sout);
    return;
  }
  const int r0 = p.seq_start[seq], cnt_all = p.seq_start[seq + 1] - r0;
  if (r0 < 0 || cnt_all <= 0 || r0 + cnt_all > p.rows) {
    if (tid == 0) report_status(p.status, kStatusBadIndex, 0xE51, seq, r0);
    return;
  }
  const int pc = tid % CB, pt = tid / CB;                              // staging role: column pc of tokens pt, pt + 128 / CB, ...
  constexpr int kStep = kHsThreads / CB > 0 ? kHsThreads / CB : 1;
  const int col = min(c0 + pc, p.vdim - 1);
  // unconditional loads (addresses clamped): nothing between the request and the work on the current tokens depends on them
  T fx[kPx], fz[kPx], fz_next[kPx], fbc[kBc], fd;
  auto fetch = [&](int t0) {
    const int cnt = min(TS, cnt_all - t0);
#pragma unroll
    for (int k = 0; k < kPx; ++k) {
      const long long r = r0 + t0 + min(pt + k * kStep, cnt - 1);
      fx[k] = __ldg(p.xbc + r * p.ldx + h * p.vdim + col);
      fz_next[k] = __ldg(p.z + r * p.ldp + h * p.vdim + col);
    }
#pragma unroll
    for (int k = 0; k < kBc; ++k) {
      const int i = tid + k * kHsThreads, t = i / (2 * NP), n = i % (2 * NP), m = min(n % NP, p.state - 1);
      fbc[k] = __ldg(p.xbc + (r0 + t0 + min(t, cnt - 1)) * p.ldx + (n < NP ? p.off_b : p.off_c) + group * p.state + m);
    }
    fd = __ldg(p.dt + (r0 + t0 + min(tid % TS, cnt - 1)) * p.ldp + h);
  };
  fetch(0);
  for (int t0 = 0; t0 < cnt_all; t0 += TS) {
    const int cnt = min(TS, cnt_all - t0);
    if (tid < TS) {
      const float d = tid < cnt ? scan_softplus<T>(act_load(&fd) + bias) : 0.f;      // a step of size zero changes nothing
      s_d[tid] = d;
      s_a[tid] = scan_exp2<T>(rate * d);
    }
#pragma unroll
    for (int k = 0; k < kBc; ++k) {
      const int i = tid + k * kHsThreads, t = i / (2 * NP), n = i % (2 * NP);
      (n < NP ? s_b[t][n] : s_c[t][n - NP]) = n % NP < p.state ? act_load(&fbc[k]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kPx; ++k) {
      const int t = pt + k * kStep;
      const float x = act_load(&fx[k]);
      s_x[t][pc] = x;
      s_u[t][pc] = s_d[t] * x;
      fz[k] = fz_next[k];
    }
    __syncthreads();
    if (t0 + TS < cnt_all) fetch(t0 + TS);
#pragma unroll 2
    for (int t = 0; t < cnt; ++t) {
      const float4 u = *reinterpret_cast<const float4*>(&s_u[t][cg * V]);
      const float uv[4] = {u.x, u.y, u.z, u.w};
      const uint64_t a2 = pack2(s_a[t], s_a[t]);
      uint64_t b[R / 2], c[R / 2];
#pragma unroll
      for (int j = 0; j < R / 2; ++j) {
        b[j] = *reinterpret_cast<const uint64_t*>(&s_b[t][l * R + 2 * j]);
        c[j] = *reinterpret_cast<const uint64_t*>(&s_c[t][l * R + 2 * j]);
      }
      float y[V];
#pragma unroll
      for (int v = 0; v < V; ++v) {
        const uint64_t u2 = pack2(uv[v], uv[v]);
        uint64_t acc = 0;
#pragma unroll
        for (int j = 0; j < R / 2; ++j) {
          S[v][j] = fma2(a2, S[v][j], mul2(u2, b[j]));
          acc = fma2(S[v][j], c[j], acc);
        }
        float lo, hi;
        unpack2(acc, lo, hi);
        y[v] = lo + hi;
      }
      // four sums over the lanes of a column group at once: lane l of the first four ends up with column l
      const bool b0 = l & 1, b1 = l & 2;
      float k0 = b0 ? y[1] : y[0], k1 = b0 ? y[3] : y[2];
      k0 += __shfl_xor_sync(0xffffffffu, b0 ? y[0] : y[1], 1);
      k1 += __shfl_xor_sync(0xffffffffu, b0 ? y[2] : y[3], 1);
      float w = b1 ? k1 : k0;
      w += __shfl_xor_sync(0xffffffffu, b1 ? k0 : k1, 2);
#pragma unroll
      for (int o = 4; o < LPC; o <<= 1) w += __shfl_xor_sync(0xffffffffu, w, o);
      if (LPC == 4 || l < 4) s_y[t][cg * V + (l & 3)] = w;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kPx; ++k) {
      const int t = pt + k * kStep;
      if (t < cnt && c0 + pc < p.vdim)
        act_store(p.out + (r0 + t0 + t) * p.ldo + h * p.vdim + c0 + pc,
                  fmaf(skip, s_x[t][pc], s_y[t][pc]) * scan_silu<T>(act_load(&fz[k])));
    }
    // the last columns of an output row are padding
    if (h == p.heads - 1 && blockIdx.x == 0)
      for (int i = tid; i < cnt * (p.out_cols - p.heads * p.vdim); i += kHsThreads) {
        const int pad = p.out_cols - p.heads * p.vdim;
        act_store(p.out + (r0 + t0 + i / pad) * p.ldo + p.heads * p.vdim + i % pad, 0.f);
      }
  }
  pdl_launch_dependents();
  if (sout < 0) return;
  float* dst = p.states + (static_cast<long long>(sout) * p.heads + h) * plane;
#pragma unroll
  for (int v = 0; v < V; ++v)
#pragma unroll
    for (int j = 0; j < R / 2; ++j) {
      float s[2];
      unpack2(S[v][j], s[0], s[1]);
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int n = l * R + 2 * j + e, c = c0 + cg * V + v;
        if (n < p.state && c < p.vdim) dst[static_cast<long long>(n) * p.vdim + c] = s[e];
      }
    }
}

constexpr int kHsStepThreads = 256;
constexpr int kHsStepRows = 8;       // state rows of a thread requested at a time

// four consecutive columns, of which `n` exist; vec: 16-byte aligned and all four exist
__device__ __forceinline__ float4 load_cols(const float* p, int n, bool vec) {
  if (vec) return *reinterpret_cast<const float4*>(p);
  return make_float4(n > 0 ? p[0] : 0.f, n > 1 ? p[1] : 0.f, n > 2 ? p[2] : 0.f, n > 3 ? p[3] : 0.f);
}
__device__ __forceinline__ void store_cols(float* p, int n, bool vec, const float4& v) {
  if (vec) {
    *reinterpret_cast<float4*>(p) = v;
    return;
  }
  if (n > 0) p[0] = v.x;
  if (n > 1) p[1] = v.y;
  if (n > 2) p[2] = v.z;
  if (n > 3) p[3] = v.w;
}

template <typename T>
__global__ void __launch_bounds__(kHsStepThreads)
head_scan_step_kernel(const HeadScanParams<T> p) {
  pdl_launch_dependents();
  extern __shared__ __align__(16) float hs_sm[];                       // [state] B, [state] C, [vdim] x, [row groups][quads * 4] partial sums
  const int h = blockIdx.x, seq = blockIdx.y, tid = threadIdx.x, group = h / (p.heads / p.groups);
  const int quads = (p.vdim + 3) / 4, lanes = min(quads, kHsStepThreads), n_groups = kHsStepThreads / lanes;
  const int n_pad = (p.state + 3) / 4 * 4;               // 16-byte alignment of what follows
  float* s_b = hs_sm;
  float* s_c = s_b + n_pad;
  float* s_x = s_c + n_pad;
  float* s_y = s_x + (p.vdim + 3) / 4 * 4;
  int sin, sout;
  const bool ok = scan_bind(p, seq, sin, sout);
  const long long plane = static_cast<long long>(p.state) * p.vdim;
  const float* old = p.states + (static_cast<long long>(max(ok ? sin : 0, 0)) * p.heads + h) * plane;
  float* dst = p.states + (static_cast<long long>(max(ok ? sout : 0, 0)) * p.heads + h) * plane;
  const int q = tid % lanes, ng = tid / lanes;
  const bool active = ng < n_groups, vec = p.vdim % 4 == 0;
  float4 S[kHsStepRows];
  auto request = [&](int n0, int c, int left) {
#pragma unroll
    for (int j = 0; j < kHsStepRows; ++j) {
      const int n = min(n0 + j * n_groups, p.state - 1);
      S[j] = load_cols(old + static_cast<long long>(n) * p.vdim + c, left, vec);
    }
  };
  if (active) request(ng, q * 4, p.vdim - q * 4);
  const float bias = p.dt_bias[h], rate = p.a_neg[h] * 1.4426950408889634f, skip = p.d_skip[h];
  pdl_wait();
  const int r = p.seq_start[seq];
  if (ok && r >= 0 && p.seq_start[seq + 1] > r + 1 && p.skip_single) return;     // beside a chunked launch: not a single row
  if (!ok || r < 0 || r >= p.rows || p.seq_start[seq + 1] != r + 1) {
    if (tid == 0) report_status(p.status, kStatusBadIndex, 0xE52, seq, r);
    return;
  }
  const T* row = p.xbc + r * p.ldx;
  for (int i = tid; i < p.state; i += kHsStepThreads) {
    s_b[i] = act_load(row + p.off_b + group * p.state + i);
    s_c[i] = act_load(row + p.off_c + group * p.state + i);
  }
  for (int i = tid; i < p.vdim; i += kHsStepThreads) s_x[i] = act_load(row + h * p.vdim + i);
  const float d = scan_softplus<T>(act_load(p.dt + r * p.ldp + h) + bias), a = scan_exp2<T>(rate * d);
  __syncthreads();
  if (active)
    for (int qq = q; qq < quads; qq += lanes) {
      const int c = qq * 4, left = p.vdim - c;
      if (qq != q) request(ng, c, left);
      float4 u = make_float4(0.f, 0.f, 0.f, 0.f), y = u;
      u.x = d * s_x[c];
      if (left > 1) u.y = d * s_x[c + 1];
      if (left > 2) u.z = d * s_x[c + 2];
      if (left > 3) u.w = d * s_x[c + 3];
      for (int n0 = ng; n0 < p.state; n0 += kHsStepRows * n_groups) {
        if (n0 != ng) request(n0, c, left);
#pragma unroll
        for (int j = 0; j < kHsStepRows; ++j) {
          const int n = n0 + j * n_groups;
          if (n >= p.state) break;
          const float b = s_b[n], cc = s_c[n], f = sin >= 0 ? a : 0.f;
          float4 s;
          s.x = sin >= 0 ? fmaf(f, S[j].x, u.x * b) : u.x * b;
          s.y = sin >= 0 ? fmaf(f, S[j].y, u.y * b) : u.y * b;
          s.z = sin >= 0 ? fmaf(f, S[j].z, u.z * b) : u.z * b;
          s.w = sin >= 0 ? fmaf(f, S[j].w, u.w * b) : u.w * b;
          y.x = fmaf(s.x, cc, y.x);
          y.y = fmaf(s.y, cc, y.y);
          y.z = fmaf(s.z, cc, y.z);
          y.w = fmaf(s.w, cc, y.w);
          if (sout >= 0) store_cols(dst + static_cast<long long>(n) * p.vdim + c, left, vec, s);
        }
      }
      *reinterpret_cast<float4*>(s_y + (static_cast<size_t>(ng) * quads + qq) * 4) = y;
    }
  __syncthreads();
  for (int v = tid; v < p.vdim; v += kHsStepThreads) {
    float y = 0.f;
    for (int g = 0; g < n_groups; ++g) y += s_y[static_cast<size_t>(g) * quads * 4 + v];
    act_store(p.out + r * p.ldo + h * p.vdim + v,
              fmaf(skip, s_x[v], y) * scan_silu<T>(act_load(p.z + r * p.ldp + h * p.vdim + v)));
  }
  if (h == p.heads - 1)
    for (int i = p.heads * p.vdim + tid; i < p.out_cols; i += kHsStepThreads) act_store(p.out + r * p.ldo + i, 0.f);
}

template <typename T, int LPC>
static int launch_head_scan(const HeadScanParams<T>& p, cudaStream_t s) {
  constexpr int CB = kHsThreads / LPC * kHsCols;
  launch_pdl(head_scan_kernel<T, LPC>, dim3((p.vdim + CB - 1) / CB, p.heads, p.n_seqs), dim3(kHsThreads), 0, s, p);
  return cudaGetLastError() == cudaSuccess ? FB_OK : FB_ERR_LAUNCH;
}

template <typename T>
static int launch_step(const HeadScanParams<T>& p, cudaStream_t s) {
  const int quads = (p.vdim + 3) / 4, lanes = quads < kHsStepThreads ? quads : kHsStepThreads;
  const size_t smem = (2 * static_cast<size_t>((p.state + 3) / 4 * 4) + quads * 4 + static_cast<size_t>(kHsStepThreads / lanes) * quads * 4) * sizeof(float);
  if (smem > 48 * 1024) return FB_ERR_LIMIT;
  launch_pdl(head_scan_step_kernel<T>, dim3(p.heads, p.n_seqs), dim3(kHsStepThreads), smem, s, p);
  return cudaGetLastError() == cudaSuccess ? FB_OK : FB_ERR_LAUNCH;
}

template <typename T>
static int run_head_scan(const FbHeadScanArgs* a, cudaStream_t s) {
  HeadScanParams<T> p{};
  p.xbc = static_cast<const T*>(a->xbc); p.ldx = a->ldx; p.off_b = a->off_b; p.off_c = a->off_c;
  p.dt = static_cast<const T*>(a->dt); p.z = static_cast<const T*>(a->z); p.ldp = a->ldp;
  p.dt_bias = a->dt_bias; p.a_neg = a->a_neg; p.d_skip = a->d_skip; p.states = a->states;
  p.seq_start = a->seq_start; p.state_in = a->state_in; p.state_out = a->state_out;
  p.out = static_cast<T*>(a->out); p.ldo = a->ldo;
  p.rows = a->rows; p.n_seqs = a->n_seqs; p.heads = a->heads; p.vdim = a->vdim; p.state = a->state; p.groups = a->groups;
  p.n_states = a->n_states;
  p.out_cols = (a->heads * a->vdim + 7) / 8 * 8;
  p.status = static_cast<DeviceStatus*>(a->status);
  if (p.n_seqs == p.rows) return launch_step<T>(p, s);
  if constexpr (sizeof(T) == 2) {
    if (!a->by_token && head_scan_chunk_ok(p.vdim, p.state, p.groups)) {
      p.skip_single = a->long_seqs != p.n_seqs;
      if (p.skip_single) {
        const int rc = launch_step<T>(p, s);
        if (rc != FB_OK) return rc;
      }
      return run_head_scan_chunk(p, s);
    }
  }
  if (p.state <= 32) return launch_head_scan<T, 4>(p, s);
  if (p.state <= 64) return launch_head_scan<T, 8>(p, s);
  if (p.state <= 128) return launch_head_scan<T, 16>(p, s);
  return launch_head_scan<T, 32>(p, s);
}

}  // namespace fb

using namespace fb;

extern "C" int fb_head_scan(const FbHeadScanArgs* a, void* stream) {
  if (!a || !a->xbc || !a->dt || !a->z || !a->dt_bias || !a->a_neg || !a->d_skip || !a->states || !a->seq_start || !a->state_in ||
      !a->state_out || !a->out)
    return FB_ERR_SHAPE;
  if (a->rows <= 0 || a->n_seqs <= 0 || a->n_seqs > 65535 || a->heads <= 0 || a->heads > 65535 || a->vdim <= 0 || a->state <= 0 ||
      a->groups <= 0 || a->heads % a->groups || a->n_states <= 0)
    return FB_ERR_SHAPE;
  if (a->state > 256 || a->vdim > 1024) return FB_ERR_LIMIT;
  const long long inner = static_cast<long long>(a->heads) * a->vdim, bc = static_cast<long long>(a->groups) * a->state;
  if (a->ldo < (inner + 7) / 8 * 8 || a->off_b < inner || a->off_c < 0 || a->ldx < a->off_b + bc || a->ldx < a->off_c + bc ||
      a->ldp < inner)
    return FB_ERR_SHAPE;
  if (reinterpret_cast<uintptr_t>(a->states) & 15) return FB_ERR_ALIGN;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  return a->fp32 ? run_head_scan<float>(a, s) : run_head_scan<__nv_bfloat16>(a, s);
}
