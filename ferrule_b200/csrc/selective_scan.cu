// Selective scan: a diagonal recurrence per channel c and state n, with the token's own step size, input and read-out:
//
//     d = softplus(dt_c + bias_c);   S[c, n] <- exp(d A[c, n]) S[c, n] + d x_c B_n;   y_c = sum_n S[c, n] C_n + D_c x_c
//     out_c = y_c * silu(z_c)
//
// Any mix of row counts: CTA = (128 / LPC channels) x sequence, LPC lanes share a channel and hold SPL states each in
// registers.  Tokens are staged sixteen at a time; the next ones are requested before the staged ones
// are worked on.  The exponentials do not depend on the state, so a token's chain is one multiply-add per state.
// Decode steps (one row per sequence): a thread owns a channel, nothing is shared; states are requested before the
// dependency wait.
//
// State of a sequence: fp32 [state, inner], channels innermost.  Buffer `state_in[seq]` is read (-1: a new sequence,
// zeros), buffer `state_out[seq]` written (-1: nothing is kept), never the same one.
#include "act_type.cuh"
#include "common.cuh"
#include "f32x2.cuh"
#include "ferrule_b200.h"
#include "launch.cuh"
#include "scan_math.cuh"

namespace fb {

constexpr int kScanThreads = 128;
constexpr int kScanTokens = 16;

template <typename T>
struct ScanParams {
  const T* x;
  long long ldx;
  const T* z;
  long long ldz;
  const T* bc;
  long long ldbc;
  int off_b, off_c;
  const float* dt;
  long long lddt;
  const float* dt_bias;
  const float* a_log2;
  const float* d_skip;
  float* states;
  const int* seq_start;
  const int* state_in;
  const int* state_out;
  T* out;
  long long ldo;
  int rows, n_seqs, inner, state, n_states;
  DeviceStatus* status;
};

// SPL states of a lane times one token: S <- exp2(d a) S + u B, returns this lane's share of S . C
template <typename T, int SPL>
__device__ __forceinline__ float scan_token(uint64_t (&S)[SPL / 2], const uint64_t (&a2)[SPL / 2], float2 du, const float* b,
                                            const float* c) {
  const uint64_t d2 = pack2(du.x, du.x), u2 = pack2(du.y, du.y);
  uint64_t y = 0;
#pragma unroll
  for (int j = 0; j < SPL / 2; ++j) {
    float e0, e1;
    unpack2(mul2(d2, a2[j]), e0, e1);
    S[j] = fma2(pack2(scan_exp2<T>(e0), scan_exp2<T>(e1)), S[j], mul2(u2, *reinterpret_cast<const uint64_t*>(b + 2 * j)));
    y = fma2(S[j], *reinterpret_cast<const uint64_t*>(c + 2 * j), y);
  }
  float y0, y1;
  unpack2(y, y0, y1);
  return y0 + y1;
}

template <typename T, int LPC, int SPL>
__global__ void __launch_bounds__(kScanThreads)
selective_scan_kernel(const ScanParams<T> p) {
  constexpr int CH = kScanThreads / LPC, NP = LPC * SPL, TS = kScanTokens;
  constexpr int kPf = TS * CH / kScanThreads;                        // staged (token, channel) pairs per thread
  constexpr int kBc = (2 * TS * NP + kScanThreads - 1) / kScanThreads;
  static_assert(LPC >= 4 && SPL % 2 == 0, "four tokens share one reduction");
  __shared__ float2 s_du[TS][CH];                                    // step size, step size times input
  __shared__ float s_x[TS][CH], s_y[TS][CH];
  __shared__ __align__(16) float s_b[TS][NP], s_c[TS][NP];
  const int tid = threadIdx.x, l = tid % LPC, ch = tid / LPC;
  // (a mixed batch lists its decode rows first: the long sequences' CTAs start first and spread over all SMs)
  const int seq = gridDim.y - 1 - blockIdx.y, c0 = blockIdx.x * CH, c = c0 + ch;
  const int sin = p.state_in[seq], sout = p.state_out[seq];
  const bool ok = sin < p.n_states && sout < p.n_states && !(sin >= 0 && sin == sout);
  const bool cin = c < p.inner;
  uint64_t a2[SPL / 2], S[SPL / 2];
#pragma unroll
  for (int j = 0; j < SPL / 2; ++j) {
    float av[2], sv[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int n = l * SPL + 2 * j + e;
      const bool in = cin && n < p.state;
      av[e] = in ? p.a_log2[static_cast<long long>(n) * p.inner + c] : 0.f;
      sv[e] = in && ok && sin >= 0 ? p.states[(static_cast<long long>(sin) * p.state + n) * p.inner + c] : 0.f;
    }
    a2[j] = pack2(av[0], av[1]);
    S[j] = pack2(sv[0], sv[1]);
  }
  // staging role of this thread: channel `pc` of tokens pt, pt + 128 / CH, ...
  const int pc = tid % CH, pt = tid / CH;
  constexpr int kStep = kScanThreads / CH;
  const bool pin = c0 + pc < p.inner;
  const float bias = pin ? p.dt_bias[c0 + pc] : 0.f, skip = pin ? p.d_skip[c0 + pc] : 0.f;
  pdl_wait();
  if (!ok) {
    if (tid == 0) report_status(p.status, kStatusBadIndex, 0xD40, seq, sout);
    return;
  }
  const int r0 = p.seq_start[seq], cnt_all = p.seq_start[seq + 1] - r0;
  if (r0 < 0 || cnt_all <= 0 || r0 + cnt_all > p.rows) {
    if (tid == 0) report_status(p.status, kStatusBadIndex, 0xD41, seq, r0);
    return;
  }
  // The loads of the next tokens are unconditional (addresses clamped) and their conversion waits until they are staged:
  // nothing between the request and the work on the current tokens depends on them.
  float fd[kPf];
  T fx[kPf], fz[kPf], fz_next[kPf], fbc[kBc];
  const int pcc = min(c0 + pc, p.inner - 1);
  auto fetch = [&](int t0) {
    const int cnt = min(TS, cnt_all - t0);
#pragma unroll
    for (int k = 0; k < kPf; ++k) {
      const int t = pt + k * kStep;
      const long long r = r0 + t0 + min(t, cnt - 1);
      fd[k] = __ldg(p.dt + r * p.lddt + pcc);
      fx[k] = __ldg(p.x + r * p.ldx + pcc);
      fz_next[k] = __ldg(p.z + r * p.ldz + pcc);
    }
#pragma unroll
    for (int k = 0; k < kBc; ++k) {
      const int i = tid + k * kScanThreads, t = i / (2 * NP), n = i % (2 * NP), m = n % NP;
      fbc[k] = __ldg(p.bc + (r0 + t0 + min(t, cnt - 1)) * p.ldbc + (n < NP ? p.off_b : p.off_c) + min(m, p.state - 1));
    }
  };
  fetch(0);
  for (int t0 = 0; t0 < cnt_all; t0 += TS) {
    const int cnt = min(TS, cnt_all - t0);
#pragma unroll
    for (int k = 0; k < kPf; ++k) {
      const int t = pt + k * kStep;
      const float d = t < cnt ? scan_softplus<T>(fd[k] + bias) : 0.f;    // a step of size zero changes nothing
      const float x = act_load(&fx[k]);
      s_du[t][pc] = make_float2(d, d * x);
      s_x[t][pc] = x;
      fz[k] = fz_next[k];
    }
#pragma unroll
    for (int k = 0; k < kBc; ++k) {
      const int i = tid + k * kScanThreads, t = i / (2 * NP), n = i % (2 * NP);
      // (padding states have a decay of one and start at zero: their input must be zero)
      if (t < TS) (n < NP ? s_b[t][n] : s_c[t][n - NP]) = n % NP < p.state ? act_load(&fbc[k]) : 0.f;
    }
    __syncthreads();
    if (t0 + TS < cnt_all) fetch(t0 + TS);
    if (cnt == 1) {
      float y = scan_token<T, SPL>(S, a2, s_du[0][ch], &s_b[0][l * SPL], &s_c[0][l * SPL]);
#pragma unroll
      for (int o = 1; o < LPC; o <<= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
      if (l == 0) s_y[0][ch] = y;
    } else {
#pragma unroll 1
      for (int t = 0; t < cnt; t += 4) {
        float y[4];
#pragma unroll
        for (int q = 0; q < 4; ++q)
          y[q] = scan_token<T, SPL>(S, a2, s_du[t + q][ch], &s_b[t + q][l * SPL], &s_c[t + q][l * SPL]);
        // four sums over the channel's lanes at once: lane l of the first four ends up with token t + l
        const bool b0 = l & 1, b1 = l & 2;
        float k0 = b0 ? y[1] : y[0], k1 = b0 ? y[3] : y[2];
        k0 += __shfl_xor_sync(0xffffffffu, b0 ? y[0] : y[1], 1);
        k1 += __shfl_xor_sync(0xffffffffu, b0 ? y[2] : y[3], 1);
        float v = b1 ? k1 : k0;
        v += __shfl_xor_sync(0xffffffffu, b1 ? k0 : k1, 2);
#pragma unroll
        for (int o = 4; o < LPC; o <<= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
        if (LPC == 4 || l < 4) s_y[t + (l & 3)][ch] = v;
      }
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kPf; ++k) {
      const int t = pt + k * kStep;
      if (t < cnt && pin)
        act_store(p.out + (r0 + t0 + t) * p.ldo + c0 + pc, fmaf(skip, s_x[t][pc], s_y[t][pc]) * scan_silu<T>(act_load(&fz[k])));
    }
    // the next round overwrites this thread's own s_du / s_x entries and s_b / s_c, last read before the barrier above;
    // s_y is written again behind the next barrier
  }
  pdl_launch_dependents();
  if (sout >= 0 && cin) {
#pragma unroll
    for (int j = 0; j < SPL / 2; ++j) {
      float sv[2];
      unpack2(S[j], sv[0], sv[1]);
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int n = l * SPL + 2 * j + e;
        if (n < p.state) p.states[(static_cast<long long>(sout) * p.state + n) * p.inner + c] = sv[e];
      }
    }
  }
}

constexpr int kStepStates = 16;      // states requested at a time

template <typename T>
__global__ void __launch_bounds__(128)
selective_step_kernel(const ScanParams<T> p) {
  pdl_launch_dependents();
  const int seq = blockIdx.y, c = blockIdx.x * blockDim.x + threadIdx.x;
  const int sin = p.state_in[seq], sout = p.state_out[seq];
  const bool ok = sin < p.n_states && sout < p.n_states && !(sin >= 0 && sin == sout);
  const int cc = min(c, p.inner - 1);
  const float* old = p.states + static_cast<long long>(max(ok ? sin : 0, 0)) * p.state * p.inner + cc;
  float S[kStepStates], a[kStepStates];
  auto request = [&](int n0) {
#pragma unroll
    for (int j = 0; j < kStepStates; ++j) {
      const long long n = min(n0 + j, p.state - 1);
      a[j] = p.a_log2[n * p.inner + cc];
      S[j] = old[n * p.inner];
    }
  };
  request(0);
  const float bias = p.dt_bias[cc], skip = p.d_skip[cc];
  pdl_wait();
  const int r = p.seq_start[seq];
  if (!ok || r < 0 || r >= p.rows || p.seq_start[seq + 1] != r + 1) {
    if (threadIdx.x == 0) report_status(p.status, kStatusBadIndex, 0xD42, seq, r);
    return;
  }
  const float x = act_load(p.x + r * p.ldx + cc), z = act_load(p.z + r * p.ldz + cc);
  const float d = scan_softplus<T>(p.dt[r * p.lddt + cc] + bias), u = d * x;
  const T* row = p.bc + r * p.ldbc;
  float* dst = p.states + static_cast<long long>(max(sout, 0)) * p.state * p.inner + cc;
  float y = 0.f;
  for (int n0 = 0; n0 < p.state; n0 += kStepStates) {
    if (n0 > 0) request(n0);
#pragma unroll
    for (int j = 0; j < kStepStates; ++j) {
      const int n = n0 + j;
      if (n < p.state) {
        const float s = fmaf(scan_exp2<T>(d * a[j]), sin >= 0 ? S[j] : 0.f, u * act_load(row + p.off_b + n));
        y = fmaf(s, act_load(row + p.off_c + n), y);
        if (sout >= 0 && c < p.inner) dst[static_cast<long long>(n) * p.inner] = s;
      }
    }
  }
  if (c < p.inner) act_store(p.out + r * p.ldo + c, fmaf(skip, x, y) * scan_silu<T>(z));
}

template <typename T, int LPC, int SPL>
static int launch_scan_form(const ScanParams<T>& p, cudaStream_t s) {
  constexpr int CH = kScanThreads / LPC;
  launch_pdl(selective_scan_kernel<T, LPC, SPL>, dim3((p.inner + CH - 1) / CH, p.n_seqs), dim3(kScanThreads), 0, s, p);
  return cudaGetLastError() == cudaSuccess ? FB_OK : FB_ERR_LAUNCH;
}

template <typename T>
static int run_scan(const FbScanArgs* a, cudaStream_t s) {
  ScanParams<T> p{};
  p.x = static_cast<const T*>(a->x); p.ldx = a->ldx;
  p.z = static_cast<const T*>(a->z); p.ldz = a->ldz;
  p.bc = static_cast<const T*>(a->bc); p.ldbc = a->ldbc; p.off_b = a->off_b; p.off_c = a->off_c;
  p.dt = a->dt; p.lddt = a->lddt; p.dt_bias = a->dt_bias; p.a_log2 = a->a_log2; p.d_skip = a->d_skip;
  p.states = a->states; p.seq_start = a->seq_start; p.state_in = a->state_in; p.state_out = a->state_out;
  p.out = static_cast<T*>(a->out); p.ldo = a->ldo;
  p.rows = a->rows; p.n_seqs = a->n_seqs; p.inner = a->inner; p.state = a->state; p.n_states = a->n_states;
  p.status = static_cast<DeviceStatus*>(a->status);
  if (p.n_seqs == p.rows) {
    launch_pdl(selective_step_kernel<T>, dim3((p.inner + 127) / 128, p.n_seqs), dim3(128), 0, s, p);
    return cudaGetLastError() == cudaSuccess ? FB_OK : FB_ERR_LAUNCH;
  }
  if (p.state <= 8) return launch_scan_form<T, 4, 2>(p, s);
  if (p.state <= 16) return launch_scan_form<T, 4, 4>(p, s);
  if (p.state <= 32) return launch_scan_form<T, 4, 8>(p, s);
  if (p.state <= 64) return launch_scan_form<T, 8, 8>(p, s);
  return launch_scan_form<T, 16, 8>(p, s);
}

}  // namespace fb

using namespace fb;

extern "C" int fb_selective_scan(const FbScanArgs* a, void* stream) {
  if (!a || !a->x || !a->z || !a->bc || !a->dt || !a->dt_bias || !a->a_log2 || !a->d_skip || !a->states || !a->seq_start ||
      !a->state_in || !a->state_out || !a->out)
    return FB_ERR_SHAPE;
  if (a->rows <= 0 || a->n_seqs <= 0 || a->n_seqs > 65535 || a->inner <= 0 || a->state <= 0 || a->n_states <= 0)
    return FB_ERR_SHAPE;
  if (a->state > 128) return FB_ERR_LIMIT;
  if (a->ldx < a->inner || a->ldz < a->inner || a->lddt < a->inner || a->ldo < a->inner || a->off_b < 0 || a->off_c < 0 ||
      a->ldbc < a->off_b + a->state || a->ldbc < a->off_c + a->state)
    return FB_ERR_SHAPE;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  return a->fp32 ? run_scan<float>(a, s) : run_scan<__nv_bfloat16>(a, s);
}
