// Head-decay scan (head_scan.cu) of prompts in chunks of 64 tokens on tensor cores, bf16 inputs.
//
// With L_t the sum of the decays' logarithms up to token t of the chunk and S the state before it,
//
//     y_t = exp(L_t) C_t S + sum_{j <= t} (C_t . B_j) exp(L_t - L_j) d_j x_j,
//     S  <- exp(L_end) S + sum_j exp(L_end - L_j) d_j B_j x_j^T
//
// are matrix products over bf16 inputs (B, C, x as the convolution wrote them) and fp32 factors.  Every fp32 factor enters as
// the sum of two bf16 numbers (error 2^-17 of its size), accumulators and the state are fp32.
//
// CTA = (64 columns of a head, head, sequence), four warps with 16 columns each.  A warp keeps the transposed state of its
// columns as MMA accumulators: their layout is that of the B operand of C S.  Per chunk: the warps compute the masked and
// decayed products P of C and B together (16 rows each, two bf16 parts in shared memory), then every warp its columns of y and
// of the state.  L is summed in double and kept as two floats: behind a strong decay it is large, its differences may be small.  The
// next chunk's rows are copied while this one is worked on.  A 64-token chunk of a head is too small for the 128-row tiles of
// tcgen05, and the accumulators feed the next product from registers: warp-level MMA.
#include "act_type.cuh"
#include "common.cuh"
#include "head_scan.cuh"
#include "launch.cuh"
#include "ferrule_b200.h"
#include "mma_sync.cuh"
#include "scan_math.cuh"

namespace fb {

constexpr int kHcThreads = 128;
constexpr int kHcTokens = 64;
constexpr int kHcCols = 64;

template <int NP>
struct HcCfg {
  static constexpr int kPitchN = NP + 8, kPitchV = kHcCols + 8, kPitchP = kHcTokens + 8;   // conflict-free ldmatrix
  static constexpr int kB = 0, kC = kHcTokens * kPitchN, kX = 2 * kHcTokens * kPitchN;
  static constexpr int kStage = kX + kHcTokens * kPitchV;                                  // bf16 elements
  static constexpr int kP = 2 * kStage, kEnd = kP + 2 * kHcTokens * kPitchP;
  static constexpr int kSmem = kEnd * 2 + 2 * 5 * kHcTokens * 4;
};

// 16 bytes global -> shared; bytes past `valid` are zeros
__device__ __forceinline__ void hc_copy16(void* dst, const void* src, int valid) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(dst)), "l"(src), "r"(valid) : "memory");
}

// a pair of fp32 numbers as the sum of two pairs of bf16 numbers
__device__ __forceinline__ void two_parts(float a, float b, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  const float2 f = __bfloat1622float2(h);
  const __nv_bfloat162 l = __floats2bfloat162_rn(a - f.x, b - f.y);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = *reinterpret_cast<const uint32_t*>(&l);
}

template <int NP>
__global__ void __launch_bounds__(kHcThreads)
head_scan_chunk_kernel(const HeadScanParams<__nv_bfloat16> p) {
  using C = HcCfg<NP>;
  extern __shared__ __align__(128) uint8_t hc_smem[];
  __nv_bfloat16* sm = reinterpret_cast<__nv_bfloat16*>(hc_smem);
  float* factors = reinterpret_cast<float*>(hc_smem + C::kEnd * 2);        // [2][L | its rest | exp L | d | exp(L_end - L) d][64]
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g4 = lane >> 2, t4 = lane & 3;
  const int lrow = lane & 7, lmat = lane >> 3;
  const int seq = gridDim.z - 1 - blockIdx.z, h = blockIdx.y, c0 = blockIdx.x * kHcCols, group = h / (p.heads / p.groups);
  int sin, sout;
  const bool ok = scan_bind(p, seq, sin, sout);
  const long long plane = static_cast<long long>(p.state) * p.vdim;
  const int v0 = c0 + warp * 16;                                           // first column of this warp
  const bool mine = v0 < p.vdim;
  // transposed state: tile n holds states 8 n + 2 t4, + 1 of columns v0 + g4 and v0 + g4 + 8
  float S[NP / 8][4];
  {
    const float* old = p.states + (static_cast<long long>(max(ok ? sin : 0, 0)) * p.heads + h) * plane;
#pragma unroll
    for (int n = 0; n < NP / 8; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int s = n * 8 + t4 * 2 + (e & 1), v = v0 + g4 + (e >> 1) * 8;
        S[n][e] = ok && sin >= 0 && s < p.state && v < p.vdim ? old[static_cast<long long>(s) * p.vdim + v] : 0.f;
      }
  }
  const float bias = p.dt_bias[h], rate = p.a_neg[h] * 1.4426950408889634f, skip = p.d_skip[h];
  pdl_wait();
  if (!ok) {
    if (tid == 0) report_status(p.status, kStatusBadIndex, 0xE53, seq, sout);
    return;
  }
  const int r0 = p.seq_start[seq], total = p.seq_start[seq + 1] - r0;
  if (r0 < 0 || total <= 0 || r0 + total > p.rows) {
    if (tid == 0) report_status(p.status, kStatusBadIndex, 0xE54, seq, r0);
    return;
  }
  if (total == 1 && p.skip_single) return;
  // rows of a chunk: B, C (padding states are zeros) and this CTA's columns of x; rows past the end are zeros
  auto request = [&](int t0, int stage) {
    __nv_bfloat16* st = sm + stage * C::kStage;
    const int cnt = total - t0;
    const __nv_bfloat16* src = p.xbc + static_cast<long long>(r0 + t0) * p.ldx;
    constexpr int kN = NP / 8, kV = kHcCols / 8;
    for (int i = tid; i < kHcTokens * kN; i += kHcThreads) {
      const int t = i / kN, c = (i - t * kN) * 8, left = t < cnt ? min(max(p.state - c, 0), 8) * 2 : 0;
      const long long at = left ? t * p.ldx + group * p.state + c : 0;
      hc_copy16(st + C::kB + t * C::kPitchN + c, src + at + (left ? p.off_b : 0), left);
      hc_copy16(st + C::kC + t * C::kPitchN + c, src + at + (left ? p.off_c : 0), left);
    }
    for (int i = tid; i < kHcTokens * kV; i += kHcThreads) {
      const int t = i / kV, c = (i - t * kV) * 8, in = t < cnt && c0 + c < p.vdim;
      hc_copy16(st + C::kX + t * C::kPitchV + c, src + (in ? t * p.ldx + h * p.vdim + c0 + c : 0), in ? 16 : 0);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  // step sizes of two tokens per lane
  float raw[2];
  auto steps = [&](int t0) {
#pragma unroll
    for (int e = 0; e < 2; ++e)
      raw[e] = __bfloat162float(p.dt[static_cast<long long>(r0 + min(t0 + lane * 2 + e, total - 1)) * p.ldp + h]);
  };
  // factors of the chunk at t0 from the step sizes in `raw` (one warp)
  auto prepare = [&](int t0, float* f) {
    const int cnt = min(kHcTokens, total - t0);
    float d[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) d[e] = lane * 2 + e < cnt ? scan_softplus<__nv_bfloat16>(raw[e] + bias) : 0.f;
    const double a0 = static_cast<double>(rate) * d[0], a1 = static_cast<double>(rate) * d[1];
    double sum = a0 + a1;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const double up = __shfl_up_sync(0xffffffffu, sum, o);
      if (lane >= o) sum += up;
    }
    const double end = __shfl_sync(0xffffffffu, sum, 31), l[2] = {sum - a1, sum};
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int t = lane * 2 + e;
      const float hi = static_cast<float>(l[e]);
      f[t] = hi;
      f[kHcTokens + t] = static_cast<float>(l[e] - hi);
      f[2 * kHcTokens + t] = exp2_approx(hi);
      f[3 * kHcTokens + t] = d[e];
      f[4 * kHcTokens + t] = exp2_approx(static_cast<float>(end - l[e])) * d[e];
    }
  };
  request(0, 0);
  if (warp == 0) {
    steps(0);
    prepare(0, factors);
    if (total > kHcTokens) steps(kHcTokens);
  }
  const int chunks = (total + kHcTokens - 1) / kHcTokens;
  for (int k = 0; k < chunks; ++k) {
    const int t0 = k * kHcTokens, cnt = min(kHcTokens, total - t0);
    const float* f_l = factors + (k & 1) * 5 * kHcTokens;
    const float* f_r = f_l + kHcTokens;
    const float* f_e = f_r + kHcTokens;
    const float* f_d = f_e + kHcTokens;
    const float* f_s = f_d + kHcTokens;
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                       // this chunk's rows and factors; nobody reads the other stage any more
    if (k + 1 < chunks) request(t0 + kHcTokens, (k + 1) & 1);
    const __nv_bfloat16* st = sm + (k & 1) * C::kStage;
    const __nv_bfloat16* sb = st + C::kB;
    const __nv_bfloat16* sc = st + C::kC;
    const __nv_bfloat16* sx = st + C::kX;
    __nv_bfloat16* p_hi = sm + C::kP;
    __nv_bfloat16* p_lo = p_hi + kHcTokens * C::kPitchP;
    const int tiles = (cnt + 15) / 16;                                      // token tiles with rows
    // ---- P of token tile `warp`: all tokens up to its own ----
    if (warp < tiles) {
      uint32_t a[NP / 16][4];
      const uint32_t ca = smem_u32(sc + (warp * 16 + (lane & 15)) * C::kPitchN + (lane >> 4) * 8);
#pragma unroll
      for (int s = 0; s < NP / 16; ++s) ldsm_x4(a[s], ca + s * 32);
      const int ra = warp * 16 + g4, rb = ra + 8;
      const float la = f_l[ra], lb = f_l[rb], ma = f_r[ra], mb = f_r[rb];
      auto decay = [](float l, float m, float lc, float mc) { return exp2_approx((l - lc) + (m - mc)); };
      for (int j = 0; j <= warp; ++j) {
        float q[2][4] = {};
        const uint32_t ba = smem_u32(sb + (j * 16 + (lmat >> 1) * 8 + lrow) * C::kPitchN + (lmat & 1) * 8);
#pragma unroll
        for (int s = 0; s < NP / 16; ++s) {
          uint32_t b[4];
          ldsm_x4(b, ba + s * 32);
          mma_bf16_16816(q[0], a[s], b[0], b[1]);
          mma_bf16_16816(q[1], a[s], b[2], b[3]);
        }
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          const int c = j * 16 + n * 8 + t4 * 2;
          const float l0 = f_l[c], l1 = f_l[c + 1], m0 = f_r[c], m1 = f_r[c + 1], d0 = f_d[c], d1 = f_d[c + 1];
          uint32_t hi, lo;
          two_parts(c <= ra ? q[n][0] * (decay(la, ma, l0, m0) * d0) : 0.f, c + 1 <= ra ? q[n][1] * (decay(la, ma, l1, m1) * d1) : 0.f,
                    hi, lo);
          *reinterpret_cast<uint32_t*>(p_hi + ra * C::kPitchP + c) = hi;
          *reinterpret_cast<uint32_t*>(p_lo + ra * C::kPitchP + c) = lo;
          two_parts(c <= rb ? q[n][2] * (decay(lb, mb, l0, m0) * d0) : 0.f, c + 1 <= rb ? q[n][3] * (decay(lb, mb, l1, m1) * d1) : 0.f,
                    hi, lo);
          *reinterpret_cast<uint32_t*>(p_hi + rb * C::kPitchP + c) = hi;
          *reinterpret_cast<uint32_t*>(p_lo + rb * C::kPitchP + c) = lo;
        }
      }
    }
    // (the warp with the fewest products) the next chunk's factors
    if (warp == 0 && k + 1 < chunks) {
      prepare(t0 + kHcTokens, factors + ((k + 1) & 1) * 5 * kHcTokens);
      if (k + 2 < chunks) steps(t0 + 2 * kHcTokens);
    }
    // output gates of this warp's columns, requested before the products
    __nv_bfloat162 z[4][2][2];
#pragma unroll
    for (int m = 0; m < 4; ++m)
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int t = min(m * 16 + g4 + e * 8, cnt - 1), v = min(v0 + n * 8 + t4 * 2, p.vdim - 2);
          z[m][n][e] = *reinterpret_cast<const __nv_bfloat162*>(p.z + static_cast<long long>(r0 + t0 + t) * p.ldp + h * p.vdim + v);
        }
    __syncthreads();                       // P of all tiles
    if (mine) {
      // ---- y = exp(L) C S + P x ----
      float y[4][2][4];
#pragma unroll
      for (int m = 0; m < 4; ++m)
#pragma unroll
        for (int n = 0; n < 2; ++n) y[m][n][0] = y[m][n][1] = y[m][n][2] = y[m][n][3] = 0.f;
#pragma unroll
      for (int s = 0; s < NP / 16; ++s) {
        uint32_t hi[2][2], lo[2][2];
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
          for (int i = 0; i < 2; ++i) two_parts(S[2 * s + i][2 * n], S[2 * s + i][2 * n + 1], hi[n][i], lo[n][i]);
#pragma unroll
        for (int m = 0; m < 4; ++m) {
          if (m < tiles) {
            uint32_t a[4];
            ldsm_x4(a, smem_u32(sc + (m * 16 + (lane & 15)) * C::kPitchN + s * 16 + (lane >> 4) * 8));
#pragma unroll
            for (int n = 0; n < 2; ++n) {
              mma_bf16_16816(y[m][n], a, hi[n][0], hi[n][1]);
              mma_bf16_16816(y[m][n], a, lo[n][0], lo[n][1]);
            }
          }
        }
      }
#pragma unroll
      for (int m = 0; m < 4; ++m) {
        const float ea = f_e[m * 16 + g4], eb = f_e[m * 16 + g4 + 8];
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          y[m][n][0] *= ea;
          y[m][n][1] *= ea;
          y[m][n][2] *= eb;
          y[m][n][3] *= eb;
        }
      }
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        if (j >= tiles) break;
        uint32_t x[4];
        ldsm_x4_t(x, smem_u32(sx + (j * 16 + (lmat & 1) * 8 + lrow) * C::kPitchV + warp * 16 + (lmat >> 1) * 8));
#pragma unroll
        for (int m = 0; m < 4; ++m) {
          if (m >= j && m < tiles) {
            const int at = (m * 16 + (lane & 15)) * C::kPitchP + j * 16 + (lane >> 4) * 8;
            uint32_t a[4], b[4];
            ldsm_x4(a, smem_u32(p_hi + at));
            ldsm_x4(b, smem_u32(p_lo + at));
#pragma unroll
            for (int n = 0; n < 2; ++n) {
              mma_bf16_16816(y[m][n], a, x[2 * n], x[2 * n + 1]);
              mma_bf16_16816(y[m][n], b, x[2 * n], x[2 * n + 1]);
            }
          }
        }
      }
      // ---- skip, output gate ----
#pragma unroll
      for (int m = 0; m < 4; ++m)
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const int t = m * 16 + g4 + e * 8, c = warp * 16 + n * 8 + t4 * 2;
            if (t >= cnt || c0 + c >= p.vdim) continue;
            const float2 x = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(sx + t * C::kPitchV + c));
            const float2 gz = __bfloat1622float2(z[m][n][e]);
            const float o0 = fmaf(skip, x.x, y[m][n][2 * e]) * scan_silu<__nv_bfloat16>(gz.x);
            const float o1 = fmaf(skip, x.y, y[m][n][2 * e + 1]) * scan_silu<__nv_bfloat16>(gz.y);
            *reinterpret_cast<__nv_bfloat162*>(p.out + static_cast<long long>(r0 + t0 + t) * p.ldo + h * p.vdim + c0 + c) =
                __floats2bfloat162_rn(o0, o1);
          }
      // ---- S <- exp(L_end) S + sum of the decayed inputs ----
      if (k + 1 < chunks || sout >= 0) {
        const float e_end = f_e[kHcTokens - 1];
#pragma unroll
        for (int n = 0; n < NP / 8; ++n)
#pragma unroll
          for (int e = 0; e < 4; ++e) S[n][e] *= e_end;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          if (j >= tiles) break;
          uint32_t x[4], hi[4], lo[4];
          ldsm_x4_t(x, smem_u32(sx + (j * 16 + (lmat >> 1) * 8 + lrow) * C::kPitchV + warp * 16 + (lmat & 1) * 8));
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            const int t = j * 16 + t4 * 2 + (i >> 1) * 8;
            const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&x[i]));
            two_parts(v.x * f_s[t], v.y * f_s[t + 1], hi[i], lo[i]);
          }
#pragma unroll
          for (int n = 0; n < NP / 16; ++n) {
            uint32_t b[4];
            ldsm_x4_t(b, smem_u32(sb + (j * 16 + (lmat & 1) * 8 + lrow) * C::kPitchN + n * 16 + (lmat >> 1) * 8));
            mma_bf16_16816(S[2 * n], hi, b[0], b[1]);
            mma_bf16_16816(S[2 * n + 1], hi, b[2], b[3]);
            mma_bf16_16816(S[2 * n], lo, b[0], b[1]);
            mma_bf16_16816(S[2 * n + 1], lo, b[2], b[3]);
          }
        }
      }
    }
  }
  pdl_launch_dependents();
  if (sout < 0) return;
  float* dst = p.states + (static_cast<long long>(sout) * p.heads + h) * plane;
#pragma unroll
  for (int n = 0; n < NP / 8; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int s = n * 8 + t4 * 2 + (e & 1), v = v0 + g4 + (e >> 1) * 8;
      if (s < p.state && v < p.vdim) dst[static_cast<long long>(s) * p.vdim + v] = S[n][e];
    }
}

template <int NP>
static int launch_chunk(const HeadScanParams<__nv_bfloat16>& p, cudaStream_t s) {
  static bool attr = false;
  if (!attr) {
    if (cudaFuncSetAttribute(head_scan_chunk_kernel<NP>, cudaFuncAttributeMaxDynamicSharedMemorySize, HcCfg<NP>::kSmem) != cudaSuccess)
      return FB_ERR_LAUNCH;
    attr = true;
  }
  launch_pdl(head_scan_chunk_kernel<NP>, dim3((p.vdim + kHcCols - 1) / kHcCols, p.heads, p.n_seqs), dim3(kHcThreads), HcCfg<NP>::kSmem,
             s, p);
  return cudaGetLastError() == cudaSuccess ? FB_OK : FB_ERR_LAUNCH;
}

int run_head_scan_chunk(const HeadScanParams<__nv_bfloat16>& p, cudaStream_t s) {
  const uintptr_t bits = reinterpret_cast<uintptr_t>(p.xbc) | reinterpret_cast<uintptr_t>(p.z) | reinterpret_cast<uintptr_t>(p.out);
  if ((bits & 15) || p.ldx % 8 || p.ldp % 8 || p.ldo % 8 || p.off_b % 8 || p.off_c % 8) return FB_ERR_ALIGN;
  if (p.state <= 32) return launch_chunk<32>(p, s);
  if (p.state <= 64) return launch_chunk<64>(p, s);
  return launch_chunk<128>(p, s);
}

}  // namespace fb
