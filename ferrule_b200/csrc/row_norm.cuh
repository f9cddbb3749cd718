// RMS norm of equal parts of a row whose elements lie in the registers of one CTA: vectors of 8 consecutive elements, VPT per
// thread.
#pragma once
#include "act_type.cuh"
#include "common.cuh"

namespace fb {

constexpr int kRowThreads = 256;

// Sums of squares meet in shared memory: of a warp's 256 consecutive elements each when parts are multiples of that, else of
// 8 elements each (of single ones when a part is no multiple of 8), followed by the inverse root mean square of every part.
struct GroupScratch {
  float* sums;
  float* inv;
  float (*red)[64];
};

template <int VPT>
__device__ __forceinline__ void group_norm(const float (&v)[VPT][8], int dim, int groups, float eps, const GroupScratch& g,
                                           int turn, float (&out)[VPT][8]) {
  const int part = dim / groups;
  if (part % 256 == 0) {
    const int lane = threadIdx.x & 31;
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
      const int i = (k * blockDim.x + threadIdx.x) * 8;
      float ss = 0.f;
#pragma unroll
      for (int j = 0; j < 8; ++j) ss = fmaf(v[k][j], v[k][j], ss);
      ss = warp_sum(ss);
      if (lane == 0 && i < dim) g.red[turn][i / 256] = ss;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < VPT; ++k) {
      const int i = (k * blockDim.x + threadIdx.x) * 8, n = part / 256, first = i < dim ? i / part * n : 0;
      float ss = 0.f;
      for (int w = 0; w < n; ++w) ss += g.red[turn][first + w];
      const float f = 1.f / sqrtf(ss / part + eps);
#pragma unroll
      for (int j = 0; j < 8; ++j) out[k][j] = v[k][j] * f;
    }
    return;
  }
  if (groups == 1) {
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < VPT; ++k)
#pragma unroll
      for (int j = 0; j < 8; ++j) ss = fmaf(v[k][j], v[k][j], ss);      // columns past `dim` are zero
    const float f = 1.f / sqrtf(cta_sum(ss, g.red[turn]) / dim + eps);
#pragma unroll
    for (int k = 0; k < VPT; ++k)
#pragma unroll
      for (int j = 0; j < 8; ++j) out[k][j] = v[k][j] * f;
    return;
  }
  const bool aligned = part % 8 == 0;
#pragma unroll
  for (int k = 0; k < VPT; ++k) {
    const int i = (k * blockDim.x + threadIdx.x) * 8;
    if (i >= dim) continue;
    if (aligned) {
      float ss = 0.f;
#pragma unroll
      for (int j = 0; j < 8; ++j) ss = fmaf(v[k][j], v[k][j], ss);
      g.sums[i / 8] = ss;
    } else {
#pragma unroll
      for (int j = 0; j < 8; ++j)
        if (i + j < dim) g.sums[i + j] = v[k][j] * v[k][j];
    }
  }
  __syncthreads();
  const int n = aligned ? part / 8 : part, lane = threadIdx.x & 31;
  for (int p = threadIdx.x >> 5; p < groups; p += blockDim.x >> 5) {
    float ss = 0.f;
    for (int i = lane; i < n; i += 32) ss += g.sums[p * n + i];
    ss = warp_sum(ss);
    if (lane == 0) g.inv[p] = 1.f / sqrtf(ss / part + eps);
  }
  __syncthreads();
#pragma unroll
  for (int k = 0; k < VPT; ++k) {
    const int i = (k * blockDim.x + threadIdx.x) * 8;
    const float f = i < dim ? g.inv[i / part] : 0.f;
#pragma unroll
    for (int j = 0; j < 8; ++j)
      out[k][j] = v[k][j] * (aligned || i + j >= dim ? f : g.inv[(i + j) / part]);
  }
}

// threads of a row CTA and vectors of 8 per thread
inline int row_threads(int dim_pad) {
  const int vecs = dim_pad / 8, t = (vecs + 31) / 32 * 32;
  return t < kRowThreads ? t : kRowThreads;
}
inline int row_vpt(int dim_pad) {
  const int t = row_threads(dim_pad), n = (dim_pad / 8 + t - 1) / t;
  return n <= 1 ? 1 : n <= 2 ? 2 : n <= 4 ? 4 : n <= 8 ? 8 : 0;
}
// partial sums `GroupScratch` holds
inline int group_sums(int dim, int groups) { return groups == 1 ? 0 : dim / groups % 8 ? dim : dim / 8; }

}  // namespace fb
