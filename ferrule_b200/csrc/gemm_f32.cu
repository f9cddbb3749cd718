// out = x @ w^T in full 32 bits on the FMA units: the GEMM of models that run in fp32 (no tensor-core mode has 32-bit
// operands).  Takes the argument block of the tcgen05 GEMM - dense, batched per head, grouped by a MoE row-tile
// table; store and GELU (with bias), SwiGLU (clamped, scaled, shifted), GeGLU and weighted scatter epilogues - with fp32 tensors and pitches in elements.
//
// 64 rows x 64 channels per CTA, 256 threads with 4 x 4 outputs each, K in steps of 16 through shared memory.
#include "common.cuh"
#include "ferrule_b200.h"
#include "launch.cuh"

namespace fb {

constexpr int kF32Tile = 64, kF32K = 16;

struct GemmF32Params {
  const float* w;
  const float* x;
  float* out;
  long long ldw, w_group_stride, ldx, ldo;
  int n_out, k, groups, x_rows, ntok, dual_offset, x_group_koff, out_group_coff, batched, gelu, geglu;
  float limit, alpha, shift;
  const float* bias;
  const int* tile_group;
  const int* tile_row0;
  const int* tile_rows;
  const int* num_tiles;
  const int* dst_row;
  const float* row_scale;
};

template <bool DUAL>
__global__ void __launch_bounds__(256)
gemm_f32_kernel(const GemmF32Params p) {
  pdl_launch_dependents();
  pdl_wait();
  __shared__ float xs[kF32K][kF32Tile + 4], ws[kF32K][kF32Tile + 4], us[DUAL ? kF32K : 1][kF32Tile + 4];
  int group = 0, row0, rows;
  if (p.tile_group) {
    // grid.y = table tile * sub-tiles of 64 rows
    const int subs = (p.ntok + kF32Tile - 1) / kF32Tile;
    const int t = blockIdx.y / subs, sub = blockIdx.y - t * subs;
    if (t >= *p.num_tiles) return;
    group = p.tile_group[t];
    row0 = p.tile_row0[t] + sub * kF32Tile;
    rows = min(p.tile_rows[t] - sub * kF32Tile, kF32Tile);
    if (rows <= 0 || group < 0 || group >= p.groups || row0 < 0 || row0 + rows > p.x_rows) return;
  } else {
    row0 = blockIdx.y * kF32Tile;
    rows = min(p.x_rows - row0, kF32Tile);
    group = p.batched ? blockIdx.z : 0;
  }
  const int n0 = blockIdx.x * kF32Tile;
  const float* x = p.x + (p.batched ? static_cast<long long>(group) * p.x_group_koff : 0);
  const float* w = p.w + group * p.w_group_stride;
  const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
  const int lr = tid >> 2, lk = (tid & 3) * 4;      // loader: row of the tile, first of four k
  float acc[4][4] = {}, up[4][4] = {};
  for (int k0 = 0; k0 < p.k; k0 += kF32K) {
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int k = k0 + lk + j;
      const bool kin = k < p.k;
      xs[lk + j][lr] = (kin && lr < rows) ? x[(row0 + lr) * p.ldx + k] : 0.f;
      ws[lk + j][lr] = (kin && n0 + lr < p.n_out) ? w[(n0 + lr) * p.ldw + k] : 0.f;
      if (DUAL) us[lk + j][lr] = (kin && n0 + lr < p.n_out) ? w[(p.dual_offset + n0 + lr) * p.ldw + k] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kF32K; ++k) {
      float a[4], b[4], c[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        a[i] = xs[k][ty * 4 + i];
        b[i] = ws[k][tx * 4 + i];
        if (DUAL) c[i] = us[k][tx * 4 + i];
      }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
          if (DUAL) up[i][j] = fmaf(a[i], c[j], up[i][j]);
        }
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int r = ty * 4 + i;
    if (r >= rows) continue;
    const long long orow = p.dst_row ? p.dst_row[row0 + r] : row0 + r;
    if (orow < 0) continue;
    const float sc = p.row_scale ? p.row_scale[row0 + r] : 1.f;
    float* o = p.out + orow * p.ldo + (p.batched ? static_cast<long long>(group) * p.out_group_coff : 0);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n >= p.n_out) continue;
      float v = acc[i][j];
      if (DUAL) {
        float u = up[i][j];
        if (p.limit > 0.f) {
          v = fminf(v, p.limit);
          u = fminf(fmaxf(u, -p.limit), p.limit);
        }
        v = (p.geglu ? gelu_tanh_f(v) : v / (1.f + expf(-p.alpha * v))) * (u + p.shift);
      }
      if (p.bias) v += p.bias[n];
      if (p.gelu) v = gelu_f(v);
      o[n] = v * sc;
    }
  }
}

}  // namespace fb

using namespace fb;

extern "C" int fb_gemm_f32(const FbGemmArgs* a, void* stream) {
  if (!a || !a->w || !a->x || !a->out || a->n_out <= 0 || a->k <= 0 || a->groups <= 0 || a->x_rows <= 0) return FB_ERR_SHAPE;
  if (a->epilogue < 0 || a->epilogue == 3 || a->epilogue > 5) return FB_ERR_SHAPE;
  const bool grouped = a->tile_group != nullptr, batched = !grouped && a->groups > 1;
  if (grouped && (!a->tile_row0 || !a->tile_rows || !a->num_tok_tiles || a->max_tok_tiles <= 0 || a->ntok <= 0))
    return FB_ERR_SHAPE;
  if (batched && a->epilogue != 0) return FB_ERR_SHAPE;
  GemmF32Params p{};
  p.w = static_cast<const float*>(a->w); p.x = static_cast<const float*>(a->x); p.out = static_cast<float*>(a->out);
  p.ldw = a->ldw; p.w_group_stride = a->w_group_stride; p.ldx = a->ldx; p.ldo = a->ldo;
  p.n_out = a->n_out; p.k = a->k; p.groups = a->groups; p.x_rows = a->x_rows; p.ntok = a->ntok;
  p.dual_offset = a->dual_offset; p.x_group_koff = a->x_group_koff; p.out_group_coff = a->out_group_coff;
  p.batched = batched ? 1 : 0;
  if (a->bias && (grouped || batched || (a->epilogue != 0 && a->epilogue != 4))) return FB_ERR_SHAPE;
  p.limit = a->epilogue == 1 ? a->act_limit : 0.f;
  p.alpha = a->act_alpha == 0.f ? 1.f : a->act_alpha;
  p.shift = a->act_shift;
  p.bias = a->bias;
  p.gelu = a->epilogue == 4 ? 1 : 0;
  p.geglu = a->epilogue == 5 ? 1 : 0;
  if (grouped) {
    p.tile_group = a->tile_group; p.tile_row0 = a->tile_row0; p.tile_rows = a->tile_rows; p.num_tiles = a->num_tok_tiles;
  }
  if (a->epilogue == 2) { p.dst_row = a->dst_row; p.row_scale = a->row_scale; }
  const int row_tiles = grouped ? a->max_tok_tiles * ((a->ntok + kF32Tile - 1) / kF32Tile)
                                : (a->x_rows + kF32Tile - 1) / kF32Tile;
  if (row_tiles > 65535 || (batched && a->groups > 65535)) return FB_ERR_LIMIT;
  const dim3 grid((a->n_out + kF32Tile - 1) / kF32Tile, row_tiles, batched ? a->groups : 1);
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (a->epilogue == 1 || a->epilogue == 5) launch_pdl(gemm_f32_kernel<true>, grid, dim3(256), 0, s, p);
  else launch_pdl(gemm_f32_kernel<false>, grid, dim3(256), 0, s, p);
  return cudaGetLastError() == cudaSuccess ? FB_OK : FB_ERR_LAUNCH;
}
