// Grouped-query attention inside position chunks or sliding windows for few query rows (decode steps, short portions), bf16.
//
// CTA = (query row, key / value head and block of 16 query heads, split of the visible keys).  A 16-row MMA tile holds the
// query heads (with two score maps per head: both maps' rows) that share the key / value head; the visible keys - kept first
// tokens, then the chunk or window - are walked in tiles of 16, every warp on its own tiles with its
// own asynchronous copy pipeline and online softmax, so the loop has no barrier between warps.  The four warps merge in
// shared memory, the splits of a row (one thread-block cluster) through distributed shared memory.
//
// The kernel is bound by the key / value stream, a 16-row tile is below the 64-row minimum of tcgen05: warp-level MMA.
// In a decode step the first keys of a warp (older than the step) are requested before the dependency wait.
#include "common.cuh"
#include "act_type.cuh"
#include "ferrule_b200.h"
#include "gqa_mask.cuh"
#include "launch.cuh"
#include "mma_sync.cuh"

namespace fb {

constexpr int kGdThreads = 128;
constexpr int kGdTile = 16;          // keys per warp and pipeline stage

struct GdParams {
  const __nv_bfloat16* q;
  long long ldq;
  const __nv_bfloat16* pool;
  long long pool_rows, pool_ld;
  const int* block_table;
  const int* row_seq;
  const int* row_pos;
  int num_seqs, max_blocks, page_size;
  KeySpan span;
  float scale_log2;
  const float* slopes;               // [heads]
  const __nv_bfloat16* gate;
  long long ldg;
  int maps, v_offset, vdim;
  float diff_lambda, diff_scale, eps;
  __nv_bfloat16* out;
  long long ldo;
  int rows, heads, kv_heads, key_width, vdim_pad, head_blocks;
  int early;                         // every key below a row's own position predates the preceding kernel
  DeviceStatus* status;
};

// 16 bytes global -> shared; bytes past `valid` (0 or 16) are zeros
__device__ __forceinline__ void gd_copy16(uint32_t dst, const void* src, int valid) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(valid) : "memory");
}

template <int D>
struct GdCfg {
  static constexpr int kStages = D <= 128 ? 3 : 2;
  static constexpr int kPitch = D + 8;                              // bf16 elements: conflict-free ldmatrix
  static constexpr int kTileElems = kGdTile * kPitch;
  static constexpr int kWarpElems = kStages * 2 * kTileElems;       // keys and values
  static constexpr int kOPitch = D + 4;
  static constexpr int kKvBytes = 4 * kWarpElems * 2;
  static constexpr int kMergeBytes = 4 * 16 * kOPitch * 4;
  static constexpr int kSmem = (kKvBytes > kMergeBytes ? kKvBytes : kMergeBytes) + (4 * 16 * 2 + 16 * 2) * 4;
};

template <int D>
__global__ void __launch_bounds__(kGdThreads)
gqa_decode_kernel(const GdParams p) {
  using C = GdCfg<D>;
  pdl_launch_dependents();
  extern __shared__ __align__(128) uint8_t gd_smem[];
  constexpr int kBody = C::kKvBytes > C::kMergeBytes ? C::kKvBytes : C::kMergeBytes;
  __nv_bfloat16* kv_s = reinterpret_cast<__nv_bfloat16*>(gd_smem);
  float* o_s = reinterpret_cast<float*>(gd_smem);                   // after the loop: [4][16][kOPitch]
  float* w_m = reinterpret_cast<float*>(gd_smem + kBody);           // [4][16] maxima, [4][16] sums per warp
  float* w_l = w_m + 64;
  float* c_m = w_l + 64;                                            // [16], [16]: of this CTA
  float* c_l = c_m + 16;
  const int r = blockIdx.x, split = blockIdx.y, splits = gridDim.y;
  const int g = blockIdx.z / p.head_blocks, hb = blockIdx.z - g * p.head_blocks;
  const int per = p.heads / p.kv_heads * p.maps, h0 = hb * 16, nh = min(16, per - h0);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g4 = lane >> 2, t4 = lane & 3;
  const int seq = p.row_seq[r], pos = p.row_pos[r];
  int lo = 0, hi = 0, first = 0, kept = 0, n_keys = 0;               // lo, hi: indices into the visible keys
  if (seq < 0 || seq >= p.num_seqs) {
    if (tid == 0) report_status(p.status, kStatusBadIndex, 0xD80, r, seq);
  } else if (pos >= 0) {
    first = p.span.first(pos);
    kept = p.span.head(pos);
    n_keys = kept + max(min(pos + 1, p.max_blocks * p.page_size) - first, 0);
    // whole tiles per split, aligned to the first visible key
    const int tiles = (n_keys + kGdTile - 1) / kGdTile, share = (tiles + splits - 1) / splits;
    lo = min(split * share * kGdTile, n_keys);
    hi = min(lo + share * kGdTile, n_keys);
  }
  auto token = [&](int i) { return i < kept ? i : first + i - kept; };
  const long long n_pages = p.pool_rows / p.page_size;
  const __nv_bfloat16* kbase = p.pool + static_cast<long long>(g) * p.key_width;
  const __nv_bfloat16* vbase = p.pool + p.v_offset + static_cast<long long>(g) * p.vdim_pad;
  __nv_bfloat16* mine = kv_s + warp * C::kWarpElems;
  const int n_tiles = (hi - lo + kGdTile - 1) / kGdTile;
  const int my_tiles = n_tiles > warp ? (n_tiles - warp + 3) / 4 : 0;

  // the tile's 16 keys: two lanes per key, each half of the 16-byte pieces
  const int trow = lane >> 1, half = lane & 1;
  auto request = [&](int i) {
    const int at = lo + (warp + 4 * i) * kGdTile + trow;
    const __nv_bfloat16* src = nullptr;
    if (at < hi) {
      const int t = token(at);
      const int page = p.block_table[static_cast<long long>(seq) * p.max_blocks + t / p.page_size];
      if (page >= 0 && page < n_pages) src = p.pool + (static_cast<long long>(page) * p.page_size + t % p.page_size) * p.pool_ld;
      else if (half == 0) report_status(p.status, kStatusBadIndex, 0xD81, seq, t);
    }
    const long long off = src ? src - p.pool : 0;
    __nv_bfloat16* ks = mine + (i % C::kStages) * 2 * C::kTileElems;
    const uint32_t kd = smem_u32(ks + trow * C::kPitch), vd = smem_u32(ks + C::kTileElems + trow * C::kPitch);
#pragma unroll
    for (int c = 0; c < D / 16; ++c) {
      const int e = (2 * c + half) * 8;
      const int kin = src && e < p.key_width, vin = src && e < p.vdim_pad;
      gd_copy16(kd + e * 2, kbase + (kin ? off + e : 0), kin ? 16 : 0);
      gd_copy16(vd + e * 2, vbase + (vin ? off + e : 0), vin ? 16 : 0);
    }
  };
  int asked = 0;
  if (p.early) {
    // tiles that end below the row's own position: written by earlier steps
    while (asked < C::kStages - 1 && asked < my_tiles && lo + (warp + 4 * asked + 1) * kGdTile < n_keys) {
      request(asked++);
      asm volatile("cp.async.commit_group;" ::: "memory");
    }
  }
  pdl_wait();
  for (; asked < C::kStages - 1; ++asked) {
    if (asked < my_tiles) request(asked);
    asm volatile("cp.async.commit_group;" ::: "memory");
  }
  // query fragments: rows are the group's heads
  uint32_t qf[D / 16][4];
  {
    const __nv_bfloat16* q0 = p.q + r * p.ldq + static_cast<long long>(g * per + h0) * p.key_width;
    auto q2 = [&](int head, int d) -> uint32_t {
      if (head >= nh || d >= p.key_width) return 0u;
      return *reinterpret_cast<const uint32_t*>(q0 + static_cast<long long>(head) * p.key_width + d);
    };
#pragma unroll
    for (int k = 0; k < D / 16; ++k) {
      qf[k][0] = q2(g4, k * 16 + t4 * 2);
      qf[k][1] = q2(g4 + 8, k * 16 + t4 * 2);
      qf[k][2] = q2(g4, k * 16 + 8 + t4 * 2);
      qf[k][3] = q2(g4 + 8, k * 16 + 8 + t4 * 2);
    }
  }
  // distance bias of this thread's two rows, base 2
  auto slope = [&](int row) {
    return p.slopes && row < nh ? p.slopes[(g * per + h0 + row) / p.maps] * 1.4426950408889634f : 0.f;
  };
  const float sl0 = slope(g4), sl1 = slope(g4 + 8);
  float o[D / 8][4];
#pragma unroll
  for (int n = 0; n < D / 8; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;
  float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;
  const int lrow = lane & 7, lmat = lane >> 3;
  for (int i = 0; i < my_tiles; ++i) {
    if (i + C::kStages - 1 < my_tiles) request(i + C::kStages - 1);
    asm volatile("cp.async.commit_group;" ::: "memory");
    asm volatile("cp.async.wait_group %0;" ::"n"(C::kStages - 1) : "memory");
    __syncwarp();
    const __nv_bfloat16* ks = mine + (i % C::kStages) * 2 * C::kTileElems;
    const __nv_bfloat16* vs = ks + C::kTileElems;
    float s[2][4] = {};
    // matrices: keys 0-7 / 8-15 x features 0-7 / 8-15
    const uint32_t ka = smem_u32(ks + ((lmat >> 1) * 8 + lrow) * C::kPitch + (lmat & 1) * 8);
#pragma unroll
    for (int k = 0; k < D / 16; ++k) {
      if (k * 16 < p.key_width) {
        uint32_t b[4];
        ldsm_x4(b, ka + k * 32);
        mma_bf16_16816(s[0], qf[k], b[0], b[1]);
        mma_bf16_16816(s[1], qf[k], b[2], b[3]);
      }
    }
    const int t0 = lo + (warp + 4 * i) * kGdTile + t4 * 2;
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) s[n][e] = t0 + n * 8 + (e & 1) < hi ? s[n][e] * p.scale_log2 : -INFINITY;
    if (p.slopes) {
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e)
          s[n][e] = fmaf(e < 2 ? -sl0 : -sl1, static_cast<float>(pos - token(t0 + n * 8 + (e & 1))), s[n][e]);
    }
    float x0 = fmaxf(fmaxf(s[0][0], s[0][1]), fmaxf(s[1][0], s[1][1]));
    float x1 = fmaxf(fmaxf(s[0][2], s[0][3]), fmaxf(s[1][2], s[1][3]));
#pragma unroll
    for (int w = 1; w < 4; w <<= 1) {
      x0 = fmaxf(x0, __shfl_xor_sync(0xffffffffu, x0, w));
      x1 = fmaxf(x1, __shfl_xor_sync(0xffffffffu, x1, w));
    }
    if (__any_sync(0xffffffffu, x0 > m0 || x1 > m1)) {
      const float n0 = fmaxf(m0, x0), n1 = fmaxf(m1, x1);        // finite: a tile has at least one visible key
      const float f0 = exp2f(m0 - n0), f1 = exp2f(m1 - n1);
      m0 = n0;
      m1 = n1;
      l0 *= f0;
      l1 *= f1;
#pragma unroll
      for (int n = 0; n < D / 8; ++n) {
        o[n][0] *= f0;
        o[n][1] *= f0;
        o[n][2] *= f1;
        o[n][3] *= f1;
      }
    }
#pragma unroll
    for (int n = 0; n < 2; ++n) {
      s[n][0] = exp2f(s[n][0] - m0);
      s[n][1] = exp2f(s[n][1] - m0);
      s[n][2] = exp2f(s[n][2] - m1);
      s[n][3] = exp2f(s[n][3] - m1);
      l0 += s[n][0] + s[n][1];
      l1 += s[n][2] + s[n][3];
    }
    auto pack = [](float a, float b) -> uint32_t {
      const __nv_bfloat162 v = __floats2bfloat162_rn(a, b);
      return *reinterpret_cast<const uint32_t*>(&v);
    };
    const uint32_t pf[4] = {pack(s[0][0], s[0][1]), pack(s[0][2], s[0][3]), pack(s[1][0], s[1][1]), pack(s[1][2], s[1][3])};
    // matrices (transposed): keys 0-7 / 8-15 x features 0-7, then features 8-15
    const uint32_t va = smem_u32(vs + ((lmat & 1) * 8 + lrow) * C::kPitch + (lmat >> 1) * 8);
#pragma unroll
    for (int n = 0; n < D / 16; ++n) {
      if (n * 16 < p.vdim_pad) {
        uint32_t b[4];
        ldsm_x4_t(b, va + n * 32);
        mma_bf16_16816(o[2 * n], pf, b[0], b[1]);
        mma_bf16_16816(o[2 * n + 1], pf, b[2], b[3]);
      }
    }
    __syncwarp();
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
#pragma unroll
  for (int w = 1; w < 4; w <<= 1) {
    l0 += __shfl_xor_sync(0xffffffffu, l0, w);
    l1 += __shfl_xor_sync(0xffffffffu, l1, w);
  }
  __syncthreads();                                                   // the tiles' memory now holds the partial outputs
  if (t4 == 0) {
    w_m[warp * 16 + g4] = m0;
    w_m[warp * 16 + g4 + 8] = m1;
    w_l[warp * 16 + g4] = l0;
    w_l[warp * 16 + g4 + 8] = l1;
  }
#pragma unroll
  for (int n = 0; n < D / 8; ++n) {
    float* d0 = o_s + (warp * 16 + g4) * C::kOPitch + n * 8 + t4 * 2;
    d0[0] = o[n][0];
    d0[1] = o[n][1];
    d0[8 * C::kOPitch] = o[n][2];
    d0[8 * C::kOPitch + 1] = o[n][3];
  }
  __syncthreads();
  // the four warps of this CTA; the merged rows replace warp 0's
  if (tid < 16) {
    float m = -INFINITY, l = 0.f;
#pragma unroll
    for (int w = 0; w < 4; ++w) m = fmaxf(m, w_m[w * 16 + tid]);
#pragma unroll
    for (int w = 0; w < 4; ++w) {
      const float f = w_m[w * 16 + tid] == -INFINITY ? 0.f : exp2f(w_m[w * 16 + tid] - m);
      l += f * w_l[w * 16 + tid];
      w_m[w * 16 + tid] = f;
    }
    c_m[tid] = m;
    c_l[tid] = l;
  }
  __syncthreads();
  for (int i = tid; i < nh * (D / 4); i += kGdThreads) {
    const int h = i / (D / 4), d = (i - h * (D / 4)) * 4;
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int w = 0; w < 4; ++w) {
      const float f = w_m[w * 16 + h];
      const float4 v = *reinterpret_cast<const float4*>(o_s + (w * 16 + h) * C::kOPitch + d);
      a.x = fmaf(f, v.x, a.x);
      a.y = fmaf(f, v.y, a.y);
      a.z = fmaf(f, v.z, a.z);
      a.w = fmaf(f, v.w, a.w);
    }
    *reinterpret_cast<float4*>(o_s + h * C::kOPitch + d) = a;
  }
  if (splits > 1) cluster_sync_all();
  else __syncthreads();
  // every CTA of the cluster finishes its share of the output over all splits
  const int quads = p.vdim_pad / 4, out_per = p.heads / p.kv_heads;
  auto merged = [&](int h, int d) -> float4 {
    float m = -INFINITY, l = 0.f;
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
    if (splits == 1) {
      l = c_l[h];
      a = *reinterpret_cast<const float4*>(o_s + h * C::kOPitch + d);
    } else {
      for (int s = 0; s < splits; ++s) m = fmaxf(m, ld_cluster_f32(mapa_shared(smem_u32(c_m + h), s)));
      for (int s = 0; s < splits; ++s) {
        const float ms = ld_cluster_f32(mapa_shared(smem_u32(c_m + h), s));
        const float f = ms == -INFINITY ? 0.f : exp2f(ms - m);
        l = fmaf(f, ld_cluster_f32(mapa_shared(smem_u32(c_l + h), s)), l);
        const float4 v = ld_cluster_f32x4(mapa_shared(smem_u32(o_s + h * C::kOPitch + d), s));
        a.x = fmaf(f, v.x, a.x);
        a.y = fmaf(f, v.y, a.y);
        a.z = fmaf(f, v.z, a.z);
        a.w = fmaf(f, v.w, a.w);
      }
    }
    const float inv = l > 0.f ? 1.f / l : 0.f;
    return make_float4(a.x * inv, a.y * inv, a.z * inv, a.w * inv);
  };
  // head: of this key / value head
  auto finish = [&](int head, int d, float4 a) {
    const long long col = static_cast<long long>(g * out_per + head) * p.vdim_pad + d;
    if (p.gate) {
      const __nv_bfloat162* z = reinterpret_cast<const __nv_bfloat162*>(p.gate + r * p.ldg + col);
      const float2 z0 = __bfloat1622float2(z[0]), z1 = __bfloat1622float2(z[1]);
      a = make_float4(a.x * sigmoid_f(z0.x), a.y * sigmoid_f(z0.y), a.z * sigmoid_f(z1.x), a.w * sigmoid_f(z1.y));
    }
    __nv_bfloat16* dst = p.out + r * p.ldo + col;
    *reinterpret_cast<__nv_bfloat162*>(dst) = __floats2bfloat162_rn(a.x, a.y);
    *reinterpret_cast<__nv_bfloat162*>(dst + 2) = __floats2bfloat162_rn(a.z, a.w);
  };
  if (p.maps == 2) {
    // one warp per head: difference of its two rows, RMS norm over the head
    constexpr int kQ = (D / 4 + 31) / 32;
    for (int h = warp + 4 * split; h < nh / 2; h += 4 * splits) {
      float4 a[kQ];
      float ss = 0.f;
#pragma unroll
      for (int k = 0; k < kQ; ++k) {
        const int c = lane + 32 * k;
        a[k] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (c < quads) {
          const float4 x = merged(2 * h, c * 4), y = merged(2 * h + 1, c * 4);
          a[k] = make_float4(x.x - p.diff_lambda * y.x, x.y - p.diff_lambda * y.y, x.z - p.diff_lambda * y.z,
                             x.w - p.diff_lambda * y.w);
        }
        ss += a[k].x * a[k].x + a[k].y * a[k].y + a[k].z * a[k].z + a[k].w * a[k].w;
      }
      const float f = p.diff_scale / sqrtf(warp_sum(ss) / p.vdim + p.eps);
#pragma unroll
      for (int k = 0; k < kQ; ++k)
        if (lane + 32 * k < quads)
          finish(h0 / 2 + h, (lane + 32 * k) * 4, make_float4(a[k].x * f, a[k].y * f, a[k].z * f, a[k].w * f));
    }
  } else {
    for (int i = tid + split * kGdThreads; i < nh * quads; i += kGdThreads * splits) {
      const int h = i / quads, d = (i - h * quads) * 4;
      finish(h0 + h, d, merged(h, d));
    }
  }
  if (splits > 1) cluster_sync_all();                                // no CTA leaves while a peer reads its rows
}

template <int D>
static int launch_gd(const GdParams& p, int splits, cudaStream_t stream) {
  static bool attr_set = false;
  if (!attr_set) {
    if (cudaFuncSetAttribute(gqa_decode_kernel<D>, cudaFuncAttributeMaxDynamicSharedMemorySize, GdCfg<D>::kSmem) != cudaSuccess)
      return FB_ERR_LAUNCH;
    attr_set = true;
  }
  cudaLaunchConfig_t cfg{};
  cfg.gridDim = dim3(p.rows, splits, p.kv_heads * p.head_blocks);
  cfg.blockDim = dim3(kGdThreads);
  cfg.dynamicSmemBytes = GdCfg<D>::kSmem;
  cfg.stream = stream;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = 1;
  attr[0].val.clusterDim.y = splits;
  attr[0].val.clusterDim.z = 1;
  attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[1].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr;
  cfg.numAttrs = pdl_enabled() ? 2 : 1;
  if (cudaLaunchKernelEx(&cfg, gqa_decode_kernel<D>, p) != cudaSuccess) return FB_ERR_LAUNCH;
  return cudaGetLastError() == cudaSuccess ? FB_OK : FB_ERR_LAUNCH;
}

}  // namespace fb

using namespace fb;

extern "C" int fb_gqa_decode(const FbGqaArgs* a, int splits, int early, void* stream) {
  if (!a || !a->q || !a->pool || !a->out || !a->block_table || !a->row_seq || !a->row_pos || a->fp32) return FB_ERR_SHAPE;
  if (a->rows <= 0 || a->heads <= 0 || a->kv_heads <= 0 || a->heads % a->kv_heads || a->vdim_pad <= 0 || a->vdim_pad % 8 ||
      a->pool_rows <= 0 || a->pool_ld % 8 || a->num_seqs <= 0 || a->max_blocks <= 0 || a->page_size <= 0)
    return FB_ERR_SHAPE;
  if (!gqa_form_ok(a) || !gqa_plain_form(a) || a->key_stride == 0 || a->ldq % 8 || a->ldo % 4 || a->ldg % 4) return FB_ERR_SHAPE;
  if (splits != 1 && splits != 2 && splits != 4 && splits != 8) return FB_ERR_SHAPE;
  const uintptr_t bits = reinterpret_cast<uintptr_t>(a->q) | reinterpret_cast<uintptr_t>(a->pool) |
                         reinterpret_cast<uintptr_t>(a->out) | reinterpret_cast<uintptr_t>(a->gate);
  if (bits & 15) return FB_ERR_ALIGN;
  GdParams p{};
  p.q = static_cast<const __nv_bfloat16*>(a->q); p.ldq = a->ldq;
  p.pool = static_cast<const __nv_bfloat16*>(a->pool); p.pool_rows = a->pool_rows; p.pool_ld = a->pool_ld;
  p.block_table = a->block_table; p.row_seq = a->row_seq; p.row_pos = a->row_pos;
  p.num_seqs = a->num_seqs; p.max_blocks = a->max_blocks; p.page_size = a->page_size;
  p.span = key_span(a);
  p.slopes = a->slopes; p.gate = static_cast<const __nv_bfloat16*>(a->gate); p.ldg = a->ldg;
  p.maps = a->maps; p.v_offset = a->v_offset; p.vdim = a->vdim;
  p.diff_lambda = a->diff_lambda; p.diff_scale = a->diff_scale; p.eps = a->eps;
  p.scale_log2 = a->scale * 1.4426950408889634f;
  p.out = static_cast<__nv_bfloat16*>(a->out); p.ldo = a->ldo;
  p.rows = a->rows; p.heads = a->heads; p.kv_heads = a->kv_heads; p.key_width = a->key_width; p.vdim_pad = a->vdim_pad;
  p.head_blocks = (a->heads / a->kv_heads * a->maps + 15) / 16;
  p.early = early;
  p.status = static_cast<DeviceStatus*>(a->status);
  if (static_cast<long long>(p.kv_heads) * p.head_blocks > 65535) return FB_ERR_LIMIT;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const int d = a->key_width > a->vdim_pad ? a->key_width : a->vdim_pad;
  if (d <= 64) return launch_gd<64>(p, splits, s);
  if (d <= 128) return launch_gd<128>(p, splits, s);
  if (d <= 256) return launch_gd<256>(p, splits, s);
  return FB_ERR_LIMIT;
}
