// Window attention of few query rows (decode steps, short portions) whose query rows meet the keys or the values of all kv heads,
// bf16.
//
// Scores that are mixed across heads are products of one wide query row per head with the concatenated keys of a token
// (head_prep.cu), so a CTA takes all of a token's cache row: keys and values of every kv head lie side by side there and come
// as one bulk copy per token.  Softmax weights that are mixed across heads need every head's weights on the values of every kv
// head: the keys of the CTA's own kv heads (a query is zero in the others' columns) and all values, and every CTA mixes its outputs
// before the cluster adds them up.  Mean rows of the blocks before the window (gqa_mask.cuh) are keys like any other.  CTA = (query row, split of the visible keys, block of 16 heads); a tile is KT tokens.
//
//   copies   warp 8 looks up a token per lane and keeps all stages requested
//   scores   warp w of 8 multiplies the 16 query rows with 8 of the tile's keys over a share of the features (MMA, partial
//            sums in shared memory); query fragments stay in registers when their share is at most 16 steps
//   softmax  two rows per warp, a key per lane: distance bias, running maximum and sum, probabilities to shared memory
//   values   warp w accumulates 16-column pieces w, w + 8, ... of the values for all 16 rows; a head keeps the columns of
//            its own kv head (mixed weights: all of them)
//
// The splits of a row (one thread-block cluster; with mixed weights the row's head blocks too) merge through distributed shared
// memory; the output gate is applied there.
// The kernel is bound by the cache stream, a 16-row tile is below the 64-row minimum of tcgen05: warp-level MMA.  In a decode
// step the first tiles (older than the step) are requested before the dependency wait.  Every wait is bounded.
#include "act_type.cuh"
#include "common.cuh"
#include "ferrule_b200.h"
#include "gqa_mask.cuh"
#include "launch.cuh"
#include "mma_sync.cuh"

namespace fb {

constexpr int kGwThreads = 256;      // of the 8 computing warps
constexpr int kGwMaxStages = 8;
constexpr int kGwSmemLimit = 227 * 1024;

struct GwParams {
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
  const float* slopes;
  const __nv_bfloat16* gate;
  long long ldg;
  __nv_bfloat16* out;
  long long ldo;
  int heads, kv_heads, key_width, vdim_pad;
  int own_keys;                                    // > 0: a query row is this wide and meets the keys of its kv head; key_width
                                                   //   is then that of the most kv heads a block of 16 heads has
  int v_offset;                                    // first value column of a cache row in memory
  float cap_log2, cap_in;                          // soft cap: score2 <- cap_log2 tanh(raw * cap_in / 2); 0: none
  PooledRows<__nv_bfloat16> pooled;
  const float* talk;
  int row_bytes, pitch, stages, head_blocks;       // bytes of a token's keys and values, and of its place in a tile
  int early;
  DeviceStatus* status;
};

// shared memory behind the tiles
struct GwLayout {
  int q_pitch, q, part, prob, factor, talk, bars, total;
  __host__ __device__ GwLayout(int key_width, int tile_bytes, int kt, int talk_heads) {
    q_pitch = (key_width + 15) / 16 * 16 + 8;
    q = tile_bytes;
    part = q + 16 * q_pitch * 2;
    prob = part + (64 / kt) * 16 * (kt + 1) * 4;
    factor = prob + 16 * (kt + 8) * 2;
    talk = factor + 48 * 4;
    bars = talk + talk_heads * 16 * 4;
    total = bars + (2 * kGwMaxStages + 1) * 8;
  }
};

// untiled copy of one cache row; both addresses and the size are multiples of 16 bytes
__device__ __forceinline__ void gw_copy_row(void* dst, const void* src, uint32_t bytes, uint64_t* bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(smem_u32(dst)),
               "l"(reinterpret_cast<uint64_t>(src)), "r"(bytes), "r"(smem_u32(bar))
               : "memory");
}
__device__ __forceinline__ void ldsm_x2(uint32_t (&r)[2], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0, %1}, [%2];" : "=r"(r[0]), "=r"(r[1]) : "r"(addr));
}

__device__ __forceinline__ void gw_sync() { asm volatile("bar.sync 1, %0;" ::"n"(kGwThreads) : "memory"); }

// NC: 16-column value pieces per warp; KQ: query fragments in registers (steps of 16 features per share), 0: in shared memory
template <int KT, int NC, int KQ>
__global__ void __launch_bounds__(kGwThreads + 32)
gqa_decode_wide_kernel(const GwParams p) {
  constexpr int kNt = KT / 8, kShares = 8 / kNt;   // 8-key columns of the score tile, feature shares
  pdl_launch_dependents();
  extern __shared__ __align__(128) uint8_t gw_sm[];
  const int tile_bytes = KT * p.pitch;
  const GwLayout at(p.key_width, p.stages * tile_bytes, KT, p.talk ? p.heads : 0);
  __nv_bfloat16* q_s = reinterpret_cast<__nv_bfloat16*>(gw_sm + at.q);
  float* part_s = reinterpret_cast<float*>(gw_sm + at.part);               // [kShares][16][KT + 1]
  __nv_bfloat16* prob_s = reinterpret_cast<__nv_bfloat16*>(gw_sm + at.prob);   // [16][KT + 8]
  float* f_s = reinterpret_cast<float*>(gw_sm + at.factor);                // [16] rescale factors
  float* c_m = f_s + 16;
  float* c_l = c_m + 16;
  float* talk_s = reinterpret_cast<float*>(gw_sm + at.talk);                // [heads][16]: shares of this block's heads
  uint64_t* full = reinterpret_cast<uint64_t*>(gw_sm + at.bars);
  uint64_t* empty = full + kGwMaxStages;
  volatile uint32_t* abort_flag = reinterpret_cast<volatile uint32_t*>(empty + kGwMaxStages);

  const int r = blockIdx.x, split = blockIdx.y, splits = gridDim.y, h0 = blockIdx.z * 16, nh = min(16, p.heads - h0);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g4 = lane >> 2, t4 = lane & 3;
  const int seq = p.row_seq[r], pos = p.row_pos[r], per = p.heads / p.kv_heads;
  int lo = 0, hi = 0, first = 0, kept = 0, n_keys = 0;                     // lo, hi: indices into the visible keys
  long long mean_row = 0;
  if (seq < 0 || seq >= p.num_seqs) {
    if (tid == 0) report_status(p.status, kStatusBadIndex, 0xE80, r, seq);
  } else if (pos >= 0) {
    first = p.span.first(pos);
    kept = p.span.head(pos);
    if (p.span.pool > 0 && kept > 0) {
      mean_row = p.pooled.first(seq);
      if (mean_row < 0 || kept > p.pooled.stride) {
        if (tid == 0) report_status(p.status, kStatusBadIndex, 0xE82, r, seq);
        kept = 0;
      }
    }
    n_keys = kept + max(min(pos + 1, p.max_blocks * p.page_size) - first, 0);
    const int tiles = (n_keys + KT - 1) / KT, share = (tiles + splits - 1) / splits;
    lo = min(split * share * KT, n_keys);
    hi = min(lo + share * KT, n_keys);
  }
  const int n_tiles = (hi - lo + KT - 1) / KT;
  // columns of this block's keys
  const int g0 = p.own_keys > 0 ? h0 / per : 0;
  const int width = p.own_keys > 0 ? ((h0 + nh - 1) / per - g0 + 1) * p.own_keys : p.key_width;
  auto token = [&](int i) { return i < kept ? i : first + i - kept; };
  if (p.talk)
    for (int i = tid; i < p.heads * 16; i += blockDim.x)
      talk_s[i] = (i & 15) < nh ? p.talk[static_cast<long long>(i >> 4) * p.heads + h0 + (i & 15)] : 0.f;
  if (tid == 0) {
    for (int i = 0; i < p.stages; ++i) {
      mbar_init(full + i, 1);
      mbar_init(empty + i, 8);
    }
    *abort_flag = 0;
    fence_barrier_init();
  }
  __syncthreads();
  const int vcols = (p.vdim_pad + 15) / 16, n_cols = p.kv_heads * vcols;
  float o[NC][2][4];
#pragma unroll
  for (int c = 0; c < NC; ++c)
#pragma unroll
    for (int n = 0; n < 2; ++n) o[c][n][0] = o[c][n][1] = o[c][n][2] = o[c][n][3] = 0.f;
  if (warp == 8) {
    // a token per lane; places past the last key repeat it (their probability is zero, their values must be finite)
    const long long n_pages = p.pool_rows / p.page_size;
    bool waited = false, ok = true;
    int asked = 0;
    for (; asked < n_tiles; ++asked) {
      const int st = asked % p.stages;
      // tiles that end below the row's own position were written by earlier steps
      if (!waited && !(p.early && asked < p.stages && lo + (asked + 1) * KT < n_keys)) {
        pdl_wait();
        waited = true;
      }
      long long slot = 0;
      const __nv_bfloat16* rows = p.pool;
      const int key = min(lo + asked * KT + lane, hi - 1);
      if (lane < KT && p.span.pool > 0 && key < kept) {
        rows = p.pooled.base;
        slot = mean_row + key;
      } else if (lane < KT) {
        const int t = token(key);
        const int page = p.block_table[static_cast<long long>(seq) * p.max_blocks + t / p.page_size];
        if (page >= 0 && page < n_pages) slot = static_cast<long long>(page) * p.page_size + t % p.page_size;
        else report_status(p.status, kStatusBadIndex, 0xE81, seq, t);
      }
      if (asked >= p.stages) {
        ok = mbar_wait(empty + st, (asked / p.stages - 1) & 1, abort_flag, p.status, 0xE91);
        ok = __all_sync(0xffffffffu, ok);
        if (!ok) break;
      }
      // fewer keys than there is room for: whole k-steps (queries are zero in the columns that follow, values have to be finite)
      const uint32_t key_bytes = (width < p.key_width ? (width + 15) / 16 * 16 : width) * 2;
      const uint32_t value_bytes = p.row_bytes - p.key_width * 2;
      if (lane == 0) mbar_arrive_expect_tx(full + st, KT * (key_bytes + value_bytes));
      __syncwarp();
      if (lane < KT) {
        uint8_t* dst = gw_sm + st * tile_bytes + lane * p.pitch;
        const __nv_bfloat16* src = rows + slot * p.pool_ld;
        if (width == p.v_offset) {
          gw_copy_row(dst, src, key_bytes + value_bytes, full + st);
        } else {
          gw_copy_row(dst, src + g0 * p.own_keys, key_bytes, full + st);
          gw_copy_row(dst + p.key_width * 2, src + p.v_offset, value_bytes, full + st);
        }
      }
    }
    if (!waited) pdl_wait();
    if (*abort_flag) {
      // copies may be in flight, and neither the merge nor the exit may happen under them
      for (int i = max(asked - p.stages, 0); i < asked; ++i) {
        const uint64_t t0 = globaltimer_ns();
        while (!mbar_try_wait(full + i % p.stages, (i / p.stages) & 1) && globaltimer_ns() - t0 < 2000000ull) {
        }
      }
    }
  } else {
    pdl_wait();
    // query rows of this block; rows past the last head and columns past the width are zeros
    for (int i = tid; i < 16 * (at.q_pitch / 8); i += kGwThreads) {
      const int row = i / (at.q_pitch / 8), c = (i - row * (at.q_pitch / 8)) * 8;
      uint4 v = make_uint4(0u, 0u, 0u, 0u);
      if (p.own_keys > 0) {
        const int e = c - ((h0 + row) / per - g0) * p.own_keys;
        if (row < nh && e >= 0 && e < p.own_keys)
          v = *reinterpret_cast<const uint4*>(p.q + r * p.ldq + static_cast<long long>(h0 + row) * p.own_keys + e);
      } else if (row < nh && c < p.key_width) {
        v = *reinterpret_cast<const uint4*>(p.q + r * p.ldq + static_cast<long long>(h0 + row) * p.key_width + c);
      }
      *reinterpret_cast<uint4*>(q_s + row * at.q_pitch + c) = v;
    }
    float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f}, sl[2];         // rows 2 warp, 2 warp + 1
#pragma unroll
    for (int k = 0; k < 2; ++k) {
      const int row = 2 * warp + k;
      sl[k] = p.slopes && row < nh ? p.slopes[h0 + row] * 1.4426950408889634f : 0.f;
    }
    const int ksteps = (width + 15) / 16, share = (ksteps + kShares - 1) / kShares;
    const int nt = warp % kNt, part = warp / kNt, k0 = min(part * share, ksteps), k1 = min(k0 + share, ksteps);
    const uint32_t qa = smem_u32(q_s + (lane & 15) * at.q_pitch + (lane >> 4) * 8);
    gw_sync();
    uint32_t qf[KQ > 0 ? KQ : 1][4];
    if constexpr (KQ > 0) {
#pragma unroll
      for (int k = 0; k < KQ; ++k) {
        qf[k][0] = qf[k][1] = qf[k][2] = qf[k][3] = 0u;
        if (k0 + k < k1) ldsm_x4(qf[k], qa + (k0 + k) * 32);
      }
    }
    for (int i = 0; i < n_tiles; ++i) {
      const uint8_t* tile = gw_sm + (i % p.stages) * tile_bytes;
      // a wait that gives up leaves its mark in the status word; the loop goes on so that the barriers stay in step
      mbar_wait(full + i % p.stages, (i / p.stages) & 1, abort_flag, p.status, 0xE90);
      {
        float s0[4] = {}, s1[4] = {};
        const uint32_t kr = smem_u32(tile + (nt * 8 + (lane & 7)) * p.pitch) + k0 * 32;
        const uint32_t ka = kr + (lane >> 3) * 16;                         // two steps of 16 features
        if constexpr (KQ > 0) {
#pragma unroll
          for (int k = 0; k < KQ; k += 2) {
            if (k0 + k + 1 < k1) {
              uint32_t b[4];
              ldsm_x4(b, ka + k * 32);
              mma_bf16_16816(s0, qf[k], b[0], b[1]);
              mma_bf16_16816(s1, qf[k + 1], b[2], b[3]);
            } else if (k0 + k < k1) {
              uint32_t b[2];
              ldsm_x2(b, kr + ((lane >> 3) & 1) * 16 + k * 32);
              mma_bf16_16816(s0, qf[k], b[0], b[1]);
            }
          }
        } else {
          int k = 0;
          for (; k0 + k + 1 < k1; k += 2) {
            uint32_t a0[4], a1[4], b[4];
            ldsm_x4(b, ka + k * 32);
            ldsm_x4(a0, qa + (k0 + k) * 32);
            ldsm_x4(a1, qa + (k0 + k) * 32 + 32);
            mma_bf16_16816(s0, a0, b[0], b[1]);
            mma_bf16_16816(s1, a1, b[2], b[3]);
          }
          if (k0 + k < k1) {
            uint32_t a0[4], b[2];
            ldsm_x2(b, kr + ((lane >> 3) & 1) * 16 + k * 32);
            ldsm_x4(a0, qa + (k0 + k) * 32);
            mma_bf16_16816(s0, a0, b[0], b[1]);
          }
        }
        float* dst = part_s + (part * 16 + g4) * (KT + 1) + nt * 8 + t4 * 2;
        dst[0] = s0[0] + s1[0];
        dst[1] = s0[1] + s1[1];
        dst[8 * (KT + 1)] = s0[2] + s1[2];
        dst[8 * (KT + 1) + 1] = s0[3] + s1[3];
      }
      gw_sync();
      const int key = lo + i * KT + lane;
      const bool seen = lane < KT && key < hi;
      const float dist = static_cast<float>(pos - token(min(key, hi - 1)));
      float x[2], w[2];
#pragma unroll
      for (int k = 0; k < 2; ++k) {
        const int row = 2 * warp + k;
        x[k] = -INFINITY;
        if (seen) {
          float s = 0.f;
#pragma unroll
          for (int q = 0; q < kShares; ++q) s += part_s[(q * 16 + row) * (KT + 1) + lane];
          // tanh as 1 - 2 / (exp(2 x) + 1)
          if (p.cap_log2 > 0.f) s = fmaf(p.cap_log2, -2.f * __fdividef(1.f, exp2f(s * p.cap_in) + 1.f), p.cap_log2);
          else s *= p.scale_log2;
          x[k] = fmaf(-sl[k], dist, s);
        }
      }
      float mx0 = x[0], mx1 = x[1];
#pragma unroll
      for (int d = 16; d > 0; d >>= 1) {
        mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, d));
        mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, d));
      }
#pragma unroll
      for (int k = 0; k < 2; ++k) {
        const int row = 2 * warp + k;
        const float mn = fmaxf(m[k], k == 0 ? mx0 : mx1);                   // finite: a tile has at least one visible key
        const float f = exp2f(m[k] - mn);
        w[k] = seen ? exp2f(x[k] - mn) : 0.f;
        m[k] = mn;
        l[k] *= f;
        if (lane < KT) prob_s[row * (KT + 8) + lane] = __float2bfloat16_rn(w[k]);
        if (lane == 0) f_s[row] = f;
      }
      gw_sync();
      const float f0 = f_s[g4], f1 = f_s[g4 + 8];
      uint32_t pf[KT / 16][4];
#pragma unroll
      for (int k = 0; k < KT / 16; ++k) ldsm_x4(pf[k], smem_u32(prob_s + (lane & 15) * (KT + 8) + k * 16 + (lane >> 4) * 8));
#pragma unroll
      for (int c = 0; c < NC; ++c) {
        const int col = warp + 8 * c;
        if (col < n_cols) {
          const int g = col / vcols, d = (col - g * vcols) * 16;
#pragma unroll
          for (int n = 0; n < 2; ++n) {
            o[c][n][0] *= f0;
            o[c][n][1] *= f0;
            o[c][n][2] *= f1;
            o[c][n][3] *= f1;
          }
          // matrices (transposed): keys 0-7 / 8-15 x columns 0-7, then columns 8-15
          const uint32_t va = smem_u32(tile + ((lane >> 3 & 1) * 8 + (lane & 7)) * p.pitch) +
                              (p.key_width + g * p.vdim_pad + d + (lane >> 4) * 8) * 2;
#pragma unroll
          for (int k = 0; k < KT / 16; ++k) {
            uint32_t b[4];
            ldsm_x4_t(b, va + k * 16 * p.pitch);
            mma_bf16_16816(o[c][0], pf[k], b[0], b[1]);
            mma_bf16_16816(o[c][1], pf[k], b[2], b[3]);
          }
        }
      }
      __syncwarp();
      if (lane == 0) mbar_arrive(empty + i % p.stages);
      // the row sums, off the path to the values
#pragma unroll
      for (int d = 16; d > 0; d >>= 1) {
        w[0] += __shfl_xor_sync(0xffffffffu, w[0], d);
        w[1] += __shfl_xor_sync(0xffffffffu, w[1], d);
      }
      l[0] += w[0];
      l[1] += w[1];
    }
    if (lane == 0) {
#pragma unroll
      for (int k = 0; k < 2; ++k) {
        c_m[2 * warp + k] = m[k];
        c_l[2 * warp + k] = l[k];
      }
    }
  }
  __syncthreads();                                                         // the tiles' memory now holds the outputs
  const int o_pitch = (p.talk ? n_cols : vcols) * 16 + 4;
  float* o_s = reinterpret_cast<float*>(gw_sm);                            // [16][o_pitch]
#pragma unroll
  for (int c = 0; c < NC; ++c) {
    const int col = warp + 8 * c;
    if (col >= n_cols || warp == 8) break;
    const int g = col / vcols, d = (col - g * vcols) * 16 + t4 * 2;
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int row = g4 + 8 * half;
      if (row >= nh || (!p.talk && (h0 + row) / per != g)) continue;
      const int at = row * o_pitch + (p.talk ? g * vcols * 16 : 0) + d;
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        o_s[at + n * 8] = o[c][n][2 * half];
        o_s[at + n * 8 + 1] = o[c][n][2 * half + 1];
      }
    }
  }
  const bool cluster = splits > 1 || (p.talk && p.head_blocks > 1);
  if (cluster) cluster_sync_all();
  else __syncthreads();
  const int quads = p.vdim_pad / 4;
  if (p.talk) {
    // Mixing is linear, so every CTA mixes what it has - its rows and its keys, weighted as the whole row's softmax says - and
    // the cluster adds these up.
    const int z = static_cast<int>(blockIdx.z), all = n_cols * 4, ctas = splits * p.head_blocks;
    if (tid < 16 && splits > 1) {
      float mm = -INFINITY, ll = 0.f;
      for (int s = 0; s < splits; ++s) mm = fmaxf(mm, ld_cluster_f32(mapa_shared(smem_u32(c_m + tid), s + z * splits)));
      for (int s = 0; s < splits; ++s) {
        const float ms = ld_cluster_f32(mapa_shared(smem_u32(c_m + tid), s + z * splits));
        ll = fmaf(ms == -INFINITY ? 0.f : exp2f(ms - mm), ld_cluster_f32(mapa_shared(smem_u32(c_l + tid), s + z * splits)), ll);
      }
      f_s[tid] = c_m[tid] == -INFINITY || !(ll > 0.f) ? 0.f : exp2f(c_m[tid] - mm) / ll;
    } else if (tid < 16) {
      f_s[tid] = c_l[tid] > 0.f ? 1.f / c_l[tid] : 0.f;
    }
    __syncthreads();
    for (int i = tid; i < p.heads * 16; i += blockDim.x) talk_s[i] *= (i & 15) < nh ? f_s[i & 15] : 0.f;
    __syncthreads();
    float* mix_s = o_s + 16 * o_pitch;                                     // [per][all columns]
    for (int i = tid; i < per * all; i += blockDim.x) {
      const int j = i / all, col = (i - j * all) * 4, h = col / (vcols * 16) * per + j;
      const float* t = talk_s + h * 16;
      float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
      for (int row = 0; row < nh; ++row) {
        const float4 v = *reinterpret_cast<const float4*>(o_s + row * o_pitch + col);
        const float w = t[row];
        a.x = fmaf(w, v.x, a.x);
        a.y = fmaf(w, v.y, a.y);
        a.z = fmaf(w, v.z, a.z);
        a.w = fmaf(w, v.w, a.w);
      }
      *reinterpret_cast<float4*>(mix_s + j * all * 4 + col) = a;
    }
    if (cluster) cluster_sync_all();
    else __syncthreads();
    for (int i = tid + (split + z * splits) * blockDim.x; i < p.heads * quads; i += blockDim.x * ctas) {
      const int h = i / quads, d = (i - h * quads) * 4, c = h / per;
      const float* src = mix_s + (h - c * per) * all * 4 + c * vcols * 16 + d;
      float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
      if (!cluster) {
        a = *reinterpret_cast<const float4*>(src);
      } else {
        for (int k = 0; k < ctas; ++k) {
          const float4 v = ld_cluster_f32x4(mapa_shared(smem_u32(src), k));
          a.x += v.x;
          a.y += v.y;
          a.z += v.z;
          a.w += v.w;
        }
      }
      __nv_bfloat16* dst = p.out + r * p.ldo + static_cast<long long>(h) * p.vdim_pad + d;
      *reinterpret_cast<__nv_bfloat162*>(dst) = __floats2bfloat162_rn(a.x, a.y);
      *reinterpret_cast<__nv_bfloat162*>(dst + 2) = __floats2bfloat162_rn(a.z, a.w);
    }
    if (cluster) cluster_sync_all();                                       // no CTA leaves while a peer reads its rows
    return;
  }
  // columns d .. d + 3 of a row's normalised output over all splits
  auto merged = [&](int row, int d) {
    float mm = -INFINITY, ll = 0.f;
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
    if (splits == 1) {
      ll = c_l[row];
      a = *reinterpret_cast<const float4*>(o_s + row * o_pitch + d);
    } else {
      for (int s = 0; s < splits; ++s) mm = fmaxf(mm, ld_cluster_f32(mapa_shared(smem_u32(c_m + row), s)));
      for (int s = 0; s < splits; ++s) {
        const float ms = ld_cluster_f32(mapa_shared(smem_u32(c_m + row), s));
        const float f = ms == -INFINITY ? 0.f : exp2f(ms - mm);
        ll = fmaf(f, ld_cluster_f32(mapa_shared(smem_u32(c_l + row), s)), ll);
        const float4 v = ld_cluster_f32x4(mapa_shared(smem_u32(o_s + row * o_pitch + d), s));
        a.x = fmaf(f, v.x, a.x);
        a.y = fmaf(f, v.y, a.y);
        a.z = fmaf(f, v.z, a.z);
        a.w = fmaf(f, v.w, a.w);
      }
    }
    const float inv = ll > 0.f ? 1.f / ll : 0.f;
    return make_float4(a.x * inv, a.y * inv, a.z * inv, a.w * inv);
  };
  for (int i = tid + split * blockDim.x; i < nh * quads; i += blockDim.x * splits) {
    const int h = i / quads, d = (i - h * quads) * 4;
    float4 a = merged(h, d);
    const long long col = static_cast<long long>(h0 + h) * p.vdim_pad + d;
    if (p.gate) {
      const __nv_bfloat162* z = reinterpret_cast<const __nv_bfloat162*>(p.gate + r * p.ldg + col);
      const float2 z0 = __bfloat1622float2(z[0]), z1 = __bfloat1622float2(z[1]);
      a = make_float4(a.x * sigmoid_f(z0.x), a.y * sigmoid_f(z0.y), a.z * sigmoid_f(z1.x), a.w * sigmoid_f(z1.y));
    }
    __nv_bfloat16* dst = p.out + r * p.ldo + col;
    *reinterpret_cast<__nv_bfloat162*>(dst) = __floats2bfloat162_rn(a.x, a.y);
    *reinterpret_cast<__nv_bfloat162*>(dst + 2) = __floats2bfloat162_rn(a.z, a.w);
  }
  if (cluster) cluster_sync_all();                                         // no CTA leaves while a peer reads its rows
}

// tile size and stages for a cache row of this shape; kt 0: it does not fit
struct GwPlan {
  int kt, stages, nc, kq;
};
static GwPlan gw_plan(int key_width, int kv_heads, int vdim_pad, bool shared_values, int heads) {
  const int vcols = (vdim_pad + 15) / 16, cols = kv_heads * vcols, pitch = (key_width + kv_heads * vdim_pad) * 2 + 16;
  const int nc = cols <= 8 ? 1 : cols <= 16 ? 2 : cols <= 32 ? 4 : cols <= 64 ? 8 : 0;
  for (int kt = 32; kt >= 16 && nc; kt /= 2) {
    int stages = (kGwSmemLimit - GwLayout(key_width, 0, kt, shared_values ? heads : 0).total) / (kt * pitch);
    if (stages > kGwMaxStages) stages = kGwMaxStages;
    // the outputs reuse the tiles' memory: with shared values all columns, and the mixed ones of every head
    const long long outputs = 16LL * ((shared_values ? cols : vcols) * 16 + 4) * 4 + (shared_values ? 64LL * heads * vcols : 0);
    if (stages < 2 || stages * kt * pitch < outputs) continue;
    const int shares = 64 / kt, steps = ((key_width + 15) / 16 + shares - 1) / shares;
    return {kt, stages, nc, steps <= 4 ? 4 : steps <= 16 ? 16 : 0};
  }
  return {0, 0, 0, 0};
}

template <int KT, int NC, int KQ>
static int launch_gw(const GwParams& p, int rows, int splits, cudaStream_t stream) {
  static bool attr_set = false;
  if (!attr_set) {
    if (cudaFuncSetAttribute(gqa_decode_wide_kernel<KT, NC, KQ>, cudaFuncAttributeMaxDynamicSharedMemorySize, kGwSmemLimit) != cudaSuccess)
      return FB_ERR_LAUNCH;
    attr_set = true;
  }
  cudaLaunchConfig_t cfg{};
  cfg.gridDim = dim3(rows, splits, p.head_blocks);
  cfg.blockDim = dim3(kGwThreads + 32);
  cfg.dynamicSmemBytes = GwLayout(p.key_width, p.stages * KT * p.pitch, KT, p.talk ? p.heads : 0).total;
  cfg.stream = stream;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = 1;
  attr[0].val.clusterDim.y = splits;
  attr[0].val.clusterDim.z = p.talk ? p.head_blocks : 1;
  attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[1].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr;
  cfg.numAttrs = pdl_enabled() ? 2 : 1;
  if (cudaLaunchKernelEx(&cfg, gqa_decode_wide_kernel<KT, NC, KQ>, p) != cudaSuccess) return FB_ERR_LAUNCH;
  return cudaGetLastError() == cudaSuccess ? FB_OK : FB_ERR_LAUNCH;
}
template <int KT, int NC>
static int launch_gw_steps(const GwParams& p, int kq, int rows, int splits, cudaStream_t s) {
  if (kq == 4) return launch_gw<KT, NC, 4>(p, rows, splits, s);
  if (kq == 16) return launch_gw<KT, NC, 16>(p, rows, splits, s);
  return launch_gw<KT, NC, 0>(p, rows, splits, s);
}
template <int KT>
static int launch_gw_cols(const GwParams& p, const GwPlan& plan, int rows, int splits, cudaStream_t s) {
  if (plan.nc == 1) return launch_gw_steps<KT, 1>(p, plan.kq, rows, splits, s);
  if (plan.nc == 2) return launch_gw_steps<KT, 2>(p, plan.kq, rows, splits, s);
  if (plan.nc == 4) return launch_gw_steps<KT, 4>(p, plan.kq, rows, splits, s);
  return launch_gw_steps<KT, 8>(p, plan.kq, rows, splits, s);
}

}  // namespace fb

using namespace fb;

// key columns of a CTA: of the most kv heads that a block of 16 heads has, when query rows meet their own kv head's keys
static int gw_key_width(int key_width, int own_keys, int heads, int kv_heads) {
  if (!own_keys) return key_width;
  int most = 0;
  for (int h0 = 0, per = heads / kv_heads; h0 < heads; h0 += 16) {
    const int last = (h0 + 16 < heads ? h0 + 16 : heads) - 1, n = last / per - h0 / per + 1;
    if (n > most) most = n;
  }
  return most * key_width;
}

extern "C" int fb_gqa_decode_wide_ok(int key_width, int kv_heads, int vdim_pad, int shared_values, int heads, int own_keys) {
  if (kv_heads <= 0 || heads <= 0 || heads % kv_heads) return 0;
  if (shared_values && (heads + 15) / 16 > 8) return 0;       // the row's head blocks form one cluster
  key_width = gw_key_width(key_width, own_keys, heads, kv_heads);
  return key_width > 0 && key_width % 8 == 0 && kv_heads > 0 && vdim_pad > 0 && vdim_pad % 8 == 0 &&
         gw_plan(key_width, kv_heads, vdim_pad, shared_values != 0, heads).kt > 0;
}

extern "C" int fb_gqa_decode_wide(const FbGqaArgs* a, int splits, int early, void* stream) {
  if (!a || !a->q || !a->pool || !a->out || !a->block_table || !a->row_seq || !a->row_pos || a->fp32) return FB_ERR_SHAPE;
  if (a->rows <= 0 || a->heads <= 0 || a->kv_heads <= 0 || a->heads % a->kv_heads || a->vdim_pad <= 0 || a->vdim_pad % 8 ||
      a->pool_rows <= 0 || a->pool_ld % 8 || a->num_seqs <= 0 || a->max_blocks <= 0 || a->page_size <= 0)
    return FB_ERR_SHAPE;
  // the keys, the values, or both are shared by all query rows
  const bool shared_values = a->value_stride == 0;
  const long long key_width = a->key_stride ? static_cast<long long>(a->kv_heads) * a->key_width : a->key_width;
  if (!gqa_form_ok(a) || a->maps != 1 || (a->key_stride != 0 && !shared_values) || key_width > 16384 ||
      a->v_offset != key_width || a->ldq % 8 || a->ldo % 4 || a->ldg % 4 || shared_values != (a->talk != nullptr) ||
      (shared_values && a->gate))
    return FB_ERR_SHAPE;
  if (shared_values && (a->heads + 15) / 16 * splits > 8) return FB_ERR_LIMIT;
  if (splits != 1 && splits != 2 && splits != 4 && splits != 8) return FB_ERR_SHAPE;
  const uintptr_t bits = reinterpret_cast<uintptr_t>(a->q) | reinterpret_cast<uintptr_t>(a->pool) |
                         reinterpret_cast<uintptr_t>(a->out) | reinterpret_cast<uintptr_t>(a->gate) |
                         reinterpret_cast<uintptr_t>(a->pooled);
  if (bits & 15) return FB_ERR_ALIGN;
  const int cta_width = gw_key_width(a->key_width, a->key_stride, a->heads, a->kv_heads);
  const GwPlan plan = gw_plan(cta_width, a->kv_heads, a->vdim_pad, shared_values, a->heads);
  if (plan.kt == 0) return FB_ERR_LIMIT;
  GwParams p{};
  p.q = static_cast<const __nv_bfloat16*>(a->q); p.ldq = a->ldq;
  p.pool = static_cast<const __nv_bfloat16*>(a->pool); p.pool_rows = a->pool_rows; p.pool_ld = a->pool_ld;
  p.block_table = a->block_table; p.row_seq = a->row_seq; p.row_pos = a->row_pos;
  p.num_seqs = a->num_seqs; p.max_blocks = a->max_blocks; p.page_size = a->page_size;
  p.span = key_span(a);
  p.pooled = pooled_rows<__nv_bfloat16>(a);
  p.talk = a->talk;
  p.own_keys = a->key_stride ? a->key_width : 0;
  p.scale_log2 = a->scale * 1.4426950408889634f;
  if (a->softcap > 0.f) {
    p.cap_log2 = a->softcap * 1.4426950408889634f;
    p.cap_in = 2.f * p.scale_log2 / a->softcap;
  }
  p.slopes = a->slopes; p.gate = static_cast<const __nv_bfloat16*>(a->gate); p.ldg = a->ldg;
  p.out = static_cast<__nv_bfloat16*>(a->out); p.ldo = a->ldo;
  p.heads = a->heads; p.kv_heads = a->kv_heads; p.key_width = cta_width; p.v_offset = a->v_offset; p.vdim_pad = a->vdim_pad;
  p.row_bytes = (p.key_width + a->kv_heads * a->vdim_pad) * 2;
  p.pitch = p.row_bytes + 16;
  p.stages = plan.stages;
  p.head_blocks = (a->heads + 15) / 16;
  p.early = early;
  p.status = static_cast<DeviceStatus*>(a->status);
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  return plan.kt == 32 ? launch_gw_cols<32>(p, plan, a->rows, splits, s) : launch_gw_cols<16>(p, plan, a->rows, splits, s);
}
