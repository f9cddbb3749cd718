// Prefill attention of grouped-query layers inside position chunks or sliding windows on the 5th-generation tensor cores,
// bf16.
//
// CTA = one tile of consecutive query positions of one sequence x the query heads of one key / value head (with two score
// maps per head: both maps' rows): up to 128 (position, row) rows, P = 128 / rows-per-group positions.  Keys are taken in
// tiles of 64 tokens at absolute positions 64 j: the tiles with kept first tokens (or tiles of 64 mean rows of the blocks before
// the window, gqa_mask.cuh), then from the first tile that holds a key of the first position's chunk or window.  Query rows that
// meet the values of all kv heads take them in slices of up to 256 columns, a CTA each.
//
//   TMA producer (warp 0): the query rows once (boxes of 64 features x group x P), then per token tile the feature blocks of
//     the keys and of the values straight from the paged pool (box = 64 features x min(page, 64) rows; features past the
//     head's width and rows past the sequence are zeros; one copy for all blocks when the width is a multiple of 64), two
//     stages each with their own barriers.  Wide keys (those of all kv heads side by side) come in pieces of `kb` feature
//     blocks, a stage each (two or four stages); query rows that do not fit in shared memory come with them, piece by piece,
//     for every token tile.
//   MMA issuer (warp 1): S[128 x 64] = Q K^T, both operands K-major in shared memory, double buffered in TMEM; O[128 x DV]
//     += P V with P in TMEM as the A operand and the value tile read as an MN-major B operand.  The next tile's S is issued
//     before the current P is waited for.
//   Softmax (warps 2..9, two threads per row with half of the tile's columns each): scores from TMEM, scale, distance bias or soft cap,
//     mask, running maximum (the halves meet in shared memory), exp2, bf16 P written over the score buffer.  The
//     accumulator is rescaled only when a row's maximum has grown by more than 2^8 since the reference it was scaled by;
//     the sum uses the same reference, so the result is exact up to rounding.  The difference of a head's two maps is
//     taken between neighbouring lanes, its RMS norm and the output gate on the way out.
//
// A row's result depends on the row and the cache contents, not on which rows share its tile or how a prompt was cut,
// beyond the rounding of a rescale that another row of its warp asked for.
// Every wait is bounded (status word, then teardown with TMEM freed); page ids are range-checked.
#include "act_type.cuh"
#include "attn_tc.cuh"
#include "common.cuh"
#include "f32x2.cuh"
#include "ferrule_b200.h"
#include "gqa_mask.cuh"
#include "launch.cuh"

namespace fb {

constexpr int kGpThreads = 320;
constexpr int kGpM = 128;
constexpr int kGpKv = 64;
constexpr int kGpQBlock = kGpM * 128;         // bytes of a 64-feature block of the query tile
constexpr int kGpKvBlock = kGpKv * 128;
constexpr int kGpSmemLimit = 227 * 1024;

struct GpParams {
  const int* tiles;          // [n_tiles, 4] = sequence, first query row, query rows, position of the first
  const int* block_table;
  __nv_bfloat16* out;
  long long ldo;
  DeviceStatus* status;
  long long pool_rows;
  int rows, heads, kv_heads, per;      // per: query rows of a key / value head
  int positions;             // positions per tile the query box holds
  int num_seqs, max_blocks, page_size, box_rows;
  KeySpan span;
  int key_width, value_width, qb, vb;  // qb, vb: 64-feature blocks of a query / key row and of a slice of a value row
  int shared_values;
  PooledRows<__nv_bfloat16> pooled;
  float cap_log2, cap_in;              // soft cap: score2 = cap_log2 tanh(raw * cap_in / 2)
  float cap_poly[6];                   // kGpBounded: coefficients of score2 in powers of (raw * cap_in / 2)^2, times that
  int kb, pieces, ks, q_resident;      // blocks per key stage, stages per token tile, key stages (2 or 4)
  int shared_keys, k_whole, v_whole;   // whole: one copy brings all feature blocks of a stage
  uint32_t tmem_cols;
  float scale_log2;
  const float* slopes;                 // [heads]
  const __nv_bfloat16* gate;
  long long ldg;
  int maps, vdim;
  float diff_lambda, diff_scale, eps;
};

constexpr float kLog2e = 1.4426950408889634f;
// What happens to the scores before the softmax.  kGpBounded: a soft cap where the caller bounds the score by 0.7 of the cap:
// tanh is then a polynomial (below), and as capped scores cannot leave [-cap, cap] no maximum is taken.
enum { kGpPlain = 0, kGpBias = 1, kGpCap = 2, kGpBounded = 3 };
constexpr float kGpMaxCap = 40.f;                      // exp(cap) times a long sum fits fp32 without a reference

// tanh(u) = u p(u^2) for |u| <= 0.7: p interpolates tanh(sqrt(w)) / sqrt(w) at the six Chebyshev nodes of [0, 0.49]
// (error below 1e-8, in fp32 below 1e-7)
constexpr float kTanhPoly[6] = {1.f, -0.33333128690719604f, 0.13328377902507782f, -0.053523916751146317f, 0.02001960761845112f,
                                -0.005084393545985222f};

__device__ __forceinline__ float rcp_ftz(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

template <int FORM>
__global__ void __launch_bounds__(kGpThreads, 2)
gqa_prefill_tc_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k,
                      const __grid_constant__ CUtensorMap map_v, const __grid_constant__ CUtensorMap map_pk,
                      const __grid_constant__ CUtensorMap map_pv, const GpParams p) {
  constexpr bool BIAS = FORM == kGpBias, READY = FORM != kGpPlain;      // READY: scores are scaled (base 2) before the mask
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int qb = p.qb, vb = p.vb;
  uint8_t* q_s = smem;
  uint8_t* k_s = q_s + (p.q_resident ? qb : p.ks * p.kb) * kGpQBlock;   // [ks][kb] blocks
  uint8_t* v_s = k_s + p.ks * p.kb * kGpKvBlock;         // [2][vb] blocks
  uint64_t* bars = reinterpret_cast<uint64_t*>(v_s + 2 * vb * kGpKvBlock);
  uint64_t* q_full = bars + 0;
  uint64_t* k_full = bars + 1;          // [4]
  uint64_t* v_full = bars + 5;          // [2]
  uint64_t* k_free = bars + 7;          // [4]
  uint64_t* v_free = bars + 11;         // [2]
  uint64_t* s_full = bars + 13;         // [2]
  uint64_t* p_full = bars + 15;         // [2]
  uint64_t* o_done = bars + 17;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 18);
  volatile uint32_t* abort_flag = reinterpret_cast<volatile uint32_t*>(bars + 19);
  // exchange between the two halves of a row: maxima [tile parity][half][row] (bf16, rounded up), after the loop sums [half][row]
  __nv_bfloat16* max_x = reinterpret_cast<__nv_bfloat16*>(bars + 20);
  float* sum_x = reinterpret_cast<float*>(bars + 20);
  const int k_mask = p.ks - 1, k_shift = p.ks == 4 ? 2 : 1;

  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int g = blockIdx.y;
  const int4 tile = reinterpret_cast<const int4*>(p.tiles)[blockIdx.x];
  const int seq = tile.x, row0 = tile.y, nrows = tile.z, pos0 = tile.w;
  if (seq < 0 || seq >= p.num_seqs || row0 < 0 || nrows <= 0 || nrows > p.positions || row0 + nrows > p.rows || pos0 < 0) {
    if (tid == 0) report_status(p.status, kStatusBadIndex, 0xA80, blockIdx.x, seq);
    return;
  }
  const int kv_len = min(pos0 + nrows, p.max_blocks * p.page_size);
  const int j0 = p.span.first(pos0) / kGpKv;                             // first token tile of the chunk or window
  int n_pre = (p.span.head(pos0 + nrows - 1) + kGpKv - 1) / kGpKv;       // tiles of mean rows, or of kept tokens before it
  if (p.span.pool == 0) n_pre = min(n_pre, j0);
  auto is_mean = [&](int j) { return p.span.pool > 0 && j < n_pre; };
  const int slice = blockIdx.z;
  const int n_kv = n_pre + (kv_len + kGpKv - 1) / kGpKv - j0;
  // with a distance bias the latest keys come first: a row's maximum is then mostly among them
  auto tile_of = [&](int j) {
    if (BIAS) j = n_kv - 1 - j;
    return j < n_pre ? j : j0 + j - n_pre;
  };
  if (n_kv <= 0) {
    if (tid == 0) report_status(p.status, kStatusBadIndex, 0xA81, blockIdx.x, pos0);
    return;
  }

  if (tid == 0) {
    mbar_init(q_full, 1);
    for (int i = 0; i < 4; ++i) {
      mbar_init(k_full + i, 1);
      mbar_init(k_free + i, 1);
    }
    for (int i = 0; i < 2; ++i) {
      mbar_init(v_full + i, 1);
      mbar_init(v_free + i, 1);
      mbar_init(s_full + i, 1);
      mbar_init(p_full + i, 8);
    }
    mbar_init(o_done, 1);
    *abort_flag = 0;
    fence_barrier_init();
    tma_prefetch_desc(&map_q);
    tma_prefetch_desc(&map_k);
    tma_prefetch_desc(&map_v);
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, p.tmem_cols);
    tmem_relinquish();
  }
  pdl_launch_dependents();
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot;
  const uint32_t col_s = static_cast<uint32_t>(vb * 64);                 // S0, S1 behind the accumulator; P over S
  pdl_wait();

  if (warp == 0) {
    // ------------------------------------------------------------------ TMA producer
    if (elect_one()) {
      const uint32_t q_block_tx = static_cast<uint32_t>(p.positions * p.per * 128);
      if (p.q_resident) {
        mbar_arrive_expect_tx(q_full, qb * q_block_tx);
        for (int b = 0; b < qb; ++b) tma_load_3d(q_s + b * kGpQBlock, &map_q, q_full, b * 64, g * p.per, row0);
      }
      const int subs = kGpKv / p.box_rows, key_head = p.shared_keys ? 0 : g, value_head = p.shared_values ? 0 : g;
      const int vblock0 = slice * vb;
      long long mean_row = 0;
      if (is_mean(0)) {
        mean_row = p.pooled.first(seq);
        if (mean_row < 0) {
          report_status(p.status, kStatusBadIndex, 0xA83, seq, pos0);
          mean_row = p.pooled.rows;                                      // out of range: the copies fill zeros
        }
      }
      const long long n_pages = p.pool_rows / p.page_size;
      const int* pages = p.block_table + static_cast<long long>(seq) * p.max_blocks;
      auto page_of = [&](int t0) { return t0 < kv_len ? pages[t0 / p.page_size] : -1; };
      auto row_of = [&](int t0, int page) {
        if (t0 < kv_len && page >= 0 && page < n_pages) return page * p.page_size + t0 % p.page_size;
        if (t0 < kv_len) report_status(p.status, kStatusBadIndex, 0xA82, seq, t0);
        return static_cast<int>(p.pool_rows);                            // out of range: the copy fills zeros
      };
      bool ok = true;
      int k_armed = 0, v_armed = 0;                                      // key stages / value tiles that were requested
      int next_page = is_mean(0) ? -1 : page_of(tile_of(0) * kGpKv);     // read a tile ahead
      for (int j = 0; j < n_kv && ok; ++j) {
        const int st = j & 1, tok = tile_of(j) * kGpKv;
        const bool mean = is_mean(j);
        const int row = mean ? static_cast<int>(min(mean_row + tok, p.pooled.rows)) : row_of(tok, next_page);   // of its first box
        if (j + 1 < n_kv && !is_mean(j + 1)) next_page = page_of(tile_of(j + 1) * kGpKv);
        auto sub_row = [&](int s) {
          if (mean) return row + s * p.box_rows;
          return s == 0 ? row : row_of(tok + s * p.box_rows, page_of(tok + s * p.box_rows));
        };
        const CUtensorMap* mk = mean ? &map_pk : &map_k;
        const CUtensorMap* mv = mean ? &map_pv : &map_v;
        for (int c = 0; c < p.pieces && ok; ++c) {
          const int i = j * p.pieces + c, ks = i & k_mask, b0 = c * p.kb, nb = min(p.kb, qb - b0);
          if (i >= p.ks) ok = mbar_wait(k_free + ks, ((i >> k_shift) - 1) & 1, abort_flag, p.status, 0xA90);
          if (!ok) break;
          mbar_arrive_expect_tx(k_full + ks, nb * (static_cast<uint32_t>(kGpKvBlock) + (p.q_resident ? 0u : q_block_tx)));
          uint8_t* dst = k_s + ks * p.kb * kGpKvBlock;
          if (p.k_whole) {
            tma_load_4d(dst, mk, k_full + ks, 0, row, b0, key_head);
          } else {
            for (int s = 0; s < subs; ++s) {
              const int rc = sub_row(s);
              for (int b = 0; b < nb; ++b)
                tma_load_3d(dst + b * kGpKvBlock + s * p.box_rows * 128, mk, k_full + ks, (b0 + b) * 64, key_head, rc);
            }
          }
          if (!p.q_resident)
            for (int b = 0; b < nb; ++b)
              tma_load_3d(q_s + (ks * p.kb + b) * kGpQBlock, &map_q, k_full + ks, (b0 + b) * 64, g * p.per, row0);
          k_armed = i + 1;
        }
        if (!ok) break;
        if (j > 1) ok = mbar_wait(v_free + st, ((j - 2) >> 1) & 1, abort_flag, p.status, 0xA91);
        if (!ok) break;
        mbar_arrive_expect_tx(v_full + st, static_cast<uint32_t>(vb * kGpKvBlock));
        if (p.v_whole) {
          tma_load_4d(v_s + st * vb * kGpKvBlock, mv, v_full + st, 0, row, vblock0, value_head);
        } else {
          for (int s = 0; s < subs; ++s) {
            const int rc = sub_row(s);
            for (int b = 0; b < vb; ++b)
              tma_load_3d(v_s + (st * vb + b) * kGpKvBlock + s * p.box_rows * 128, mv, v_full + st, (vblock0 + b) * 64,
                          value_head, rc);
          }
        }
        v_armed = j + 1;
      }
      // after an abort: copies of the last stages may still be in flight, and the CTA may not exit under them
      if (*abort_flag) {
        auto drain = [&](uint64_t* bar, uint32_t parity) {
          const uint64_t t0 = globaltimer_ns();
          while (!mbar_try_wait(bar, parity) && globaltimer_ns() - t0 < 2000000ull) {
          }
        };
        if (p.q_resident) drain(q_full, 0);
        for (int i = max(k_armed - p.ks, 0); i < k_armed; ++i) drain(k_full + (i & k_mask), (i >> k_shift) & 1);
        for (int j = max(v_armed - 2, 0); j < v_armed; ++j) drain(v_full + (j & 1), (j >> 1) & 1);
      }
    }
  } else if (warp == 1) {
    // ------------------------------------------------------------------ MMA issuer
    if (elect_one()) {
      const uint32_t q_addr = smem_u32(q_s), k_addr = smem_u32(k_s), v_addr = smem_u32(v_s);
      constexpr uint32_t idesc_qk = umma_idesc(kGpM, kGpKv, 1, 1);
      const uint32_t idesc_pv = umma_idesc(kGpM, static_cast<uint32_t>(vb * 64), 1, 1) | (1u << 16);   // B is MN-major
      const int ksteps = (p.key_width + 15) / 16;
      auto qk = [&](int j) {
        for (int c = 0; c < p.pieces; ++c) {
          const int i = j * p.pieces + c, st = i & k_mask, k0 = c * p.kb * 4, k1 = min(k0 + p.kb * 4, ksteps);
          if (!mbar_wait(k_full + st, (i >> k_shift) & 1, abort_flag, p.status, 0xAA2)) return false;
          tc_fence_after();
          const uint32_t ks = k_addr + st * p.kb * kGpKvBlock;
          const uint32_t qs = p.q_resident ? q_addr + c * p.kb * kGpQBlock : q_addr + st * p.kb * kGpQBlock;
          // one thread issues everything: descriptors are advanced (16-byte units), not rebuilt
          uint64_t dq = umma_desc_k128(qs), dk = umma_desc_k128(ks);
          const uint32_t d = tmem + col_s + (j & 1) * kGpKv;
          int k = k0;
          for (; k + 4 <= k1; k += 4) {
#pragma unroll
            for (int e = 0; e < 4; ++e) umma_bf16(d, dq + 2 * e, dk + 2 * e, idesc_qk, (k > 0 || e > 0) ? 1u : 0u);
            dq += kGpQBlock >> 4;
            dk += kGpKvBlock >> 4;
          }
          for (int e = 0; k < k1; ++k, ++e) umma_bf16(d, dq + 2 * e, dk + 2 * e, idesc_qk, k > 0 ? 1u : 0u);
          if (c + 1 == p.pieces) umma_commit(s_full + (j & 1));
          umma_commit(k_free + st);
        }
        return true;
      };
      bool ok = !p.q_resident || mbar_wait(q_full, 0, abort_flag, p.status, 0xAA0);
      if (ok) {
        tc_fence_after();
        ok = qk(0);
      }
      for (int j = 0; j < n_kv && ok; ++j) {
        const uint32_t ph = (j >> 1) & 1;
        if (j + 1 < n_kv) {
          // the score buffer of tile j + 1 held P of tile j - 1, whose product was issued before
          ok = qk(j + 1);
          if (!ok) break;
        }
        ok = mbar_wait(v_full + (j & 1), ph, abort_flag, p.status, 0xAA3);
        if (ok) ok = mbar_wait(p_full + (j & 1), ph, abort_flag, p.status, 0xAA4);
        if (!ok) break;
        tc_fence_after();
        const uint64_t dv = umma_desc_mn128(v_addr + (j & 1) * vb * kGpKvBlock, kGpKvBlock);
#pragma unroll
        for (int k = 0; k < 4; ++k)
          umma_bf16_ts(tmem, tmem + col_s + (j & 1) * kGpKv + (k >> 1) * 32 + (k & 1) * 8, dv + k * (2048 >> 4), idesc_pv, (j > 0 || k > 0) ? 1u : 0u);
        umma_commit(v_free + (j & 1));
        if (j + 1 == n_kv) umma_commit(o_done);
      }
    }
  } else {
    // ------------------------------------------------------------------ softmax + epilogue: two threads per row
    const int quarter = warp & 3, half = (warp - 2) >> 2;
    const int r = quarter * 32 + lane;
    const int at = r / p.per, head = (g * p.per + r - at * p.per) / p.maps;
    const bool valid = at < nrows;
    const int pos = pos0 + at;
    const int hi_tok = valid ? min(pos + 1, kv_len) : 0;
    const int lo_tok = p.span.first(pos), keep = p.span.keep, n_mean = valid && p.span.pool > 0 ? p.span.head(pos) : 0;
    const float slope = BIAS && valid ? p.slopes[head] * kLog2e : 0.f;
    const uint32_t lane_base = tmem + (static_cast<uint32_t>(quarter * 32) << 16);
    auto pair_sync = [&]() { asm volatile("bar.sync %0, 64;" ::"r"(quarter + 1) : "memory"); };
    float m_ref = -INFINITY, l_sum = 0.f;
    bool ok = true;
    for (int j = 0; j < n_kv; ++j) {
      const uint32_t s_t = lane_base + col_s + (j & 1) * kGpKv;
      // a wait that gives up leaves its mark in the status word; the loop goes on so that the barriers stay in step
      ok = mbar_wait(s_full + (j & 1), (j >> 1) & 1, abort_flag, p.status, 0xAB0) && ok;
      __syncwarp();
      tc_fence_after();
      uint32_t sv[2][16];
#pragma unroll
      for (int c = 0; c < 2; ++c) tmem_ld16(s_t + half * 32 + c * 16, sv[c]);
      tmem_ld_wait();
      const int tok0 = tile_of(j) * kGpKv + half * 32;
      const int lo = is_mean(j) ? 0 : lo_tok, hi = is_mean(j) ? n_mean : hi_tok;
      // four independent chains for the maximum and the sum, packed multiply-adds
      float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
      if (BIAS) {
        // the score in base 2 with its distance bias
        const float b0 = slope * static_cast<float>(tok0 - pos);
        const uint64_t sc2 = pack2(p.scale_log2, p.scale_log2), sl2 = pack2(slope, slope), b02 = pack2(b0, b0);
#pragma unroll
        for (int c = 0; c < 2; ++c)
#pragma unroll
          for (int i = 0; i < 16; i += 2) {
            const uint64_t bias = fma2(sl2, pack2(static_cast<float>(c * 16 + i), static_cast<float>(c * 16 + i + 1)), b02);
            float x0, x1;
            unpack2(fma2(pack2(__uint_as_float(sv[c][i]), __uint_as_float(sv[c][i + 1])), sc2, bias), x0, x1);
            sv[c][i] = __float_as_uint(x0);
            sv[c][i + 1] = __float_as_uint(x1);
          }
      }
      if (FORM == kGpCap) {
        // tanh as 1 - 2 / (exp(2 x) + 1)
        const float cap_in2 = p.cap_in * kLog2e;
#pragma unroll
        for (int c = 0; c < 2; ++c)
#pragma unroll
          for (int i = 0; i < 16; ++i)
            sv[c][i] = __float_as_uint(fmaf(-2.f * p.cap_log2, rcp_ftz(exp2_ftz(__uint_as_float(sv[c][i]) * cap_in2) + 1.f), p.cap_log2));
      }
      if (FORM == kGpBounded) {
        const uint64_t in2 = pack2(0.5f * p.cap_in, 0.5f * p.cap_in);
        uint64_t c2[6];
#pragma unroll
        for (int e = 0; e < 6; ++e) c2[e] = pack2(p.cap_poly[e], p.cap_poly[e]);
#pragma unroll
        for (int c = 0; c < 2; ++c)
#pragma unroll
          for (int i = 0; i < 16; i += 2) {
            const uint64_t u = mul2(pack2(__uint_as_float(sv[c][i]), __uint_as_float(sv[c][i + 1])), in2), w = mul2(u, u);
            uint64_t y = c2[5];
#pragma unroll
            for (int e = 4; e >= 0; --e) y = fma2(y, w, c2[e]);
            float x0, x1;
            unpack2(mul2(u, y), x0, x1);
            sv[c][i] = __float_as_uint(x0);
            sv[c][i + 1] = __float_as_uint(x1);
          }
      }
      if (__all_sync(0xffffffffu, tok0 + 32 <= hi && (tok0 >= lo || tok0 + 32 <= keep))) {
#pragma unroll
        for (int i = 0; i < 16; ++i)
#pragma unroll
          for (int c = 0; c < 2; ++c) mx4[2 * c + (i & 1)] = fmaxf(mx4[2 * c + (i & 1)], __uint_as_float(sv[c][i]));
      } else {
#pragma unroll
        for (int i = 0; i < 16; ++i)
#pragma unroll
          for (int c = 0; c < 2; ++c) {
            const int t = tok0 + c * 16 + i;
            const float x = ((t >= lo || t < keep) && t < hi) ? __uint_as_float(sv[c][i]) : -INFINITY;
            sv[c][i] = __float_as_uint(x);
            mx4[2 * c + (i & 1)] = fmaxf(mx4[2 * c + (i & 1)], x);
          }
      }
      if constexpr (FORM != kGpBounded) {
        float mx = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3]));
        if (!READY) mx *= p.scale_log2;                         // the scale is positive
        {
          // both halves see the same two rounded maxima; behind the barrier both have read their scores
          __nv_bfloat16* slot = max_x + (j & 1) * 256;
          const __nv_bfloat16 mine = __float2bfloat16_ru(mx);
          slot[half * 128 + r] = mine;
          tc_fence_before();
          pair_sync();
          tc_fence_after();
          mx = fmaxf(__bfloat162float(mine), __bfloat162float(slot[(half ^ 1) * 128 + r]));
        }
        const float m_new = fmaxf(m_ref, mx);
        if (j == 0) {
          m_ref = m_new;                                        // nothing accumulated yet
        } else if (__any_sync(0xffffffffu, m_new > m_ref + 8.f)) {
          // rescale this warp's share of 32 accumulator rows: the previous product must have retired
          ok = mbar_wait(v_free + ((j - 1) & 1), ((j - 1) >> 1) & 1, abort_flag, p.status, 0xAB2) && ok;
          __syncwarp();
          tc_fence_after();
          const float f = (m_new == -INFINITY) ? 1.f : exp2f(m_ref - m_new);
          m_ref = m_new;
          l_sum *= f;
#pragma unroll 1
          for (int c = half; c < vb * 4; c += 2) {
            uint32_t ov[16];
            tmem_ld16(lane_base + c * 16, ov);
            tmem_ld_wait();
#pragma unroll
            for (int i = 0; i < 16; ++i) ov[i] = __float_as_uint(__uint_as_float(ov[i]) * f);
            tmem_st16(lane_base + c * 16, ov);
          }
        }
      }
      const float m_use = (m_ref == -INFINITY) ? 0.f : m_ref;
      const uint64_t scale2 = pack2(p.scale_log2, p.scale_log2), ref2 = pack2(-m_use, -m_use);
      uint64_t add[2] = {0ull, 0ull};
      uint32_t pk[16];
#pragma unroll
      for (int i = 0; i < 16; ++i) {
        const uint64_t x = pack2(__uint_as_float(sv[i >> 3][(2 * i) & 15]), __uint_as_float(sv[i >> 3][((2 * i) & 15) + 1]));
        float p0, p1;
        unpack2(FORM == kGpBounded ? x : READY ? add2(x, ref2) : fma2(x, scale2, ref2), p0, p1);
        p0 = exp2_ftz(p0);
        p1 = exp2_ftz(p1);
        add[i & 1] = add2(add[i & 1], pack2(p0, p1));
        pk[i] = pack_bf16x2(p0, p1);
      }
      tmem_st16(s_t + half * 32, pk);                         // over this half's own scores
      float add_lo, add_hi;
      unpack2(add2(add[0], add[1]), add_lo, add_hi);
      l_sum += add_lo + add_hi;
      tmem_st_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(p_full + (j & 1));
    }
    ok = mbar_wait(o_done, 0, abort_flag, p.status, 0xAB1) && ok;
    ok = __all_sync(0xffffffffu, ok);
    tc_fence_after();
    pair_sync();                                              // the last maxima are read: their place takes the sums
    sum_x[half * 128 + r] = l_sum;
    pair_sync();
    l_sum += sum_x[(half ^ 1) * 128 + r];
    const float inv = l_sum > 0.f ? 1.f / l_sum : 0.f;
    __nv_bfloat16* dst = p.out + static_cast<long long>(row0 + at) * p.ldo + static_cast<long long>(head) * p.value_width +
                         slice * vb * 64;
    const __nv_bfloat16* gate = p.gate ? p.gate + static_cast<long long>(row0 + at) * p.ldg + static_cast<long long>(head) * p.value_width
                                       : nullptr;
    const int cols = min(vb * 64, p.value_width - slice * vb * 64);
    const int chunks = (cols + 15) / 16;                // of 16 columns: every second one per half
    // eight columns of a row: output gate, rounding, store
    auto finish = [&](float (&d)[8], int col) {
      if (!valid || !ok || col >= cols) return;
      if (gate) {
        float z[8];
        act_load8(gate + col, z);
#pragma unroll
        for (int i = 0; i < 8; ++i) d[i] = __fdividef(d[i], 1.f + __expf(-z[i]));
      }
      act_store8(dst + col, d);
    };
    if (p.maps == 2) {
      // rows of a head's two maps are neighbouring lanes: both compute the difference, each writes half of it
      const bool second = lane & 1;
      const float own = second ? -p.diff_lambda * inv : inv;
      float ss = 0.f;
#pragma unroll 1
      for (int c = half; c < chunks; c += 2) {
        uint32_t ov[16];
        tmem_ld16(lane_base + c * 16, ov);
        tmem_ld_wait();
#pragma unroll
        for (int i = 0; i < 16; ++i) {
          const float x = __uint_as_float(ov[i]) * own, d = x + __shfl_xor_sync(0xffffffffu, x, 1);
          ss = fmaf(d, d, ss);
        }
      }
      pair_sync();
      sum_x[half * 128 + r] = ss;
      pair_sync();
      ss += sum_x[(half ^ 1) * 128 + r];
      const float f = p.diff_scale / sqrtf(ss / p.vdim + p.eps);
#pragma unroll 1
      for (int c = half; c < chunks; c += 2) {
        uint32_t ov[16];
        tmem_ld16(lane_base + c * 16, ov);
        tmem_ld_wait();
        float d[8];
#pragma unroll
        for (int i = 0; i < 16; ++i) {
          const float x = __uint_as_float(ov[i]) * own, y = (x + __shfl_xor_sync(0xffffffffu, x, 1)) * f;
          if (i < 8) d[i] = y;
          else if (second) d[i - 8] = y;
        }
        finish(d, c * 16 + (second ? 8 : 0));
      }
    } else {
#pragma unroll 2
      for (int c = half; c < chunks; c += 2) {
        uint32_t ov[16];
        tmem_ld16(lane_base + c * 16, ov);
        tmem_ld_wait();
#pragma unroll
        for (int e = 0; e < 16; e += 8) {
          float d[8];
#pragma unroll
          for (int i = 0; i < 8; ++i) d[i] = __uint_as_float(ov[e + i]) * inv;
          finish(d, c * 16 + e);
        }
      }
    }
  }
  // ---------------------------------------------------------------------- teardown
  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem, p.tmem_cols);
  }
}

// bf16 map over [rows][heads][width]: box 64 features x box_heads x box_rows, 128-byte swizzle, zeros outside
static int gp_map(CUtensorMap* map, const void* base, int width, int heads, uint64_t rows, long long ld, uint32_t box_heads,
                  uint32_t box_rows) {
  TcEncodeFn fn = tc_encoder();
  if (!fn) return FB_ERR_DRIVER;
  if ((reinterpret_cast<uintptr_t>(base) & 15) || width % 8 || ld % 8) return FB_ERR_ALIGN;
  cuuint64_t dims[3] = {static_cast<cuuint64_t>(width), static_cast<cuuint64_t>(heads), rows};
  cuuint64_t strides[2] = {static_cast<cuuint64_t>(width) * 2, static_cast<cuuint64_t>(ld) * 2};
  cuuint32_t box[3] = {64, box_heads, box_rows};
  cuuint32_t estr[3] = {1, 1, 1};
  const CUresult r = fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(base), dims, strides, box, estr,
                        CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                        CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  return r == CUDA_SUCCESS ? FB_OK : FB_ERR_DRIVER;
}

// the same with a head's features as blocks of 64 (width % 64 == 0): box 64 features x 64 rows x box_blocks
static int gp_map_blocks(CUtensorMap* map, const void* base, int width, int heads, uint64_t rows, long long ld, uint32_t box_blocks) {
  TcEncodeFn fn = tc_encoder();
  if (!fn) return FB_ERR_DRIVER;
  if ((reinterpret_cast<uintptr_t>(base) & 15) || width % 64 || ld % 8) return FB_ERR_ALIGN;
  cuuint64_t dims[4] = {64, rows, static_cast<cuuint64_t>(width / 64), static_cast<cuuint64_t>(heads)};
  cuuint64_t strides[3] = {static_cast<cuuint64_t>(ld) * 2, 128, static_cast<cuuint64_t>(width) * 2};
  cuuint32_t box[4] = {64, kGpKv, box_blocks, 1};
  cuuint32_t estr[4] = {1, 1, 1, 1};
  const CUresult r = fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 4, const_cast<void*>(base), dims, strides, box, estr,
                        CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                        CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  return r == CUDA_SUCCESS ? FB_OK : FB_ERR_DRIVER;
}

}  // namespace fb

using namespace fb;

template <int FORM>
static int launch_gp(const CUtensorMap (&m)[5], const GpParams& p, int n_tiles, int slices, int smem, cudaStream_t stream) {
  static bool attr = false;
  if (!attr) {
    if (cudaFuncSetAttribute(gqa_prefill_tc_kernel<FORM>, cudaFuncAttributeMaxDynamicSharedMemorySize, kGpSmemLimit) != cudaSuccess)
      return FB_ERR_LAUNCH;
    attr = true;
  }
  if (launch_pdl(gqa_prefill_tc_kernel<FORM>, dim3(n_tiles, p.kv_heads, slices), dim3(kGpThreads), smem, stream, m[0], m[1],
                 m[2], m[3], m[4], p) != cudaSuccess)
    return FB_ERR_LAUNCH;
  return cudaGetLastError() == cudaSuccess ? FB_OK : FB_ERR_LAUNCH;
}

extern "C" int fb_gqa_prefill_tc(const FbGqaArgs* a, const int* tiles, int n_tiles, int tile_positions, void* stream_) {
  if (!a || !a->q || !a->pool || !a->out || !a->block_table || !tiles || a->fp32) return FB_ERR_SHAPE;
  if (a->rows <= 0 || a->heads <= 0 || a->kv_heads <= 0 || a->heads % a->kv_heads || a->kv_heads > 65535 || n_tiles <= 0 ||
      a->num_seqs <= 0 || a->max_blocks <= 0 || !(a->scale > 0.f) || !gqa_form_ok(a) || a->talk ||
      (a->softcap > 0.f && a->slopes))
    return FB_ERR_SHAPE;
  const int per = a->heads / a->kv_heads * a->maps;
  if (tile_positions <= 0 || per * tile_positions > kGpM) return FB_ERR_SHAPE;
  if (a->page_size < 8 || (a->page_size & (a->page_size - 1)) != 0) return FB_ERR_SHAPE;
  if (a->vdim_pad <= 0 || a->vdim_pad % 8 || (a->value_stride != 0 && a->vdim_pad > 256) || (a->value_stride == 0 && a->gate))
    return FB_ERR_LIMIT;
  if (a->pooled && (a->pooled_rows > 0x7fffffffLL || (reinterpret_cast<uintptr_t>(a->pooled) & 15))) return FB_ERR_SHAPE;
  if (a->pool_rows <= 0 || a->pool_rows > 0x7fffffffLL || a->pool_rows % a->page_size) return FB_ERR_SHAPE;
  if (a->ldo % 8 || a->ldg % 8 || (reinterpret_cast<uintptr_t>(a->out) & 15) || (reinterpret_cast<uintptr_t>(a->gate) & 15) ||
      (reinterpret_cast<uintptr_t>(tiles) & 15))
    return FB_ERR_ALIGN;
  cudaStream_t stream = static_cast<cudaStream_t>(stream_);
  GpParams p{};
  p.box_rows = a->page_size < kGpKv ? a->page_size : kGpKv;
  CUtensorMap maps[5];
  int rc = gp_map(&maps[0], a->q, a->key_width, a->heads * a->maps, static_cast<uint64_t>(a->rows), a->ldq, per, tile_positions);
  if (rc != FB_OK) return rc;
  const __nv_bfloat16* pool = static_cast<const __nv_bfloat16*>(a->pool);
  p.shared_keys = a->key_stride == 0;
  p.tiles = tiles;
  p.block_table = a->block_table;
  p.out = static_cast<__nv_bfloat16*>(a->out); p.ldo = a->ldo;
  p.status = static_cast<DeviceStatus*>(a->status);
  p.pool_rows = a->pool_rows;
  p.rows = a->rows; p.heads = a->heads; p.kv_heads = a->kv_heads; p.per = per; p.positions = tile_positions;
  p.num_seqs = a->num_seqs; p.max_blocks = a->max_blocks; p.page_size = a->page_size;
  p.span = key_span(a);
  p.pooled = pooled_rows<__nv_bfloat16>(a);
  p.key_width = a->key_width; p.value_width = a->value_width;
  p.shared_values = a->value_stride == 0;
  const int value_blocks = (a->value_width + 63) / 64, slices = (value_blocks + 3) / 4;
  if (slices > 65535) return FB_ERR_LIMIT;
  p.qb = (a->key_width + 63) / 64; p.vb = (value_blocks + slices - 1) / slices;
  p.tmem_cols = p.vb * 64 + 2 * kGpKv <= 256 ? 256 : 512;
  p.scale_log2 = a->scale * kLog2e;
  if (a->softcap > 0.f) {
    p.cap_log2 = a->softcap * kLog2e;
    p.cap_in = 2.f * a->scale / a->softcap;
    for (int e = 0; e < 6; ++e) p.cap_poly[e] = p.cap_log2 * kTanhPoly[e];
  }
  p.slopes = a->slopes; p.gate = static_cast<const __nv_bfloat16*>(a->gate); p.ldg = a->ldg;
  p.maps = a->maps; p.vdim = a->vdim;
  p.diff_lambda = a->diff_lambda; p.diff_scale = a->diff_scale; p.eps = a->eps;
  // query rows that stay in shared memory beside the key stages; rows too wide for that are streamed with the keys
  int smem = 0;
  static const int forms[5][3] = {{1, 4, 2}, {1, 2, 4}, {1, 1, 4}, {0, 2, 2}, {0, 1, 2}};      // resident, kb, ks
  for (int f = 0; f < 5 && smem == 0; ++f) {
    p.q_resident = forms[f][0]; p.kb = forms[f][1]; p.ks = forms[f][2];
    if (p.kb > p.qb) p.kb = p.qb;
    smem = (p.q_resident ? p.qb : p.ks * p.kb) * kGpQBlock + (p.ks * p.kb + 2 * p.vb) * kGpKvBlock + 1024 + 160 + 1024;
    if (smem > kGpSmemLimit) smem = 0;
  }
  if (smem == 0) return FB_ERR_LIMIT;
  p.pieces = (p.qb + p.kb - 1) / p.kb;
  const int key_heads = p.shared_keys ? 1 : a->kv_heads, value_heads = p.shared_values ? 1 : a->kv_heads;
  p.k_whole = p.box_rows == kGpKv && a->key_width % 64 == 0 && p.qb % p.kb == 0;
  p.v_whole = p.box_rows == kGpKv && a->value_width % 64 == 0;
  for (int i = 0; i < 2; ++i) {
    // the paged pool, and the mean rows (without any, the pool again)
    const bool mean = i == 1 && a->pooled;
    const __nv_bfloat16* base = mean ? p.pooled.base : pool;
    const uint64_t rows = static_cast<uint64_t>(mean ? a->pooled_rows : a->pool_rows);
    rc = p.k_whole ? gp_map_blocks(&maps[1 + 2 * i], base, a->key_width, key_heads, rows, a->pool_ld, p.kb)
                   : gp_map(&maps[1 + 2 * i], base, a->key_width, key_heads, rows, a->pool_ld, 1, p.box_rows);
    if (rc != FB_OK) return rc;
    rc = p.v_whole ? gp_map_blocks(&maps[2 + 2 * i], base + a->v_offset, a->value_width, value_heads, rows, a->pool_ld, p.vb)
                   : gp_map(&maps[2 + 2 * i], base + a->v_offset, a->value_width, value_heads, rows, a->pool_ld, 1, p.box_rows);
    if (rc != FB_OK) return rc;
  }
  if (a->slopes) return launch_gp<kGpBias>(maps, p, n_tiles, slices, smem, stream);
  if (a->softcap > 0.f && a->softcap <= kGpMaxCap && a->score_bound > 0.f && a->score_bound <= 0.7f * a->softcap)
    return launch_gp<kGpBounded>(maps, p, n_tiles, slices, smem, stream);
  if (a->softcap > 0.f) return launch_gp<kGpCap>(maps, p, n_tiles, slices, smem, stream);
  return launch_gp<kGpPlain>(maps, p, n_tiles, slices, smem, stream);
}
