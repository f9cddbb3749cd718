// C ABI of libferrule_b200.so.  Every entry point is `extern "C"`, takes plain
// pointers / integers plus the CUDA stream as `void*`, launches asynchronously on
// that stream and returns an FB_* code.  Python binds these through ctypes
// (ferrule_b200/ops/_lib.py); argument structs are mirrored there field for field.
//
// Plays the role of the reference's same-checkout POD ABI between its device runtime
// and native kernels (crates/ferrule-backend/native/cuda/abi/core_provider.h:477-557,
// cutlass_provider.h:390-456).
#pragma once
#include <stdint.h>

#ifdef __cplusplus
extern "C" {
#endif

enum {
  FB_OK = 0,
  FB_ERR_SHAPE = 1,   // launcher rejected the arguments (nothing was launched)
  FB_ERR_ALIGN = 2,   // pointer or stride not 16-byte aligned for TMA
  FB_ERR_DRIVER = 3,  // driver entry point missing or tensor-map encode failed
  FB_ERR_LAUNCH = 4,  // cudaLaunch / attribute error
  FB_ERR_RUNTIME = 5, // other CUDA runtime error
  FB_ERR_LIMIT = 6,   // size beyond a fixed capacity
};

// ---- status word -----------------------------------------------------------------
// 16 bytes: {code, where, detail0, detail1}.  code 0 = ok.
int fb_status_bytes(void);

// ---- tcgen05 GEMM ------------------------------------------------------------------
typedef struct FbGemmArgs {
  const void* w;            // bf16 [groups, w_rows_per_group, k] (row pitch ldw elements)
  const void* x;            // bf16 [x_rows, k] (row pitch ldx elements)
  void* out;
  long long ldw;
  long long w_group_stride; // elements between groups
  long long ldx;
  long long ldo;
  int n_out;                // output channels per group
  int k;
  int groups;
  int w_rows_per_group;
  int x_rows;
  int ntok;                 // rows per tile: 16, 32, 64, 128 or 256
  int epilogue;             // 0 store, 1 swiglu (dual weights), 2 scatter, 3 all-reduce, 4 store gelu(x),
                            // 5 gelu(gate) * up, tanh form (dual weights)
  int dual_offset;          // row of the "up" block inside a group (epilogue 1)
  int out_fp32;
  int max_tok_tiles;        // capacity of the tile table (grouped mode)
  int x_group_koff;         // batched mode (groups > 1, no tile table): X column offset per group
  int out_group_coff;       // batched mode: output column offset per group
  int force_split;          // 0 = choose automatically; else split-K factor (1, 2, 4, 8)
  const int* tile_group;    // grouped mode: per row-tile expert id, first row, row count
  const int* tile_row0;
  const int* tile_rows;
  const int* num_tok_tiles; // device scalar
  const int* dst_row;       // epilogue 2
  const float* row_scale;   // epilogue 2
  float act_limit;          // epilogue 1: clamp (0 = off)
  int rank;                 // epilogue 3
  int world;
  int rows_cap;
  int flag_capacity;
  void* peer_recv[8];
  void* peer_flags[8];
  void* local_ctr;
  const void* residual;
  long long ldr;
  unsigned long long peer_wait_ns;
  void* status;
  void* trace;              // optional: 8 x uint64 globaltimer stamps written by CTA 0 (profiling)
  int ar_payload_bf16;      // epilogue 3: push partials as bf16 pairs (half the NVLink bytes) instead of fp32
  const int* remap_rank;    // epilogue 2, expert-parallel combine: output row -> destination rank and row of
  const int* remap_row;     //   that rank's bf16 combine buffer (peer_recv[rank], pitch ldo); peer_flags[r][rank]
                            //   is bumped once per call when all of this rank's rows are stored
  void* mc_recv;            // epilogue 3, optional: multicast (NVLS) address of the ranks' receive buffers; partials
                            //   are then broadcast with one multimem store instead of one store per peer
  const float* bias;        // optional [n_out]: added in epilogues 0 and 4 (one group)
  float act_alpha;          // epilogue 1: gate * sigmoid(alpha gate) * (up + shift); alpha 0 means 1
  float act_shift;
} FbGemmArgs;

int fb_gemm_bf16(const FbGemmArgs* args, void* stream);

// fp32 tensors, full 32-bit arithmetic (FMA units); same argument block (epilogues 0..2, 4 and 5, no collectives)
int fb_gemm_f32(const FbGemmArgs* args, void* stream);

// ---- block-scaled FP8 GEMM ---------------------------------------------------------------
typedef struct FbGemmFp8Args {
  const void* w;            // e4m3 [groups, w_rows_per_group, k]
  const void* x;            // e4m3 [x_rows, k]
  const void* w_scale;      // UE8M0 [groups, ceil(w_rows_per_group/128), ceil(k/128)]
  const void* x_scale;      // UE8M0 [x_rows, ldxs] (one per 1 x 128 block)
  void* out;
  long long ldw;            // bytes = elements
  long long w_group_stride;
  long long ldx;
  long long ldxs;
  long long ldo;
  int n_out;
  int k;
  int groups;
  int w_rows_per_group;
  int x_rows;
  int ntok;                 // 16, 32 or 64 (swiglu: 16 or 32)
  int epilogue;             // 0 store, 1 swiglu, 2 scatter
  int dual_offset;          // multiple of 128
  int out_fp32;
  int max_tok_tiles;
  const int* tile_group;
  const int* tile_row0;
  const int* tile_rows;
  const int* num_tok_tiles;
  const int* dst_row;
  const float* row_scale;
  float act_limit;
  int scale_group32;        // 1: w_scale is UE8M0 [groups, w_rows_per_group, k/32] (MXFP4 values in e4m3 containers)
  void* status;
  const int* slot_cnt;      // static row slots instead of a tile table: group g owns rows [g * slot_rows,
  int slot_rows;            //   (g + 1) * slot_rows), slot_cnt[g] of them filled (slot_rows % ntok == 0)
  void* out_scale;          // non-null: `out` gets e4m3 codes (ldo in bytes) and this UE8M0 [rows, ldos] the scale
  long long ldos;           //   of every 1 x 128 output block (store and swiglu epilogues, n_out % 128 == 0)
} FbGemmFp8Args;

int fb_gemm_fp8(const FbGemmFp8Args* args, void* stream);

// ---- paged latent-KV attention -------------------------------------------------------
typedef struct FbAttnArgs {
  const void* q;            // bf16 [rows, heads, kv_lora + rope_dim]
  const void* kv;           // bf16 [pool_rows, kv_lora + rope_dim] (one layer of the pool)
  void* out;                // bf16 [rows, heads, kv_lora]
  const int* block_table;   // [num_seqs, max_blocks]
  const int* row_seq;       // [rows] sequence of each query row
  const int* row_pos;       // [rows] last kv position the row may see
  const float* sink;        // optional [heads]
  float* part_o;            // split scratch [rows, splits, heads, kv_lora] fp32
  float* part_ml;           // split scratch [rows, splits, heads, 2] fp32
  void* status;
  long long ldq;
  long long ldo;
  long long pool_rows;
  int rows;
  int heads;
  int kv_lora;
  int rope_dim;
  int num_seqs;
  int max_blocks;
  int page_size;
  int group_rows;           // consecutive query rows of one sequence sharing a CTA tile (1,2,4,8,16)
  int splits;
  int split_tokens;         // multiple of 64
  float softmax_scale;
  void* merge_ctr;          // optional: zeroed uint32 [ceil(rows/group_rows) * head blocks]; merges in-kernel
  const int* selection;     // optional [rows, sel_width] explicit pool rows per query row, -1 = masked
  int sel_width;            //   (then block_table / row_seq / row_pos are unused and group_rows must be 1)
  void* trace;              // optional uint64 [32]: globaltimer stamps of CTA (0,0,0) (profiling)
  int decode_only;          // the caller asserts: every sequence has exactly one query row in this launch and its
                            // KV rows below row_pos were written before the running step began (plain decode)
  const void* gate;         // optional [rows, ldg] (element type of q): head h's output is multiplied by sigmoid(gate[row][h])
  long long ldg;
  int window;               // > 0: a row sees its last `window` tokens only; splits divide what the row of a tile sees
} FbAttnArgs;

int fb_mla_attention(const FbAttnArgs* args, void* stream);
// the same attention in 32-bit arithmetic on the FMA units (rope_dim 0, kv_lora <= 1024; no splits, sink or selection);
// fp32: q / kv / gate / out are fp32 instead of bf16
int fb_latent_attention(const FbAttnArgs* args, int fp32, void* stream);

// ---- prefill attention on tcgen05 (128-row tiles of (position, head) pairs of one sequence) ----
typedef struct FbPrefillAttnArgs {
  const void* q;            // bf16 [rows, heads, 512 + rope_dim] contiguous (ldq == heads * (512 + rope_dim))
  const void* kv;           // bf16 [pool_rows, 512 + rope_dim] (one layer of the pool)
  void* out;                // bf16 [rows, heads, 512]
  const int* tiles;         // [n_tiles, 4]: sequence, first query row, query rows (<= 128 / heads, consecutive
                            //   positions of that sequence), position of the first row; 16-byte aligned
  const int* block_table;   // [num_seqs, max_blocks]
  const float* sink;        // optional [heads]
  void* status;
  long long ldq;
  long long ldo;
  long long pool_rows;
  int n_tiles;
  int rows;
  int heads;                // must divide 128
  int kv_lora;              // 512
  int rope_dim;             // 64, or 0: keys and values are the same 512 features
  int num_seqs;
  int max_blocks;
  int page_size;            // power of two >= 8
  float softmax_scale;
  const void* gate;         // optional bf16 [rows, ldg]: head h's output is multiplied by sigmoid(gate[row][h])
  long long ldg;
  int window;               // > 0: a row sees its last `window` tokens only
} FbPrefillAttnArgs;

int fb_mla_prefill_tc(const FbPrefillAttnArgs* args, void* stream);

// ---- layer-list models: row operators (act tensors bf16, or fp32 with fp32 = 1) ---------------------------
// x = table[ids] (fp32), h = RMSNorm(x) * norm_w; norm_stride 0: norm_w is one number.  dim_pad: row width rounded up
// to 8, padding columns are zero
int fb_embed_norm(const int* ids, const void* table, long long ldt, int vocab, float* x, long long ldx,
                  const float* norm_w, int norm_stride, void* h, long long ldh, int rows, int dim, int dim_pad, float eps,
                  int fp32, void* status, void* stream);
// x += sigmoid(gate1 + bias1) * mix + sigmoid(gate2 + bias2) * sum_{s < topk} ffn[row * slots + s];
// h = RMSNorm(x) * norm_w.  mix / ffn / gates may be null
typedef struct FbLayerTailArgs {
  float* x;
  long long ldx;
  const void* mix;
  long long ldm;
  const void* gate1;
  long long ldg1;
  const float* bias1;
  const void* ffn;
  long long ldf;
  int slots;
  int topk;
  const void* gate2;
  long long ldg2;
  const float* bias2;
  const float* norm_w;
  int norm_stride;
  int rows;
  void* h;
  long long ldh;
  int dim;
  int dim_pad;
  float eps;
  int fp32;
} FbLayerTailArgs;
int fb_gated_residual_norm(const FbLayerTailArgs* args, void* stream);
// pool[write_slot[r]] = RMSNorm(src[r, :rank]) * norm_w, zero-padded to row_dim
int fb_latent_append(const void* src, long long lds, int rank, int row_dim, const float* norm_w, float eps,
                     const long long* write_slot, void* pool, long long pool_rows, int rows, int fp32, void* status,
                     void* stream);
// latent layers with a query latent or rotated parts: the query latent normalised in place, the cache row of every token
typedef struct FbLatentPrepArgs {
  void* cq;                 // [rows, ldp] query latent, normalised in place (null: none)
  const void* ckv;          // [rows, ldp] `rank` latent features, then `rot` of the key part
  long long ldp;
  int rank_q, rank, rot, row_dim, rot_off, rows;
  const float* q_w;         // [rank_q]
  const float* kv_w;        // [rank]
  const float* cos_t;       // [max_pos, rot / 2]
  const float* sin_t;
  int max_pos, fp32;
  const int* positions;
  const long long* write_slot;
  void* pool;               // [pool_rows, row_dim]: latent | turned part at rot_off | zeros
  long long pool_rows;
  float eps;
  void* status;
} FbLatentPrepArgs;
int fb_latent_prep(const FbLatentPrepArgs* args, void* stream);
// q[row, h, rot_off ..] = turned src[row, h * rot ..]
int fb_latent_turn(const void* src, long long lds, int heads, int rot, const float* cos_t, const float* sin_t, int max_pos,
                   const int* positions, void* q, long long ldq, int row_dim, int rot_off, int rows, int fp32, void* status,
                   void* stream);
int fb_softcap(float* logits, long long ldl, int rows, int vocab, float cap, void* stream);
int fb_state_rotate(int* state_in, int* state_out, int n, int buffers, void* stream);

// ---- output-norm blocks (see stream_ops.cu) ------------------------------------------------------------------
// The residual stream is fp32; activations bf16 or fp32 (`fp32`).  Pitches are multiples of 8 elements.
typedef struct FbStreamArgs {
  float* x;                 // [rows, ldx] stream; read (unless `ids`) and written
  long long ldx;
  const int* ids;           // embedding form: x = table[ids] + pos_table[positions]
  const int* positions;
  const void* table;
  const void* pos_table;    // optional
  long long ldt;
  int vocab, max_pos;
  const void* y;            // sublayer form: x += norm(y)
  long long ldy;
  const float* norm_w;      // [dim_pad]
  const float* norm_b;      // optional [dim_pad]
  int rms;                  // 0: layer norm, 1: RMS norm
  void* act;                // optional [rows, lda]: the new stream rows as activations
  long long lda;
  const float* conv;        // optional [taps, dim_pad]: h = x + conv(x), one row per sequence (decode steps)
  float* tail;              // [n_states, taps - 1, dim_pad]
  const int* state_in;
  const int* state_out;
  int taps, n_states;
  void* h;                  // [rows, ldh]
  long long ldh;
  int rows, dim, dim_pad, fp32;
  float eps;
  void* status;
} FbStreamArgs;
int fb_stream_step(const FbStreamArgs* args, void* stream);
// rows between the sublayers of a sandwich block, every norm an RMS norm of `groups` equal parts of the row:
// x (0 when `fresh`) += out_w * norm(y + y_bias) + table[ids]; act = in_w * norm(x)
typedef struct FbSandwichArgs {
  float* x;                 // [rows, ldx]
  long long ldx;
  const void* y;            // optional [rows, ldy] sublayer output
  long long ldy;
  const float* y_bias;      // optional [dim_pad]
  const float* out_w;       // [dim_pad]
  const int* ids;           // optional: add table[ids]
  const void* table;
  long long ldt;
  int vocab, fresh;
  const float* in_w;        // optional [dim_pad]
  void* act;                // [rows, lda]
  long long lda;
  int rows, dim, dim_pad, groups, fp32;
  float eps;
  void* status;
} FbSandwichArgs;
int fb_sandwich_step(const FbSandwichArgs* args, void* stream);
// out[i] = w * norm(x[rows_idx[i]]) as activations, the same norm
int fb_sandwich_rows(const float* x, long long ldx, int x_rows, const int* rows_idx, int n, const float* w, void* out,
                     long long ldo, int dim, int dim_pad, int groups, float eps, int fp32, void* status, void* stream);
// out[i] = norm(x[rows_idx[i]]) as activations
int fb_norm_rows(const float* x, long long ldx, int x_rows, const int* rows_idx, int n, const float* norm_w,
                 const float* norm_b, int rms, void* out, long long ldo, int dim, int dim_pad, float eps, int fp32,
                 void* status, void* stream);
// causal convolution over the packed rows of several sequences, one filter of `taps` per channel; inputs before a
// sequence's first row come from its state, which is brought up to date
typedef struct FbConvArgs {
  const void* x;            // [rows, ldx]
  long long ldx;
  const float* w;           // [taps, channels]
  const float* bias;        // optional [channels]
  void* tail;               // [n_states, taps - 1, channels], dtype of x
  void* out;                // [rows, ldo]
  long long ldo;
  const int* row_seq;
  const int* seq_start;
  const int* state_in;
  const int* state_out;
  int rows, channels, taps, n_states, n_seqs;
  int x_fp32;               // x and tail are fp32 instead of bf16
  int out_fp32;
  int residual;             // out = x + conv(x)
  int silu;                 // out = silu(conv(x) + bias)
  void* status;
} FbConvArgs;
int fb_short_conv(const FbConvArgs* args, void* stream);

// ---- selective scan (see selective_scan.cu) ------------------------------------------------------------------
typedef struct FbScanArgs {
  const void* x;            // [rows, ldx] convolved inputs
  long long ldx;
  const void* z;            // [rows, ldz] output gate pre-activation
  long long ldz;
  const void* bc;           // [rows, ldbc]: B at off_b, C at off_c
  long long ldbc;
  int off_b, off_c;
  const float* dt;          // [rows, lddt] step size pre-activation without bias
  long long lddt;
  const float* dt_bias;     // [inner]
  const float* a_log2;      // [state, inner]: decay exponents, base 2
  const float* d_skip;      // [inner]
  float* states;            // [n_states, state, inner]
  const int* seq_start;
  const int* state_in;
  const int* state_out;
  void* out;                // [rows, ldo]: (scan + D x) * silu(z)
  long long ldo;
  int rows, n_seqs, inner, state, n_states, fp32;
  void* status;
} FbScanArgs;
int fb_selective_scan(const FbScanArgs* args, void* stream);    // state <= 128, inner % 8 == 0

// ---- pre-norm blocks (see pre_norm.cu) --------------------------------------------------------------------------
typedef struct FbPreNormArgs {
  const float* x;           // [rows, ldx] stream before the step (unused with ids)
  float* x_out;             // [rows, ldx] after it; another buffer than x when a shift sees rows of this batch
  long long ldx;
  const int* ids;           // optional: x = table[ids] * scale
  const void* table;
  long long ldt;
  int vocab;
  float scale;
  const void* y;            // optional [rows, ldy]: added to x
  long long ldy;
  const void* ffn;          // optional [rows * slots, ldf]: the first `topk` rows of every token are added
  long long ldf;
  int slots, topk;
  const void* shared;       // optional, with ffn: [rows, lds], added times sigmoid(shared_gate[row * ldsg])
  long long lds;
  const float* shared_gate;
  long long ldsg;
  const float* norm_w;      // [dim_pad]
  void* act;                // optional [rows, lda]: x / rms(x) * norm_w, shifted
  long long lda;
  const float* shift;       // optional [dim_pad]: share of the previous token's normalised row
  float* plane;             // [n_states, dim_pad] last normalised row of every sequence
  const int* row_seq;
  const int* seq_start;
  const int* state_in;
  const int* state_out;
  int n_states, n_seqs;
  int rows, dim, dim_pad, fp32;
  float eps;
  void* status;
} FbPreNormArgs;
int fb_pre_norm_step(const FbPreNormArgs* args, void* stream);
int fb_group_norm_rows(const void* x, long long ldx, const float* norm_w, void* out, long long ldo, int rows, int dim, int dim_pad,
                       int groups, float eps, int fp32, void* stream);

// ---- scan with one decay per head (see head_scan.cu) --------------------------------------------------------------
typedef struct FbHeadScanArgs {
  const void* xbc;          // [rows, ldx] convolved inputs: x (heads x vdim) at 0, B (groups x state) at off_b, C at off_c
  long long ldx;
  int off_b, off_c;
  const void* dt;           // [rows, ldp] step size pre-activation per head, without bias
  const void* z;            // [rows, ldp] output gate pre-activation: heads x vdim
  long long ldp;
  const float* dt_bias;     // [heads]
  const float* a_neg;       // [heads] decay rates (negative)
  const float* d_skip;      // [heads]
  float* states;            // [n_states, heads, state, vdim]
  const int* seq_start;
  const int* state_in;
  const int* state_out;
  void* out;                // [rows, ldo]: (scan + D x) * silu(z); columns past heads x vdim are zero
  long long ldo;
  int rows, n_seqs, heads, vdim, state, groups, n_states, fp32;
  int long_seqs;            // sequences with more than one row, when known (0: not counted)
  int by_token;             // prompts token by token instead of in chunks
  void* status;
} FbHeadScanArgs;
int fb_head_scan(const FbHeadScanArgs* args, void* stream);     // state <= 256

// ---- grouped-query attention in position chunks (see gqa_attention.cu) -----------------------------------------
typedef struct FbGqaArgs {
  void* q;                  // [rows, ldq]: heads x dim_pad; `fb_gqa_prep` normalises and rotates it in place
  long long ldq;
  const void* k;            // fb_gqa_prep: projected keys and values [rows, ldkv]
  const void* v;
  long long ldkv;
  const float* q_norm;      // [heads * dim_pad]
  const float* k_norm;      // [kv_heads * dim_pad]
  const float* cos_t;       // [max_pos, rot_dims / 2]
  const float* sin_t;
  int max_pos, rot_dims;
  const int* positions;
  const long long* write_slot;
  void* pool;               // [pool_rows, pool_ld]: kv_heads x dim_pad keys | kv_heads x vdim_pad values
  long long pool_rows, pool_ld;
  const void* first_pool;   // optional: value mixing, pool of the layer whose values are mixed in
  long long first_off;      // its first value column
  float v_mix;
  const int* block_table;
  const int* row_seq;
  const int* row_pos;
  int num_seqs, max_blocks, page_size, chunk;
  float scale, eps;
  void* out;                // [rows, ldo]: heads x vdim_pad
  long long ldo;
  int rows, heads, kv_heads, dim, dim_pad, vdim, vdim_pad, fp32;
  // the attention kernels (not fb_gqa_prep): q holds heads x maps rows of key_width; a row of kv head g meets the cache
  // columns from g * key_stride on (stride 0: the keys of all kv heads side by side), values start at v_offset
  int maps;                 // 2: output of a head = rms(map 1 - diff_lambda * map 2) * diff_scale
  int key_width, key_stride, v_offset;
  int window, keep_first;   // chunk 0: position i sees j with i - j < window, or j < keep_first
  const float* slopes;      // optional [heads]: slopes[h] * (i - j) is taken off the scaled score
  const void* gate;         // optional [rows, ldg]: output multiplied by sigmoid(gate)
  long long ldg;
  float diff_lambda, diff_scale;
  // values of a query row of kv head g: `value_width` columns from v_offset + g * value_stride on (stride 0: the values of all
  // kv heads side by side for every row); out then holds heads x value_width columns
  int value_width, value_stride;
  float softcap;            // > 0: score <- softcap tanh(score / softcap)
  float score_bound;        // > 0: no scaled score is larger before the cap
  // blocks of `pool_tokens` tokens that lie wholly before a row's window are seen as one cache row each (see gqa_mask.cuh):
  // row b of sequence s is pooled[(slot_of[s] / slot_div) * pooled_stride + b]
  const void* pooled;       // [pooled_rows, pool_ld], element type of pool
  long long pooled_rows;
  int pool_tokens, pooled_stride, slot_div;
  const int* slot_of;
  const float* talk;        // fb_gqa_decode_wide with value_stride 0: out_h = sum_g talk[h, g] (output of head g on the values
                            // of h's kv head), and out holds heads x vdim_pad columns
  void* status;
} FbGqaArgs;
int fb_gqa_prep(const FbGqaArgs* args, void* stream);
int fb_gqa_attention(const FbGqaArgs* args, void* stream);      // vdim <= 512
// bf16, few rows (gqa_decode.cu): key_width, vdim <= 256, key_stride > 0; the visible keys of a row are divided among `splits` (1, 2, 4, 8) CTAs;
// early: one row per sequence, keys below a row's own position predate the preceding kernel
int fb_gqa_decode(const FbGqaArgs* args, int splits, int early, void* stream);
// the same for keys (key_stride 0) or values (value_stride 0, with talk) that all heads share (gqa_decode_wide.cu), one map;
// fb_gqa_decode_wide_ok: whether cache rows of this shape fit its pipeline (key_width of a query row; own_keys: key_stride > 0)
int fb_gqa_decode_wide(const FbGqaArgs* args, int splits, int early, void* stream);
int fb_gqa_decode_wide_ok(int key_width, int kv_heads, int vdim_pad, int shared_values, int heads, int own_keys);
// out[row, h] = sum_g talk[h, g] o[row, g, columns of h's kv head]: o rows hold heads x kv_heads x vdim_pad columns
int fb_value_mix(const void* o, long long ldv, const float* talk, void* out, long long ldo, int rows, int heads, int kv_heads,
                 int vdim_pad, int fp32, void* stream);
// mean cache rows of the blocks of `pool_tokens` tokens that end with a row of this batch: pooled as in FbGqaArgs, `width`
// columns of the pool's rows
typedef struct FbPoolArgs {
  const void* pool;         // [pool_rows, pool_ld]
  long long pool_rows, pool_ld;
  void* pooled;             // [pooled_rows, pool_ld]
  long long pooled_rows;
  const int* positions;     // [rows], -1: none
  const int* row_seq;
  const int* block_table;
  const int* slot_of;
  int rows, width, num_seqs, max_blocks, page_size, pool_tokens, pooled_stride, slot_div, fp32;
  void* status;
} FbPoolArgs;
int fb_pool_blocks(const FbPoolArgs* args, void* stream);
// bf16 prompts on tcgen05 (gqa_prefill_tc.cu): vdim <= 256, page_size a power of two >= 8; tiles [n_tiles, 4] =
// sequence, first row, rows (<= tile_positions), position of the first; tile_positions * maps * heads / kv_heads <= 128
int fb_gqa_prefill_tc(const FbGqaArgs* args, const int* tiles, int n_tiles, int tile_positions, void* stream);

// ---- queries and keys normalised per head, before window attention (see head_prep.cu) -------------------------
typedef struct FbHeadPrepArgs {
  const void* q;            // [rows, ldp] projected rows: heads x maps x dim_pad
  const void* k;            // kv_heads x maps x dim_pad
  const void* v;            // kv_heads x vdim_pad; null: the values are the keys before their norm
  long long ldp;
  const float* q_bias;      // optional, as wide as q and k
  const float* k_bias;
  const float* q_norm;      // [dim_pad], shared by the heads
  const float* k_norm;
  const float* q_mix;       // [heads] factors, or [heads, heads]: out row h = sum_g q_mix[h, g] q_g, kv head by kv head
  int mix;
  void* q_out;              // [rows, ldqo]: mix: heads x (kv_heads x dim_pad); else heads x maps x (maps x dim_pad), map
                            // m's query in columns m * dim_pad.., zeros elsewhere
  long long ldqo;
  const long long* write_slot;
  void* pool;               // [pool_rows, pool_ld]: kv_heads x maps x dim_pad keys | kv_heads x vdim_pad values
  long long pool_rows, pool_ld;
  int rows, heads, kv_heads, maps, dim, dim_pad, vdim_pad, fp32;
  float eps;
  void* status;
  // optional: rotation of the leading 2 * half dimensions of a head (halves paired); q_norm / k_norm may be null (weights of one)
  const float* cos_t;       // [max_pos, half]
  const float* sin_t;
  const int* positions;
  int half, max_pos;
  const FbPoolArgs* blocks; // optional, one row per sequence: also the mean rows of the blocks that end with this step's rows
} FbHeadPrepArgs;
int fb_head_prep(const FbHeadPrepArgs* args, void* stream);

// ---- gated delta rule (see delta_rule.cu) ------------------------------------------------------------------
typedef struct FbDeltaArgs {
  const void* proj;         // [rows, ldp] projected rows: q | k | v inputs of the convolutions, beta logits
  long long ldp;
  int off_q, off_k, off_v, off_b;
  const float* ag;          // [rows, ldag]: decay pre-activation [heads * dim] at 0, output gate [heads * vdim] at off_gate
  long long ldag;
  int off_gate;
  int off_a;                // >= 0: one decay per head, pre-activation in projected columns off_a .. (dt_bias: [heads])
  int off_g;                // >= 0: output gate pre-activation in projected columns off_g .. instead of `ag`
  int gate_silu;            // output gate's activation: 0 sigmoid, 1 silu
  int long_seqs;            // sequences with more than one row, 0: not known (a hint for the scan's CTA placement)
  int fp32;                 // activations (proj, tail, out) are fp32 instead of bf16
  const float* conv;        // [taps, 2 * kv_heads * dim + heads * vdim]
  const float* a_neg;       // [heads] = -exp(A_log)
  const float* dt_bias;     // [heads * dim]
  const float* norm_w;      // [vdim]
  float* state;             // [n_states, heads, dim, vdim]
  void* tail;               // [n_states, taps - 1, channels]
  const int* row_seq;       // [rows] (prefill form)
  const int* seq_start;     // [n_seqs + 1] first row of every sequence
  const int* state_in;      // [n_seqs] state index read, -1: zeros
  const int* state_out;     // [n_seqs] state index written (never the one read), -1: none
  float *qn, *kn, *v, *decay, *beta, *qk, *o;   // scratch (prefill form): [rows, kv_heads * dim] x 2,
                            // [rows, heads * vdim], [rows, heads * dim], [rows, heads], [rows, kv_heads], [rows, heads * vdim]
  void* out;                // [rows, ldo], heads * vdim columns
  long long ldo;
  void* status;
  int n_states, rows, n_seqs, heads, kv_heads, dim, vdim, taps;
  float eps;
} FbDeltaArgs;
int fb_delta_decode(const FbDeltaArgs* args, void* stream);    // one row per sequence; dim, vdim <= 128, vdim % 4 == 0
int fb_delta_prefill(const FbDeltaArgs* args, void* stream);   // dim <= 256

// ---- small fused operators ------------------------------------------------------------
int fb_embedding(const int* ids, const void* table, void* out, int rows, int dim, int vocab,
                 void* status, void* stream);
int fb_add_rmsnorm(const void* x, long long ldx, const void* delta, long long ldd,
                   const void* weight, void* res_out, long long ldr, void* norm_out, long long ldn,
                   int rows, int dim, float eps, void* stream);
// the same, and the normalised rows once more as e4m3 codes q_out [rows, dim] + UE8M0 q_scale [rows, dim / q_block],
// q_block 128 (bit-equal to fb_quant_fp8_rows of norm_out) or 32 (fb_quant_mxfp8_rows); dim % 128 == 0
int fb_add_rmsnorm_q(const void* x, long long ldx, const void* delta, long long ldd,
                     const void* weight, void* res_out, long long ldr, void* norm_out, long long ldn,
                     int rows, int dim, float eps, void* q_out, long long ldq, void* q_scale, long long lds,
                     int q_block, void* stream);
int fb_mla_prep(const void* q, long long ldq, int q_head_dim, const void* ckv, long long ldckv,
                int heads, int kv_lora, int rope_dim, const void* kv_norm_w, float eps,
                const float* cos_t,
                const float* sin_t, int max_pos, const int* positions, const long long* write_slot,
                void* kv_pool, long long pool_rows, void* q_out, long long ldq_out, int rows,
                void* status, void* stream);
// `normalize` of the routers: bit 0 = weights sum to one; bit 1 = a group's score is its best selection value instead
// of the sum of its two best
int fb_router_topk(const float* logits, long long ldl, const float* bias,
                   const long long* hash_table, const int* token_ids, int rows, int experts,
                   int topk, int score_fn, int n_groups, int topk_groups, int normalize,
                   float route_scale, int* out_idx, float* out_w, const float* logit_bias, void* stream);
int fb_moe_plan(const int* topk_idx, const float* topk_w, int routes, int topk, int e_lo, int e_hi,
                int ntok, int dst_slots, int* src_token, int* dst_row, float* row_scale, int* tile_group,
                int* tile_row0, int* tile_rows, int max_tiles, int* counts, int* meta, void* status,
                void* stream);
// second tile table (another tile height) over the expert-major rows of a plan whose counts are on the device
int fb_moe_retile(const int* counts, int local_experts, int ntok, int* tile_group, int* tile_row0, int* tile_rows,
                  int max_tiles, int* meta, void* status, void* stream);
int fb_router_plan_fused(const void* x, long long ldx, const void* w, int hidden, const float* bias,
                         const long long* hash_table, const int* token_ids, int rows, int experts,
                         int topk, int score_fn, int n_groups, int topk_groups, int normalize,
                         float route_scale, int* out_idx, float* out_w, int e_lo, int e_hi, int ntok,
                         int dst_slots, int* src_token, int* dst_row, float* row_scale, int* tile_group,
                         int* tile_row0, int* tile_rows, int max_tiles, int* counts, int* meta,
                         void* done_ctr, void* status, void* stream);
// asynchronous L2 prefetch of [ptr, ptr + bytes) (ptr 16-byte aligned)
int fb_l2_prefetch(const void* ptr, long long bytes, void* stream);
// decode-sized batches, static plan: expert e (local) owns rows [e * slot_rows, (e + 1) * slot_rows) of src_token /
// dst_row / row_scale / xg; cnt[e] (zeroed by the caller before the step) ends up as its row count
int fb_router_append(const void* x, long long ldx, const void* w, int hidden, const float* bias,
                     const long long* hash_table, const int* token_ids, int rows, int experts, int topk, int score_fn,
                     int n_groups, int topk_groups, int normalize, float route_scale, int* out_idx, float* out_w,
                     int e_lo, int e_hi, int slot_rows, int dst_slots, int* cnt, int* src_token, int* dst_row,
                     float* row_scale, void* xg, long long ldxg, void* status, void* stream);
// the same with a bias on the logits, and `n_extra` (<= 32) further rows of w behind the experts' whose products with the row
// are written to extra [rows, n_extra] as they are
int fb_router_append_extra(const void* x, long long ldx, const void* w, int hidden, const float* logit_bias, float* extra,
                           int n_extra, int rows, int experts, int topk, int score_fn, int n_groups, int topk_groups,
                           int normalize, float route_scale, int* out_idx, float* out_w, int e_lo, int e_hi, int slot_rows,
                           int dst_slots, int* cnt, int* src_token, int* dst_row, float* row_scale, void* xg, long long ldxg,
                           void* status, void* stream);
// the same with a prologue: row = bf16(x + delta) (delta may be null) -> res_out, RMSNorm(row) * norm_w -> norm_out
// and into the router, bit-equal to fb_add_rmsnorm followed by fb_router_append (norm_w null: no prologue)
int fb_norm_router_append(const void* x, long long ldx, const void* delta, long long ldd, const void* norm_w,
                          void* res_out, long long ldr, void* norm_out, long long ldn, float eps, const void* w,
                          int hidden, const float* bias, const long long* hash_table, const int* token_ids, int rows,
                          int experts, int topk, int score_fn, int n_groups, int topk_groups, int normalize,
                          float route_scale, int* out_idx, float* out_w, int e_lo, int e_hi, int slot_rows,
                          int dst_slots, int* cnt, int* src_token, int* dst_row, float* row_scale, void* xg,
                          long long ldxg, void* status, void* stream);
int fb_gather_rows(const void* x, long long ldx, const int* src_token, const int* meta, void* out,
                   long long ldo, int cap_rows, int dim, int src_rows, void* status, void* stream);
int fb_moe_reduce_norm(const void* route_out, int slots, int topk, const int* topk_idx, int e_lo, int e_hi,
                       const void* residual, long long ldr, void* out, long long ldo, int rows, int dim,
                       const void* norm_w, void* norm_out, long long ldn, float eps, void* stream);
int fb_moe_reduce(const void* route_out, int slots, int topk, const int* topk_idx, int e_lo,
                  int e_hi, const void* extra, long long lde, const void* residual, long long ldr,
                  void* out, long long ldo, int out_fp32, int rows, int dim, void* stream);
int fb_argmax(const float* logits, long long ldl, int rows, int vocab, int* out_id, float* out_val,
              void* stream);
int fb_argmax_chunked(const float* logits, long long ldl, int rows, int vocab, int chunks,
                      float* part_val, int* part_id, void* row_ctr, int* out_id, float* out_val,
                      void* stream);
int fb_topk_logits(const float* logits, long long ldl, int rows, int vocab, int k, int* out_id,
                   float* out_val, void* stream);
int fb_copy_pages(void* pool, long long layer_stride, long long page_elems, const int* pairs,
                  int n_pairs, int n_pages, int layers, void* status, void* stream);
// greedy-token feedback between decode steps that run back to back on the device: token_ids[r] = next_id[r]
// (ids outside [0, vocab) become 0); with `advance` the row also moves to the next position and looks its KV
// write slot up in the page list (block_table [num_seqs, max_blocks])
int fb_decode_advance(const int* next_id, int* token_ids, int* positions, int* row_pos, long long* write_slot,
                      const int* row_seq, const int* block_table, int max_blocks, int page_size, int num_seqs,
                      int rows, int vocab, int advance, void* stream);

// fb_norm_router_append that gathers quantised rows: with q_src set, every route's reserved row receives the token's
// codes (q_src [rows, hidden] -> xg_q) and scale bytes (s_src [rows, s_cols] -> xg_s) instead of a bf16 row
int fb_router_append_q(const void* x, long long ldx, const void* delta, long long ldd, const void* norm_w,
                       void* res_out, long long ldr, void* norm_out, long long ldn, float eps, const void* w,
                       int hidden, const float* bias, const long long* hash_table, const int* token_ids, int rows,
                       int experts, int topk, int score_fn, int n_groups, int topk_groups, int normalize,
                       float route_scale, int* out_idx, float* out_w, int e_lo, int e_hi, int slot_rows,
                       int dst_slots, int* cnt, int* src_token, int* dst_row, float* row_scale, void* xg,
                       long long ldxg, const void* q_src, long long ldq, const void* s_src, long long lds, void* xg_q,
                       long long ldxgq, void* xg_s, long long ldxgs, int s_cols, void* status, void* stream);

// ---- collectives through the NVLink switch (multimem) ------------------------------------------------
// mode 1 reduce-scatter (out = this rank's slice [ceil(rows/world), dim]), 2 all-gather (src = this rank's slice),
// 3 all-reduce.  src: route rows [rows * slots, dim] (summed per token as in fb_moe_reduce; slots = 1, topk = 0: a
// plain partial), or null when the partial already sits in the staging area of the current call parity.
// local_base / mc_base: this rank's mapping and the multicast mapping of the channel's symmetric buffer
// [flags (256 B) | stage x 2 | result x 2]; priv: 4 private uint32 (zeroed once).
int fb_mm_collective(const void* src, long long lds, int slots, int topk, const int* topk_idx, int e_lo, int e_hi,
                     const void* residual, long long ldr, void* out, long long ldo, int rows, int dim, int mode,
                     const void* norm_w, void* norm_out, long long ldn, float eps, void* local_base, void* mc_base,
                     long long stage_off, long long result_off, long long buf_bytes, void* priv, int rank, int world,
                     unsigned long long wait_ns, void* status, void* stream);

// ---- data movers (index fills, row copies; see data_movers.cu) ----------------------------------------
int fb_mv_fill(int* dst, long long n, int start, int step, void* stream);
int fb_mv_pack_pairs(const int* ids, const float* vals, int* out, int n, void* stream);
// mode 0 window (positions), 1 offset list (idx [rows, ldi]), 2 counts (idx [rows]); base [rows] int64
int fb_mv_index_fill(int* sel, long long lds, int col0, int rows, int width, int mode, const int* positions,
                     const long long* base, const int* idx, long long ldi, void* stream);
// idx null: dst[dst_row0 + r] = src[r]; else dst[dst_row0 + r] = src[idx[r]]; rows of row_bytes (multiple of 16)
int fb_mv_move_rows(void* dst, long long ldd_bytes, long long dst_row0, const void* src, long long lds_bytes,
                    const int* idx, int rows, int src_rows, int row_bytes, void* status, void* stream);
int fb_mv_scatter_add(float* dst, long long ldd, int dst_rows, const float* src, long long lds, const int* idx,
                      int rows, int dim, void* status, void* stream);
int fb_mv_saxpy(float* y, const float* x, float a, long long n, void* stream);
int fb_mv_ring_to_logical(const int* slots, long long lds, int rows, int width, int window, const int* last_position,
                          const int* n_compressed, int* out_index, int* out_plane, long long ldo, void* stream);
int fb_mv_paged_row_scatter(void* pool, long long pool_rows, int row_bytes, const int* block_table, int max_blocks,
                            int num_seqs, int page_size, const int* row_seq, const int* positions, const void* src,
                            long long lds_bytes, int rows, void* status, void* stream);

// ---- quantisation / packing ---------------------------------------------------------------
int fb_quant_fp8_rows(const void* x, long long ldx, void* q, long long ldq, void* scale, long long lds,
                      int rows, int n, int writeback_bf16, void* stream);
int fb_dequant_fp8_block(const void* q, const void* scale, void* out, int rows, int cols, int block,
                         void* stream);
int fb_quant_mxfp4_rows(const void* x, long long ldx, void* packed, void* scale, int rows, int n,
                        void* stream);
int fb_dequant_mxfp4(const void* packed, const void* scale, void* out, int rows, int n, void* stream);
int fb_hadamard_rows(void* x, long long ldx, int rows, int n, void* stream);

// ---- MXFP4 x MXFP8 block-scaled GEMM (routed experts) --------------------------------------------
typedef struct FbGemmMxfp4Args {
  const void* w;            // packed e2m1 [groups, w_rows_per_group, k / 2] (low nibble = even element), 32-byte aligned
  const void* x;            // e4m3 [x_rows, k]
  const void* w_sf;         // weight scales arranged by fb_mxfp4_prepare_sf
  const void* x_scale;      // UE8M0 [x_rows, k / 32]
  void* out;                // bf16 / fp32 [rows, n_out], or e4m3 codes with out_mode 2
  void* out_scale;          // out_mode 2: UE8M0 [rows, n_out / 32]
  long long ldw_bytes;      // bytes between weight rows (k / 2 when dense)
  long long w_group_stride_bytes;
  long long ldx;
  long long ldxs;
  long long ldo;
  long long ldos;
  int n_out;
  int k;                    // multiple of 128
  int groups;
  int w_rows_per_group;
  int x_rows;
  int ntok;                 // 16, 32, 64 (128 without SwiGLU)
  int epilogue;             // 0 store, 1 SwiGLU (w rows = [gate block | up block]), 2 weighted scatter
  int dual_offset;
  int out_mode;             // 0 bf16, 1 fp32, 2 MXFP8 (e4m3 + one UE8M0 scale per 32 channels; store / SwiGLU only)
  int max_tok_tiles;
  const int* tile_group;
  const int* tile_row0;
  const int* tile_rows;
  const int* num_tok_tiles;
  const int* dst_row;
  const float* row_scale;
  float act_limit;
  void* status;
  int w_tiled;              // w is tile-major: [groups][ceil(rows/128)][k/128][128 rows][64 bytes] (rows padded to 128)
  int w_fp8;                // weights are e4m3 bytes [groups, rows, k] (ldw_bytes = bytes per row) instead of packed e2m1;
                            //   w_sf has the same per-32 layout (128 x 128 block scales replicated)
  const int* slot_cnt;      // static row slots instead of a tile table: group g owns rows [g * slot_rows,
  int slot_rows;            //   (g + 1) * slot_rows), slot_cnt[g] of them filled (slot_rows % ntok == 0)
} FbGemmMxfp4Args;
int fb_gemm_mxfp4(const FbGemmMxfp4Args* args, void* stream);
// linear UE8M0 weight scales [groups, rows, k / 32] -> [groups, ceil(rows / 128), k / 128, 512] blocks for the kernel
// (rows beyond the weight are padded with 0x7f); out holds groups * ceil(rows / 128) * (k / 128) * 512 bytes
int fb_mxfp4_prepare_sf(const void* scale, void* out, int groups, int rows, int k, void* stream);
// bf16 [rows, n] -> e4m3 codes [rows, n] + UE8M0 scales [rows, n / 32] (1 x 32 blocks), n a multiple of 128
int fb_quant_mxfp8_rows(const void* x, long long ldx, void* q, long long ldq, void* scale, long long lds, int rows,
                        int n, void* stream);

// ---- DeepSeek-V4 operators ---------------------------------------------------------------
// hyper-connections: state bf16 [tokens, hc, hidden], fn fp32 [nmix, hc * hidden]; coeff fp32 [tokens, nmix]
// = [pre | post | comb]; nmix = hc (head reduction) or 2 hc + hc^2; hc in {2, 4}
int fb_hc_pre(const void* state, const float* fn, const float* scale, const float* base, void* hidden_out,
              int out_fp32, float* coeff, int tokens, int hc, int hidden, int nmix, float eps, float norm_eps,
              int sinkhorn_iters, void* stream);
// same result with the hc * hidden reduction split over `chunks` CTAs per token (part: tokens * chunks * 32 floats,
// ctr: zeroed uint32 [tokens])
int fb_hc_pre_split(const void* state, const float* fn, const float* scale, const float* base, void* hidden_out,
                    int out_fp32, float* coeff, int tokens, int hc, int hidden, int nmix, float eps, float norm_eps,
                    int sinkhorn_iters, int chunks, float* part, void* ctr, void* stream);
int fb_hc_post(const void* hidden_in, const void* residual, const float* coeff, void* out, int tokens, int hc,
               int hidden, void* stream);
// group g pools rows row0 + g * ratio + [0, window); rows outside [0, n_rows) are masked; kv / gate rows have
// pitch ld, ape is contiguous [ratio, cur_col + dim]; rows of the current group read columns [cur_col, cur_col + dim), rows of the previous one [0, dim)
int fb_compressor_pool(const float* kv, const float* gate, long long ld, const float* ape, void* out, long long ldo,
                       int groups, int dim, int ratio, int window, int row0, int n_rows, int cur_col, void* stream);
int fb_rope_rows(void* x, long long ld_row, long long ld_head, int rows, int heads, int off, int rdim,
                 const int* positions, const float* cos_t, const float* sin_t, int max_pos, int inverse,
                 void* status, void* stream);
int fb_indexer_scores(const void* q, const void* plane, long long ldp, const float* head_w, float* scores,
                      long long ld_s, int queries, int heads, int d, int n, void* stream);
// one draft step of the Markov proposal head: id = argmax_t(logits[t] + W2[t] . W1[*prev_token]), ties -> lower id
int fb_markov_step(const float* logits, const void* w1, const void* w2, int vocab, int rank, int chunks,
                   const int* prev_token, float* part_val, int* part_id, void* ctr, int* out_id, float* out_val,
                   void* status, void* stream);
// taps[t][tap_off : +hidden] = bf16(mean over the hc copies of state[t])
int fb_hc_mean_scatter(const void* state, void* taps, long long ld_taps, int tap_off, int tokens, int hc, int hidden,
                       void* stream);
// head reduction over GEMM-produced dots bf16 [queries * heads, n] (pitch ld): same score chain as fb_indexer_scores
int fb_indexer_reduce(const void* dots, long long ld, const float* head_w, float* scores, long long ld_s, int queries,
                      int heads, int n, void* stream);
// n_visible (per query) may be NULL, then n_fixed applies; k <= 512
int fb_indexer_topk(const float* scores, long long ld_s, const int* n_visible, int n_fixed, int k, int* out_idx,
                    long long ldo, int queries, void* stream);

// ---- stable-slot expert table (streamed routed experts) -------------------------------------
// updates: int4 records {slot, expert, generation, evicted expert or -1}, applied in order
int fb_expert_table_apply(int* expert_to_slot, int* slot_expert, int* slot_gen, const void* updates, int n,
                          int n_experts, int n_slots, void* status, void* stream);
// tile_group: expert ids -> arena slots in place; miss[0] counts tiles of absent experts, miss[1..63] lists them
int fb_expert_table_resolve(int* tile_group, int* tile_rows, const int* num_tiles, int max_tiles,
                            const int* expert_to_slot, int n_experts, int* miss, void* stream);

// ---- expert-parallel MoE over peer memory -------------------------------------------------
// Every rank owns one symmetric buffer with the same layout (byte offsets below):
//   recv_x    bf16 [world][cap][hidden]   rows dispatched to this rank, one segment per source
//   recv_meta int4 [world][cap]           {local expert, return row (token * topk + slot), weight bits, 1}
//   recv_cnt  u32  [world]                rows each source sent in the current call
//   comb      bf16 [tcap * topk][hidden]  weighted expert outputs returned to this rank
//   disp_flag / comb_flag / gath_flag  u32 [world]   arrival counters (one per source rank, only grow)
//   gath_out  bf16 [world][tcap][hidden]  all-gathered layer outputs (optional)
typedef struct FbEpArgs {
  void* base[8];
  long long off_recv_x, off_recv_meta, off_recv_cnt, off_comb, off_disp_flag, off_comb_flag, off_gath_flag,
      off_gath_out;
  int rank, world, cap, hidden, topk, experts_local, tcap;
  unsigned long long wait_ns;
  void* status;
} FbEpArgs;
// cnt_local: u32 [world] zeroed once; every ctr: u32 [2] zeroed once, private to its call site
int fb_ep_dispatch(const FbEpArgs* a, const void* x, long long ldx, const int* idx, const float* wts, int tokens,
                   void* cnt_local, void* ctr, void* stream);
int fb_ep_collect(const FbEpArgs* a, void* ctr, int e_lo, int* r_idx, float* r_w, int* remap_rank, int* remap_row,
                  void* stream);
int fb_ep_combine_reduce(const FbEpArgs* a, void* ctr, const void* extra, long long lde, const void* residual,
                         long long ldr, void* out, long long ldo, int tokens, int allgather, int gather_row0, void* stream);
int fb_ep_gather_wait(const FbEpArgs* a, void* ctr, void* stream);

// ---- peer memory and collectives --------------------------------------------------------
int fb_ipc_handle_bytes(void);
int fb_ipc_alloc(void** ptr, long long bytes, void* handle_out);   // zero-filled device buffer + IPC handle
int fb_ipc_open(const void* handle, void** ptr);                   // map a peer rank's buffer
int fb_ipc_close(void* ptr);
int fb_ipc_free(void* ptr);
// ctr: private device words {calls, ctas_done, consumed arrivals per flag ...}
int fb_moe_reduce_allreduce(const void* route_out, int slots, int topk, const int* topk_idx, int e_lo,
                            int e_hi, const void* residual, long long ldr, void* out, long long ldo,
                            int rows, int dim, int rank, int world, int rows_cap,
                            void* const* peer_recv, void* const* peer_flags, void* ctr,
                            int payload_bf16, unsigned long long wait_ns, void* status, void* stream);
// the same with the receive buffers' multicast address (null: plain peer stores)
int fb_moe_reduce_allreduce_mc(const void* route_out, int slots, int topk, const int* topk_idx, int e_lo,
                               int e_hi, const void* residual, long long ldr, void* out, long long ldo,
                               int rows, int dim, int rank, int world, int rows_cap,
                               void* const* peer_recv, void* const* peer_flags, void* ctr,
                               int payload_bf16, unsigned long long wait_ns, void* mc_recv, void* status,
                               void* stream);
int fb_argmax_allgather(int* ids, float* vals, int vocab_lo, int rows, int rank, int world, int rows_cap,
                        void* const* peer_recv, void* const* peer_flags, void* ctr,
                        unsigned long long wait_ns, void* status, void* stream);
// two ranks bounce a counter through each other's memory; out_ns[0] = total ns for `iters` round trips
int fb_peer_pingpong(void* mine, void* theirs, int iters, int initiator, unsigned long long limit_ns, void* out_ns,
                     void* status, void* stream);
int fb_flag_wait_probe(const void* flag, int target, unsigned long long wait_ns, void* status,
                       int* result, void* stream);

#ifdef __cplusplus
}
#endif
