// Launch interfaces of the layered models' kernels.  `f32` selects the storage format of activations and weights
// (false: bf16 bits, true: float); pointers to such storage are void*.  Row strides are in elements.
#pragma once
#include <stddef.h>
#include <stdint.h>

#include "model_spec.h"

struct b2_ctx;

// ---- layer_ops.cu ---------------------------------------------------------------------------------------------
// x[t, :width] (f32 residual stream) = table[ids[t]], `copies` rows of x per token
int32_t b2_embed_residual_launch(b2_ctx* ctx, bool f32, const void* table, int ld_table, const int32_t* ids, int T, int width, int vocab, float* x,
                                 int ldx, int copies = 1);
// The stream's beginning for models without a norm ahead of their layers: table[ids[t]] * scale, plus the row of the (previous, current)
// token in a table of its own (PairSpec).  The last token of every sequence is kept for its next step.
struct EmbedPairsParams {
    const void* table;
    int ld_table, T, width, vocab;
    const int32_t* ids;
    float scale;
    PairSpec pairs;
    const void* pair_table;  // [buckets + 1, ld_pairs]
    int ld_pairs;
    const int32_t *cu_seqlens, *context_lens, *token_seq, *seq_slot;
    float* kept;             // slot s: the bits of the token at kept + s * slot_stride
    int64_t slot_stride;
    float* x;                // [T, ldx]
    int ldx;
    void* out;               // [T, ldo] the same in storage format, zero beyond width
    int ldo;
};
int32_t b2_embed_pairs_launch(b2_ctx* ctx, bool f32, const EmbedPairsParams& p);
struct AddNormParams {
    float* x;               // [*, ldx] residual stream
    const float* y;         // what the last sub-layer added (f32), null: nothing
    const int32_t* y_rows;  // [T, n_src] rows of y summed (in order) into token t; null: row t
    const float* w;         // norm weight [width]; null: only the addition
    const float* vec;       // [width] added to every row as well; null: nothing
    const void* table;      // ... and row ids[t] of this table (the embedding); null: nothing
    const int32_t* ids;
    int ld_table, vocab;
    const int32_t* row_idx; // output row r takes source row row_idx[r]; null: r
    void* out;              // [rows, ldo], zero beyond width
    int ldx, ldy, ldo, rows, width, n_src;
    float eps, out_scale;   // out = norm * w * out_scale
    bool write_x;
};
int32_t b2_add_norm_launch(b2_ctx* ctx, bool f32, const AddNormParams& p);
// Several residual streams per token: the pending sub-layer's y goes to every stream beside a mixture of the old ones, then the
// next sub-layer's norm of a weighted sum of the streams.
struct StreamNormParams {
    float* x;               // [*, streams, ldx]
    int streams;
    const float *mix, *to;  // pending: x_t <- sum_s mix[s][t] x_s + to[t] y; null: nothing is pending
    const float* y;         // f32 rows summed into y as in AddNormParams; negative row numbers are left out
    const int32_t* y_rows;
    const float* pass;      // [*] y also has pass[t] * h[t], the sub-layer's own input; null: nothing
    const void* h;          // [*, ldh]
    const float* from;      // [streams] the sum that is normed; null: all ones
    const float* w;         // norm weight; null: no norm
    float* sum;             // [rows, ldx] receives the weighted sum; null: not stored
    const int32_t* row_idx;
    void* out;              // [rows, ldo], zero beyond width; may be h
    int ldx, ldy, ldh, ldo, rows, width, n_src;
    float eps, out_scale;
    bool write_x;
};
// Norm behind a sub-layer: x' = x + mult * norm(y) * w in `groups` equal parts; then, with weights `avg`, the stream goes on as
// sum_(j < depth) avg[j] past[j] + avg[depth] x'.
struct PostNormParams {
    const float* x;         // [rows, ldx] residual stream; null: zeros (the model's last norm)
    float* x_out;           // what goes on (may be x; null: not stored)
    const float* y;         // [*, ldy] the sub-layer's output
    const int32_t* y_rows;  // row r takes y's row y_rows[r]; null: r
    const float* w;         // [width]
    int groups;
    float eps, mult;
    const float* avg;       // [depth + 1]; null: x' goes on
    int depth;
    const float* past;      // j-th: past + j * past_stride, [rows, ldx]
    int64_t past_stride;
    float* keep;            // [rows, ldx] receives x'; null: not stored
    void* out;              // [rows, ldo] what goes on in storage format, zero beyond width; null: not stored
    int ldx, ldy, ldo, rows, width;
};
int32_t b2_post_norm_launch(b2_ctx* ctx, bool f32, const PostNormParams& p);
// out[t, j] = gelu(z[t, j]) * table[ids[t], col0 + j] for j < n (tanh form), zero up to ldo
struct TokenGateParams {
    const float* z;         // [T, ldz], the sum of `parts` of them
    int ldz, parts;
    int64_t part_stride;
    const void* table;
    int ld_table, col0, vocab;
    const int32_t* ids;
    int T, n;
    void* out;
    int ldo;
};
int32_t b2_token_gate_launch(b2_ctx* ctx, bool f32, const TokenGateParams& p);
constexpr int kMaxStreams = 16;
int32_t b2_stream_norm_launch(b2_ctx* ctx, bool f32, const StreamNormParams& p);
// out[r, j] = act(gu[r, j], gu[r, up_off + j]), scaled by row_w[r] when given (see GateSpec); zero for j in [ff, ldo).  Up to two such
// arrays in one launch (the second one with rows 0: none).
struct GateRows {
    const void* gu = nullptr;
    bool gu_f32 = false;  // f32 pre-activations of a bf16 model
    int ldg = 0, up_off = 0, rows = 0, ff = 0;
    const float* row_w = nullptr;
    void* out = nullptr;
    int ldo = 0;
};
int32_t b2_gate_launch(b2_ctx* ctx, bool f32, const GateSpec& g, const GateRows& a, const GateRows& b = GateRows());
int32_t b2_zero_cols_launch(b2_ctx* ctx, bool f32, void* x, int ldx, int c0, int c1, int rows);
// y[M, N] = x[M, K] . W[N, K]^T in f32 (fused multiply-add, partial sums per 32 inputs)
int32_t b2_linear_f32_launch(b2_ctx* ctx, const float* x, int ldx, const float* w, int M, int N, int K, float* y, int ldy);
int32_t b2_argmax_f32_launch(b2_ctx* ctx, const float* logits, int ld, int rows, int vocab, int32_t* out);

// ---- gemm_grouped.cu: one matrix product per group ---------------------------------------------------------------
struct GroupedGemmParams {
    const void* x;           // rows of group g: x + g * x_gstride + row * ldx
    int64_t x_gstride;
    int ldx;
    const int32_t* row_idx;  // output row r reads x row row_idx[r]; null: r
    bool map_out;            // ... and is stored at row row_idx[r] of out as well
    const void* w;           // [G][N][K]
    int N, K, G;             // N, K padded (multiples of 64)
    void* out;               // rows of group g: out + g * out_gstride + row * ldo
    int64_t out_gstride;
    int ldo, n_out;          // columns stored per row (<= N)
    bool out_f32;            // f32 results from bf16 operands
    const int32_t* offsets;  // [G + 1] device: group g owns rows [offsets[g], offsets[g + 1]); null: every group has rows 0..M-1
    int M;                   // rows per group, or the total number of rows with `offsets`
    int x_rows;              // rows of the x allocation (0: unknown; the TMA kernel needs 128)
    // small M only: stream the weights in 64-row tiles whatever M is; the last group may have fewer rows (tail_n) and an f32 result
    bool stream;
    int tail_n;              // 0: the last group is like the others
    float* tail_out;         // [M, tail_n]
    bool vec_out;            // set by the launcher: 16-byte stores are aligned
};
// True when a product of this size takes the kernel whose operands must be consecutive rows (row_idx null): a caller that
// gathers rows does so beforehand then.
bool b2_grouped_gemm_wants_rows(const b2_ctx* ctx, int M, bool sorted, int G, int N);
int32_t b2_grouped_gemm_launch(b2_ctx* ctx, bool f32, const GroupedGemmParams& p);

// ---- moe.cu -----------------------------------------------------------------------------------------------------
struct RouteParams {
    const float* logits;  // [T, ld]: experts | identity experts | the shared expert's number
    int ld, T, experts, top;
    RouteScore score;
    int identity;         // (Softmax)
    bool shared;
    const float* correction;  // [experts + identity] (Softmax)
    float scale;
    int32_t* expert;      // [T, top] chosen experts, best first
    float* weight;        // [T, top]
    int32_t* offsets;     // [experts + 1]
    int32_t* pos;         // [T, top (+ 1)] sorted position of each (token, choice), -1 for an identity expert; then T * top + t (shared)
    int32_t* src;         // [T * top] token of each sorted position (0 beyond the last one)
    float* row_w;         // [T * top] weight of each sorted position
    float *pass, *shared_w;  // [T] summed weights of the chosen identity experts; weight of the shared expert
    int32_t* counters;    // [experts + 1], zero between launches
};
int32_t b2_route_launch(b2_ctx* ctx, const RouteParams& p);

// out[i] = x[src[i]] (rows of `cols` elements, a multiple of 8, both row strides ld)
int32_t b2_gather_rows_launch(b2_ctx* ctx, const uint16_t* x, const int32_t* src, int n, int cols, int ld, uint16_t* out);

// ---- latent_attn.cu -----------------------------------------------------------------------------------------------
struct LatentPrepParams {
    const void* qkv;        // [T, ld]: q heads as [dim | rot_dim], then kv_rank latents, then rot_dim rotated-key inputs
    int ld, T;
    const int32_t* positions;
    const int32_t* slot_mapping;
    const float *cos_t, *sin_t;  // [positions, rot.dims / 2]
    const float* c_norm;    // [kv_rank]
    float eps;
    void* cache;            // [page * page_size + offset][row_pad]
    void* q;                // [T, heads, plain_pad + rot_pad]: plain | rotated part, each zero-padded
    int plain_pad, rot_pad;
    void* q_lat;            // [T, heads, row_pad]: the rotated query part goes to columns kv_rank.., zero beyond row()
};
int32_t b2_latent_prep_launch(b2_ctx* ctx, bool f32, const LatentAttnSpec& a, const LatentPrepParams& p);
struct LatentAttnParams {
    const void* q_lat;      // [T, heads, row_pad] queries in latent coordinates | rotated part
    const void* cache;
    const int32_t* block_tables;
    int max_blocks, page_size;
    const int32_t* seq_slot;   // [B]
    const int32_t* token_seq;  // [T]
    const int32_t* positions;  // [T]
    const int32_t* row_idx;    // [T] token rows to run (null: 0 .. T-1)
    void* o_lat;            // [token rows, heads, o_pad] attention-weighted latents
    int o_pad, T;
};
// Tensor-core form for single tokens (bf16): rows of a list, each with its own context, keys split over CTAs.
struct LatentDecodeParams {
    const void* q_lat;
    const void* cache;
    const int32_t* block_tables;
    int max_blocks, page_size;
    // rows: the packer's decode list (context, token row, block-table row), or (ctx null) every token of the step
    const int32_t *ctx, *qrow, *slot;
    const int32_t *positions, *token_seq, *seq_slot;
    // work items (row, chunk): the packer's list, or (work_seq null) one per row, whose chunk must hold its whole context
    const int32_t *work_seq, *work_chunk, *work_off, *n_work;
    // > 0 (rows of the decode list under a mask): item = row * row_chunks + chunk, chunks counted from the first visible key's box
    int row_chunks;
    int chunk_tiles;   // 16-key boxes per chunk (whole tiles of b2_latent_decode_tile() keys)
    int stages;        // set by the launcher: tiles in shared memory
    int64_t cache_rows;  // rows of the cache allocation
    float scale_log2;  // scale * log2(e)
    float *part_o, *part_ml;  // [work item][head][kv_rank], [work item][head][2]
    void* o_lat;
    int o_pad;
};
bool b2_latent_decode_eligible(const LatentAttnSpec& a);
int32_t b2_latent_decode_launch(b2_ctx* ctx, const LatentAttnSpec& a, LatentDecodeParams p, int items, int rows);
int b2_latent_decode_tile();  // keys per tile
int32_t b2_latent_attn_simple_launch(b2_ctx* ctx, bool f32, const LatentAttnSpec& a, const LatentAttnParams& p);

// ---- latent_prefill.cu: portions of more than one token (bf16), keys and values expanded per head --------------------
struct LatentGatherParams {
    const void* cache;
    const int32_t* block_tables;
    int max_blocks, page_size, B, rows;
    const int32_t* seq_slot;      // [B]
    const int32_t* context_lens;  // [B]
    const int32_t* kv_off;        // [B] first gathered row of each prefilling sequence, -1 for the others; holds the first key its portion sees
    const int32_t* cu_seqlens;    // [B + 1]
    void* lat;                    // [rows, ld_lat]
    int ld_lat;
    void* rot;                    // [rows, rot_pad]
    int rot_pad;
};
int32_t b2_latent_gather_launch(b2_ctx* ctx, const LatentAttnSpec& a, const LatentGatherParams& p);
struct LatentPrefillParams {
    const void* q;      // [q_rows, heads, (plain_blocks + rotated blocks) * 64]: plain | rotated part, each zero-padded
    int q_rows;
    const void* kv;     // [kv_rows, ld_kv]: plain keys head by head (plain_blocks * 64 each), from column v_col0 the values
    const void* rot;    // [kv_rows, rotated blocks * 64]
    int kv_rows, ld_kv, v_col0, plain_blocks;
    const int32_t *pf_seq, *pf_qstart, *n_work, *cu_seqlens, *context_lens, *kv_off;
    float scale_log2;
    void* out;          // [T, ldo]: heads * vdim columns
    int ldo, vdim;
};
bool b2_latent_prefill_eligible(const LatentAttnSpec& a);
int32_t b2_latent_prefill_launch(b2_ctx* ctx, const LatentAttnSpec& a, const LatentPrefillParams& p, int grid_work);

// ---- grouped_attn.cu, grouped_attn_decode.cu, grouped_attn_prefill.cu --------------------------------------------------
// Cache of a layer: keys [page][k_heads][page_size][k_row], values [page][kv_heads][page_size][v_row].  With two maps head h's queries are
// rows 2h and 2h + 1, a key / value head's keys likewise (k_heads, q_heads).
struct GqaPrepParams {
    const void* in;         // [T, ld] projections: queries from q_off, keys from k_off, values from v_off, heads (and their maps) tight
    int ld, q_off, k_off, v_off, T;
    const float *q_bias, *k_bias, *v_bias;  // null: none
    const float *q_norm, *k_norm;           // null: none; [dim], or [heads * dim] (norm_all)
    bool own_kv;            // off: queries only
    float eps;
    const int32_t *positions, *slot_mapping;
    const float *cos_t, *sin_t;  // [positions, rot.dims / 2]
    void* q;                // [T, q_heads, k_row]
    void *k_cache, *v_cache;
    int page_size;
};
int32_t b2_gqa_prep_launch(b2_ctx* ctx, bool f32, const GroupedAttnSpec& a, const GqaPrepParams& p);
struct GqaAttnParams {
    const void* q;
    const void *k_cache, *v_cache;
    const int32_t* block_tables;
    int max_blocks, page_size;
    int64_t max_pages;
    int T;                       // rows of q in use
    // every token by itself: its sequence and position
    const int32_t *positions, *token_seq, *seq_slot;
    // the packer's decode list (context, token row, block-table row) and its work items (row, chunk)
    const int32_t *dec_ctx, *dec_qrow, *dec_slot, *work_seq, *work_chunk, *work_off, *n_dec_work;
    int row_chunks;              // > 0 (under a mask): item = row * row_chunks + chunk, chunks counted from the first visible key's tile
    int chunk_tiles;             // 16-key tiles per work item
    float *part_o, *part_ml;     // [work item][q head][v_row], [work item][q head][2]
    int* counters;               // [decode rows][head blocks], zero between launches
    // the packer's prefill list (sequence, first query), 128 queries per item
    const int32_t *pf_seq, *pf_qstart, *n_pf_work, *cu_seqlens, *context_lens;
    int q_rows;                  // rows of the q allocation
    float out_scale;
    // two maps: weight of the second one, eps of the norm of their difference; head_gate: [T, ld_gate] one column per head
    float lambda, eps;
    const void* gate;
    int ld_gate;
    void* out;                   // [T, ldo]: heads * vdim columns
    int ldo;
};
int32_t b2_gqa_simple_launch(b2_ctx* ctx, bool f32, const GroupedAttnSpec& a, const GqaAttnParams& p);
bool b2_gqa_decode_eligible(const GroupedAttnSpec& a);
int b2_gqa_head_blocks(const GroupedAttnSpec& a);  // blocks of up to eight query heads that share a key / value head
// items > 0: the decode list; items == 0: every token of the step is a row of its own
int32_t b2_gqa_decode_launch(b2_ctx* ctx, const GroupedAttnSpec& a, const GqaAttnParams& p, int items);
bool b2_gqa_prefill_eligible(const GroupedAttnSpec& a);
int32_t b2_gqa_prefill_launch(b2_ctx* ctx, const GroupedAttnSpec& a, const GqaAttnParams& p, int grid_work);

// ---- memory.cu, memory_chunk.cu ------------------------------------------------------------------------------------
struct MemoryParams {
    const void* in;         // [T, ld] projections
    int ld, c_off, b_off;   // columns of q | k | v and of the step sizes' inputs
    const void* dec;        // [T, ld_dec] decay inputs (decays() columns; f32 for DecayMap::Exp); null for fixed decays
    int ld_dec;
    int T, B;
    const int32_t *cu_seqlens, *context_lens, *token_seq, *seq_slot, *positions;
    float* state;           // slot s: state + s * slot_stride: [heads][vdim][dim], then [conv - 1][channels] inputs, oldest first
    int64_t slot_stride;
    const float *conv_w;    // [taps][channels]
    const float *dt_bias, *A_log;
    const float *decay, *log_decay;  // fixed decays [heads]
    const float *cos_t, *sin_t;
    // DecayMap::Exp instead of dec: the first factor's result [T, ld_low] (f32) and the second factor [.., low_k] (bf16), `rank` wide
    const float* low;
    int ld_low, rank;
    const void* low_w;
    int low_k;
    // prepared inputs of the recurrence
    float *q, *k;           // [T, q_cols]; with a bonus q and k are read from `in`
    const void* v;          // [T, ld_v]
    int ld_v;
    float *lg, *beta;       // [T, decays()] logarithms of the decays; [T, heads]
    float* o;               // [T, heads * vdim]
    // chunked form, for portions of at least kMemoryChunkMin tokens
    int n_chunks;           // 64-token chunks of those portions; 0: every portion goes token by token
    const int32_t* chunk_off;  // [B] a portion's first chunk, -1 for the shorter ones
    void* chunk;            // scratch, n_chunks * b2_memory_chunk_bytes()
    const float* bonus;     // [heads][dim]
    const void* h;          // [T, ld_h] the normed stream, whose last row per sequence is kept (shift)
    int ld_h;
};
// Token shift: five mixtures h + (h' - h) mu[i] side by side, out [T, 5 * ldo] (zero beyond the width), h' the row of the token before
// (the kept one, or zeros, for a portion's first token).
struct ShiftParams {
    const void* h;
    int ld_h, T, width, ldo;
    const float* mu;        // [5][width]
    void* out;
    const int32_t *cu_seqlens, *context_lens, *token_seq, *seq_slot;
    const float* kept;      // slot s: kept + s * slot_stride
    int64_t slot_stride;
};
int32_t b2_token_shift_launch(b2_ctx* ctx, bool f32, const ShiftParams& p);
// out[t, j] = tanh(x[t, j]) for j < n, zero up to ldo
int32_t b2_tanh_launch(b2_ctx* ctx, const float* x, int ldx, int T, int n, float* out, int ldo);
int32_t b2_memory_launch(b2_ctx* ctx, bool f32, const MemorySpec& s, const MemoryParams& p);
constexpr int kMemoryChunk = 64, kMemoryChunkMin = 12;  // tokens per chunk; shortest portion that the chunked form takes
bool b2_memory_chunk_eligible(const MemorySpec& s);
size_t b2_memory_chunk_bytes(const MemorySpec& s);  // per chunk
int32_t b2_memory_chunk_launch(b2_ctx* ctx, const MemorySpec& s, const MemoryParams& p);
// Input row of a layer's output projection: attention heads (already there), memory heads (norm, gate), feed-forward (gelu);
// everything else zero.
struct BranchOutParams {
    void* out;              // [T, ldo]
    int ldo, T, att_cols;
    const float* o;         // memory: [T, heads * vdim]; null: none
    int heads, vdim, m_off;
    const void* gate;
    int ld_gate;
    MemGate act;
    const float* norm;      // [vdim], or [heads * vdim] (norm_heads); null: none
    bool norm_heads;
    float eps, scale;
    const void* up;         // feed-forward: [T, ld_up]; null: none
    int ld_up, ff, f_off;
};
int32_t b2_branch_out_launch(b2_ctx* ctx, bool f32, const BranchOutParams& p);

// ---- gated_average.cu: GatedAverageSpec -------------------------------------------------------------------------------
struct GatedAverageParams {
    const void* in;         // [T, ld] projections Z, U, G from these columns, each zero up to a multiple of 8
    int ld, z_off, u_off, g_off, width;
    const float *z_bias, *u_bias;  // zero up to a multiple of 8
    int T, B;
    const int32_t *cu_seqlens, *context_lens, *seq_slot;
    float* state;           // slot s: state + s * slot_stride, [width] (up to a multiple of 4)
    int64_t slot_stride;
    void* out;              // [T, ldo] zero beyond width
    int ldo;
    // portions of at least kMemoryChunkMin tokens: 64-token chunks (as the memories')
    int n_short, n_long;    // portions with fewer tokens; portions of more than one chunk
    int n_chunks;
    const int32_t* chunk_off;
    float* chunk;           // scratch, n_chunks * b2_gated_average_chunk_floats()
};
size_t b2_gated_average_chunk_floats(int width);  // per chunk
int32_t b2_gated_average_launch(b2_ctx* ctx, bool f32, const GatedAverageParams& p);

// ---- ssm.cu ---------------------------------------------------------------------------------------------------------
struct SsmParams {
    const void* zx;       // [T, ld]: z | x | B | C | dt
    int ld, T, B;
    const int32_t* cu_seqlens;    // [B + 1]
    const int32_t* context_lens;  // [B], this step's tokens included
    const int32_t* token_seq;     // [T]
    const int32_t* seq_slot;      // [B]
    float* state;         // slot s: state + s * slot_stride: heads x vdim x state, then channels x (conv - 1)
    int64_t slot_stride;
    const float *conv_w, *conv_b, *dt_bias, *A_log, *D, *norm;
    float eps;
    void* xbc;            // [T, channels] convolved inputs
    int ld_xbc;
    float* y;             // [T, inner]
    void* out;            // [T, ldo] gated and normed, zero beyond inner
    int ldo;
    bool chunked;         // set by the launcher: longer portions belong to the chunked form
};
int32_t b2_ssm_launch(b2_ctx* ctx, bool f32, const Mamba2Spec& s, const SsmParams& p);
