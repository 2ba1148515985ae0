/*
 * msa_b200_lm -- C ABI of the kernels behind the layered decoder designs (libmsa_b200_lm.so): residual / norm steps,
 * windowed latent attention, the gated delta rule, and mixtures of small experts.
 *
 * Conventions are those of msa_b200.h (raw device pointers owned by the caller, asynchronous on `stream`, strides in
 * elements, MSA_OK or a negative code with msa_last_error()).  `dtype` is the type of activations and weights
 * (MSA_BF16 or MSA_F32); norms, scores, gates, states and the residual are 32-bit in both.
 *
 * Packed step.  A step runs n_tok tokens of n_seq sequences, packed one sequence after the other: sequence s owns the
 * rows cu[s] .. cu[s+1]-1, continues at position start[s] and keeps its state in slot slot[s].  The first n_decode
 * sequences bring exactly one token each.
 */
#ifndef MSA_B200_LM_H
#define MSA_B200_LM_H

#include "msa_b200.h"

#ifdef __cplusplus
extern "C" {
#endif

/* x_out[r] = base + branch;  h_out[r] = rmsnorm(x_out[r]) * w_next;  cat_out[r] = x_out[r] rounded to dtype.
 *   base    row r of base [.., width] fp32 with base_stride (0: one vector for all rows), or null
 *   branch  null, or B = row r of y (y_dtype), or the weighted sum over k < top of rows inv[r*top+k] of y with
 *           weights mix[r*top+k] (inv != null); with w_branch: rmsnorm(B) * w_branch
 *   rows    optional: output row r works on input row rows[r] of base
 *   add     optional further rows [n_rows, width] fp32 that join x_out
 *   h_out2  a second norm of the same stream, rmsnorm(x_out[r]) * w_next2 (needs h_out)
 * Any of x_out, h_out (with w_next), cat_out may be null. */
int msa_lm_residual_norm(const float* base, int64_t base_stride, const void* y, int32_t y_dtype, int64_t y_stride,
                         const int32_t* inv, const float* mix, int32_t top, const float* w_branch, const float* w_next,
                         float eps, const int32_t* rows, int32_t n_rows, int32_t width, float* x_out, void* h_out,
                         void* cat_out, int64_t cat_stride, const float* add, const float* w_next2, void* h_out2,
                         int32_t dtype, void* stream);

/* x_out[r] = table[token[r]] (fp32; x_copy: the same again), h_out / h_out2 = rmsnorm(x_out) * w_next / w_next2, cat0 /
 * cat1[r] = the row in dtype; everything but x_out may be null.  pair_table [buckets + 1, width]: a hashed row of (previous
 * token, token) is added, number (previous * mul_prev + token * mul_cur) mod buckets, the last one for a sequence's first
 * token; last_token [slots] keeps every sequence's previous token from step to step.
 * Tokens outside 0 .. vocab-1 read row 0 and count in status[2]. */
typedef struct {
  const void* table; const int32_t* token;
  const void* pair_table; int64_t buckets, mul_prev, mul_cur;
  int32_t* last_token;
  const int32_t *tok_seq, *slot, *start, *cu;
  const float *w_next, *w_next2;
  float *x_out, *x_copy;
  void *h_out, *h_out2, *cat0, *cat1;
  int64_t cat_stride;
  int32_t* status;
  int32_t n_rows, width, vocab;
  float eps;
  int32_t dtype;
} msa_lm_embed_args;
int msa_lm_embed(const msa_lm_embed_args* args, void* stream);

/* out[r, j] = silu(gu[r, j]) * gu[r, ff + j]. */
int msa_lm_silu_mul(const void* gu, int64_t gu_stride, int32_t n_rows, int32_t ff, void* out, int64_t out_stride,
                    int32_t dtype, void* stream);

/* x = cap * tanh(x / cap) in place. */
int msa_lm_softcap(float* x, int64_t n, float cap, void* stream);

/* out [n_rows, parts, cols]: tanh(x [n_rows, cols]) as a sum of `parts` numbers of type dtype. */
int msa_lm_tanh_split(const float* x, int32_t n_rows, int32_t cols, int32_t parts, void* out, int32_t dtype, void* stream);

/* out [n_mix, n_tok, width]: h + (before - h) * mu[m], before = the sequence's previous row (zeros for its first token).
 * shift [slots, width] keeps every sequence's last row from step to step. */
int msa_lm_token_shift(const void* h, const float* mu, int32_t n_mix, int32_t n_tok, int32_t width, const int32_t* tok_seq,
                       const int32_t* slot, const int32_t* start, const int32_t* cu, void* shift, void* out, int32_t dtype,
                       void* stream);

/* ---- windowed latent attention ------------------------------------------------------------------------------------
 * proj row = [heads * (dim + rot) query | rank latent | rot shared key part].  The kernel normalises the latent with
 * w_norm, rotates the key part and (in place) every head's rotated query part, and writes [latent | key part] to the
 * sequence's ring (decode rows: ring[slot][position % ring_rows]) or to the packed context of the step (the others:
 * row ctx_off[s - n_decode] + min(start, window - 1) + t).  It also copies the ring rows that a continued portion still
 * sees (positions start - min(start, window-1) .. start-1) into the context, n_old rows in all; old_off is their prefix
 * sum over the non-decode sequences. */
int msa_lm_latent_prep(void* proj, int64_t proj_stride, const float* w_norm, float eps, const float* inv_freq,
                       int32_t heads, int32_t dim, int32_t rot, int32_t rank, const int32_t* pos, const int32_t* tok_seq,
                       const int32_t* slot, const int32_t* start, const int32_t* cu, const int32_t* ctx_off,
                       const int32_t* old_off, int32_t n_tok, int32_t n_seq, int32_t n_decode, int32_t n_old,
                       int32_t window, void* ring, int64_t ring_rows, void* ctx, int32_t dtype, void* stream);

/* The last min(tokens, ring_rows) context rows of every non-decode sequence go to its ring. */
int msa_lm_ring_store(const void* ctx, int32_t row_width, const int32_t* slot, const int32_t* start, const int32_t* cu,
                      const int32_t* ctx_off, int32_t n_seq, int32_t n_decode, int32_t max_len, int32_t window, void* ring,
                      int64_t ring_rows, int32_t dtype, void* stream);

/* General windowed attention (any sizes, both dtypes).  A query is [qa (da) | qb (db)], a key [ka | kb]; strides per row
 * and per head; query head h uses key / value head h / group (whose stride may be 0).  Queries: rows cu[s] .. of the sequences seq0 .. seq1-1, token t
 * at position start[s] + t.  Keys: ring_rows > 0: position j in row slot[s] * ring_rows + j % ring_rows; else context row
 * ctx_off[s - seq0] + (j - first), first = start[s] - min(start[s], window-1).  Position i sees 0 <= i - j < window.
 * sink: one is added to the softmax denominators (an entry with score 0 and no value).  gate (dtype, may be null): head h's
 * output is multiplied by sigmoid(gate[token * gate_row + h]), tokens counted like the query rows. */
typedef struct {
  const void* qa; int64_t qa_row, qa_head;
  const void* qb; int64_t qb_row, qb_head;
  const void* ka; int64_t ka_row, ka_head;
  const void* kb; int64_t kb_row, kb_head;
  const void* v;  int64_t v_row, v_head;
  void* out;      int64_t out_row, out_head;
  const void* gate; int64_t gate_row;
  const int32_t *slot, *start, *cu, *ctx_off;
  int64_t ring_rows;
  int32_t group, sink;
  int32_t seq0, seq1, max_len, heads, da, db, dv, window;
  int32_t qa_dtype, out_dtype, dtype;   /* qa and out may be fp32 beside bf16 keys and values */
  float scale;
} msa_lm_attn_args;
int msa_lm_window_attn(const msa_lm_attn_args* args, void* stream);

/* The same for a prompt portion on tcgen05 (bf16; da 64 or 128, db 0 or 64, dv 64 or 128; with db, qb = qa + da and one kb
 * for all heads): n_rows query rows (row 0 = packed row row0 = cu[seq0]), n_ctx context rows.  A wait that runs out sets
 * status[0]. */
int msa_lm_window_attn_tc_supported(int32_t dim, int32_t rot, int32_t vdim);
int msa_lm_window_attn_tc(const msa_lm_attn_args* args, int32_t n_rows, int32_t n_ctx, int32_t row0, int32_t* status, void* stream);

/* ---- grouped attention behind a short convolution -------------------------------------------------------------------
 * proj row = [heads*dim q | kv_heads*dim k | kv_heads*vdim v | heads gate logits].  Every channel of q, k and v passes a
 * causal convolution of `taps` taps (conv_w [taps, channels] fp32, channels = q, k, v in this order), then the first rot
 * dimensions of the q and k heads are rotated (neighbouring pairs).  q goes to q_out [n_tok, heads, q_pitch]; [keys |
 * values] (kv_heads * k_pitch | kv_heads * v_pitch elements, a head's first dim / vdim used) go to the ring or the packed
 * context as for latent_prep.  conv_state [slots, 2, taps-1, channels] in dtype: the inputs of the taps-1 positions before position p live in half p & 1; decode rows
 * advance it here, portions by msa_lm_conv_store. */
typedef struct {
  const void* proj; int64_t proj_stride;
  const float *conv_w, *inv_freq;
  void *conv_state, *q_out, *ring, *ctx;
  const int32_t *pos, *tok_seq, *slot, *start, *cu, *ctx_off, *old_off;
  int64_t ring_rows;
  int32_t heads, kv_heads, dim, vdim, rot, taps, q_pitch, k_pitch, v_pitch;
  int32_t n_tok, n_seq, n_decode, n_old, window;
  int32_t dtype;
} msa_lm_group_args;
int msa_lm_group_prep(const msa_lm_group_args* args, void* stream);

/* Convolution inputs of the last taps-1 positions of every non-decode sequence -> conv_state; `proj` points at the first
 * convolved column of the packed rows. */
int msa_lm_conv_store(const void* proj, int64_t proj_stride, int32_t channels, int32_t taps, void* conv_state, const int32_t* slot,
                      const int32_t* start, const int32_t* cu, int32_t n_seq, int32_t n_decode, int32_t dtype, void* stream);

/* Decode attention over the rings on tensor cores (bf16; k_pitch and v_pitch 64 or 128): sequence i of n at position pos[i]
 * attends with q [n, heads, dim] (row stride q_row) to the visible rows of its ring [keys | values]; out [n, heads, vdim]
 * (row stride out_row) times sigmoid(gate[i * gate_row + h]) (gate may be null).  splits > 1: part_o [n, heads, splits,
 * vdim], part_ml [n, heads, splits, 2] fp32. */
int msa_lm_group_decode_supported(int32_t dim, int32_t vdim);
int msa_lm_group_decode(const void* q, int64_t q_row, const void* ring, int64_t ring_rows, const int32_t* slot, const int32_t* pos,
                        int32_t n, int32_t heads, int32_t kv_heads, int32_t dim, int32_t vdim, int32_t window, int32_t splits,
                        float scale, int32_t sink, const void* gate, int64_t gate_row, void* out, int64_t out_row, float* part_o,
                        float* part_ml, void* stream);

/* Decode attention over the rings on tensor cores (bf16; rank a multiple of 128 up to 512, rot 0, 32 or 64): sequence i
 * of n at position pos[i] attends with qa [n, heads, rank] and qb [n, heads, rot] (row / head strides) to its ring's
 * visible rows; out [n, heads, rank].  splits > 1: part_o [n, heads, splits, rank], part_ml [n, heads, splits, 2] fp32.  A wait
 * that runs out sets status[0]. */
int msa_lm_latent_decode_supported(int32_t rank, int32_t rot);
int msa_lm_latent_decode(const void* qa, int64_t qa_row, int64_t qa_head, const void* qb, int64_t qb_row, int64_t qb_head,
                         const void* ring, int64_t ring_rows, const int32_t* slot, const int32_t* pos, int32_t n,
                         int32_t heads, int32_t rank, int32_t rot, int32_t window, int32_t splits, float scale, void* out,
                         float* part_o, float* part_ml, int32_t* status, void* stream);

/* ---- gated delta rule ---------------------------------------------------------------------------------------------
 * proj row = [kv_heads*dim q | kv_heads*dim k | heads*vdim v | heads*vdim gate | heads beta | heads decay].
 * Convolution weights conv_w [taps, 2*kv_heads*dim + heads*vdim] fp32.  Conv state [slots, 2, taps-1, channels] in dtype:
 * the inputs of the taps-1 positions before position p live in half p & 1.  Recurrent state [slots, heads, dim, vdim]
 * fp32.  A sequence at position 0 starts from zero whatever its slot held. */
typedef struct {
  const void* proj; int64_t proj_stride;
  const float *conv_w, *a_log, *dt_bias, *w_norm;
  void* conv_state;
  float* state;
  const int32_t *pos, *tok_seq, *slot, *start, *cu;
  int32_t n_tok, n_seq, n_decode;
  int32_t heads, kv_heads, dim, vdim, taps;
  float eps;
  int32_t dtype;
} msa_lm_delta_args;

/* Decode sequences: convolution, unit norms, gates, state update, read-out, gated norm -> out [n_decode, heads*vdim]. */
int msa_lm_delta_decode(const msa_lm_delta_args* a, void* out, int64_t out_stride, void* stream);
/* The other sequences: convolution + silu + unit norms -> qk [rows, 2, kv_heads, dim] fp32 (q scaled by dim^-1/2),
 * v [rows, heads, vdim] fp32, gates [rows, 2, heads] fp32 (log decay, beta); rows count from the first non-decode token. */
int msa_lm_delta_prep(const msa_lm_delta_args* a, float* qk, float* v, float* gates, void* stream);
/* The same with q and k as pairs of bf16 numbers: qk [rows, 2 (q, k), 2 (hi, lo), kv_heads, dim], v in bf16 (bf16 activations, 2 to 4
 * taps, dim <= 128, dim and vdim multiples of 4). */
int msa_lm_delta_prep_split(const msa_lm_delta_args* a, void* qk, void* v, float* gates, void* stream);
/* The recurrence in chunks of 64 tokens on tensor cores, from msa_lm_delta_prep_split's outputs, with the gated output norm
 * -> out (bf16); advances the state.  chunk_off: prefix sums of ceil(tokens / 64) over the non-decode sequences, n_chunks in
 * all; tile: value columns per CTA (32, 64 or 128, divides vdim); o [rows, heads, vdim] fp32 scratch when tile < vdim. */
int msa_lm_delta_chunk_supported(int32_t dim, int32_t vdim, int32_t taps);
int64_t msa_lm_delta_chunk_workspace(int32_t n_chunks, int32_t heads);
int msa_lm_delta_chunk(const msa_lm_delta_args* a, const void* qk, const void* v, const float* gates, const int32_t* chunk_off,
                       int32_t n_chunks, int32_t tile, void* workspace, float* o, void* out, int64_t out_stride, void* stream);
/* Convolution inputs of the last taps-1 positions -> conv_state. */
int msa_lm_delta_conv_store(const msa_lm_delta_args* a, void* stream);
/* The recurrence token by token -> o [rows, heads, vdim] fp32; advances the state. */
int msa_lm_delta_scan(const msa_lm_delta_args* a, const float* qk, const float* v, const float* gates, float* o, void* stream);
/* out = o / rms(o) * w_norm * silu(gate) for the non-decode rows. */
int msa_lm_delta_out(const msa_lm_delta_args* a, const float* o, void* out, int64_t out_stride, void* stream);

/* ---- recurrences without a correction term --------------------------------------------------------------------------
 * Per head a matrix state S [key channels, value channels] in fp32 (a sequence at position 0 starts from zero whatever its
 * slot held).  Per token the state decays and the outer product of a key and a value joins it.
 *
 * wkv: every key channel has its own decay, exp(-exp(decay + w0)); the read-out comes before the decay, with the current
 * token under the bonus u: o = S^T r + (r . (u k)) v.  Each head's o is divided by its root mean square, times norm, times
 * silu(g).  r, k, v, g: [n_tok, heads*dim] rows of row_stride elements; decay [n_tok, heads*dim] fp32 (of the portions'
 * rows the chunked kernels keep running sums there); state [slots, heads, dim, dim]. */
typedef struct {
  const void *r, *k, *v, *g; int64_t row_stride;
  float* decay;
  const float *w0, *u, *norm;
  float* state;
  const int32_t *tok_seq, *slot, *start, *cu;
  int32_t n_tok, n_seq, n_decode, heads, dim;
  float eps;
  int32_t dtype;
} msa_lm_wkv_args;
/* Decode sequences -> out [n_decode, heads*dim]. */
int msa_lm_wkv_decode(const msa_lm_wkv_args* a, void* out, int64_t out_stride, void* stream);
/* The other sequences token by token (dim up to 256): out row 0 = first non-decode row; o [rows, heads*dim] fp32 scratch. */
int msa_lm_wkv_scan(const msa_lm_wkv_args* a, float* o, void* out, int64_t out_stride, void* stream);
/* The same in chunks of 64 tokens on tensor cores (bf16; dim a multiple of 8 up to 128).  chunk_off: prefix sums of
 * ceil(tokens / 64) over the non-decode sequences, n_chunks in all; work [n_chunks, heads, dim, dim] fp32. */
int msa_lm_wkv_chunk_supported(int32_t dim);
int msa_lm_wkv_chunk(const msa_lm_wkv_args* a, const int32_t* chunk_off, int32_t n_chunks, float* work, void* out, int64_t out_stride,
                     void* stream);

/* ssd: one decay per head, exp(-exp(a_log) * dt) with dt = softplus(raw + dt_bias); keys B and queries C are shared by
 * heads / groups heads; S = decay S + B (dt x)^T, y = S^T C + d_skip x.  proj row = [heads*vdim z | heads*vdim x |
 * groups*n_state B | groups*n_state C | heads raw dt]; x, B and C pass a causal convolution (conv_w [taps, channels] fp32,
 * conv_b) and silu.  y * silu(z) leaves as y [n_tok, heads*vdim] fp32.  conv_state as for group_prep; state [slots, heads,
 * n_state, vdim]. */
typedef struct {
  const void* proj; int64_t proj_stride;
  const float *conv_w, *conv_b, *dt_bias, *a_log, *d_skip;
  void* conv_state;
  float* state;
  const int32_t *tok_seq, *slot, *start, *cu;
  float* y;
  int32_t n_tok, n_seq, n_decode, heads, vdim, n_state, groups, taps;
  int32_t dtype;
} msa_lm_ssd_args;
/* Decode sequences: everything up to y. */
int msa_lm_ssd_decode(const msa_lm_ssd_args* a, void* stream);
/* The other sequences: xbc [rows, channels] in dtype, dt [rows, heads] fp32 (rows count from the first non-decode token). */
int msa_lm_ssd_prep(const msa_lm_ssd_args* a, void* xbc, float* dt, void* stream);
/* ... the recurrence token by token (n_state up to 256). */
int msa_lm_ssd_scan(const msa_lm_ssd_args* a, const void* xbc, const float* dt, void* stream);
/* ... or in chunks of 64 tokens on tensor cores (bf16; n_state and vdim multiples of 8 up to 128): gcum [rows, heads]
 * fp64 and work [n_chunks, heads, n_state, vdim] fp32 are scratch. */
int msa_lm_ssd_chunk_supported(int32_t n_state, int32_t vdim);
int msa_lm_ssd_chunk(const msa_lm_ssd_args* a, const void* xbc, const float* dt, const int32_t* chunk_off, int32_t n_chunks, double* gcum,
                     float* work, void* stream);

/* out = x / rms(x) * w, every row in `parts` equal parts with a root mean square each. */
int msa_lm_part_norm(const float* x, int64_t x_stride, const float* w, int32_t n_rows, int32_t width, int32_t parts, float eps, void* out,
                     int64_t out_stride, int32_t dtype, void* stream);

/* ---- mixtures of experts -------------------------------------------------------------------------------------------
 * Router logits (fp32) + bias -> the top experts of every row (ties: lower index) and the softmax over their logits. */
int msa_lm_moe_topk(const float* logits, int64_t stride, const float* bias, int32_t n_rows, int32_t experts, int32_t top,
                    int32_t* idx, float* weight, void* stream);
/* Groups the n_rows*top choices by expert: src[i] = row of the i-th grouped entry, inv[r*top+k] = its place,
 * off[e] .. off[e+1] the entries of expert e, tiles [max_tiles, 2] = (expert, first entry) of every tile of tile_rows
 * entries (expert -1: unused).  counts: int32 [ceil(n_rows*top / 2048), experts] lets many choices be sorted by many
 * blocks (null: one block). */
int msa_lm_moe_sort(const int32_t* idx, int32_t n_rows, int32_t top, int32_t experts, int32_t tile_rows, int32_t* src,
                    int32_t* inv, int32_t* off, int32_t* tiles, int32_t max_tiles, int32_t* counts, void* stream);
/* out[i] = x[src[i]] (rows of row_bytes, a multiple of 16). */
int msa_lm_gather_rows(const void* x, int64_t x_stride_bytes, const int32_t* src, int32_t n, int32_t row_bytes, void* out,
                       void* stream);
/* Grouped product over the tiles of msa_lm_moe_sort (tile_rows = 32): out[i] = x[src ? src[i] : i] . w[e]^T with
 * w [experts, n_out, k].  act = 1: w holds gate rows then up rows (n_out = 2*ff) and out[i, ff] = g * sigmoid(1.702 g) *
 * (u + 1) with g = min(gate, limit), u = clamp(up, -limit, limit). */
int msa_lm_moe_gemm(const void* x, int64_t x_stride, const int32_t* src, const void* w, const int32_t* off,
                    const int32_t* tiles, int32_t max_tiles, int32_t n_out, int32_t k, int32_t act, float limit, void* out,
                    int64_t out_stride, int32_t out_dtype, int32_t dtype, void* stream);

/* The same on tcgen05 (bf16; tiles of msa_lm_moe_sort with tile_rows = 128; k, output columns and strides multiples of 8):
 * x has x_rows rows, out is bf16.  A wait that runs out sets status[0]. */
int msa_lm_moe_gemm_tc(const void* x, int64_t x_stride, int32_t x_rows, const int32_t* src, const void* w, int32_t experts,
                       const int32_t* off, const int32_t* tiles, int32_t max_tiles, int32_t n_out, int32_t k, int32_t act,
                       float limit, void* out, int64_t out_stride, int32_t* status, void* stream);

#ifdef __cplusplus
}
#endif
#endif
