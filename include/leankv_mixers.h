/*
 * leankv_b200 — C ABI of the token mixers and dense layers beside the TEAL / TurboQuant paths:
 * row-major dense GEMV with fused norms / token shift / gating / residual, window + pooled-block
 * attention with mixed heads, the matrix-state time mixing recurrence, and causal attention (whole sequence or
 * window) over per-head keys or a shared latent.
 *
 * Conventions are those of leankv_b200.h (device pointers unless marked host, stream as void*, status
 * codes, nothing allocated or synchronised, every call may be captured into a CUDA graph). Storage types
 * are given per call: weights, caches and GEMM operands are bf16 or fp32; the residual stream, small
 * parameter vectors, scores, recurrent state and every vector handed from one decode kernel to the next
 * are fp32.
 *
 * state: int32[8] as leankv_b200.h describes it; word 6 (parity) selects which half of the
 * double-buffered previous-token vectors the current step reads.
 */
#ifndef LEANKV_MIXERS_H
#define LEANKV_MIXERS_H

#include <stddef.h>
#include <stdint.h>

#ifdef __cplusplus
extern "C" {
#endif

#define LEANKV_DT_BF16 1
#define LEANKV_DT_F32 2
#define LEANKV_MAX_MIX 8        /* row segments with a token-shift coefficient of their own */

/* y[rows] = epilogue( W x' ), W row-major [rows][cols] ([2 rows][cols], gate rows first, if gated).
 *   x' = x                                                   gain == NULL
 *   x' = h := gain * x / sqrt(mean(x^2) + eps)               gain: one number, or one per column
 *   x' = h + (prev - h) * mu_s                               rows of segment s, mu[s] != NULL
 * prev is [2][cols]: half state[6] is read, h is written to the other half.
 *   delta != NULL: a branch joins the stream first, x := x + post_mult * post_gain * delta / sqrt(mean(delta^2) + eps)
 *     (post_gain per column), and that x goes to x_out (not x itself, not read by this launch).
 *   group_rows > 0: rows g * group_rows .. belong to group g and multiply x + g * group_stride (no gain, no delta).
 *   epilogue: y = acc + bias (first bias_rows rows);  gated: y = silu(acc_gate) * acc_up;
 *             softcap > 0: y = softcap * tanh(y / softcap);
 *             residual != NULL: y = residual + scale * acc (y may be residual; x may not be y). */
typedef struct leankv_dense_gemv {
    const void* w;
    const float* x;
    float* y;
    int dtype, rows, cols, gated;
    const float* gain;
    float eps;
    int n_mix;
    int mix_end[LEANKV_MAX_MIX];
    const float* mu[LEANKV_MAX_MIX];
    float* prev;
    const int32_t* state;
    const float* bias;
    int bias_rows;
    const float* scale;
    const float* residual;
    int gain_per_col;
    const float* delta;
    const float* post_gain;
    float post_mult;
    float* x_out;
    int group_rows, group_stride;
    float softcap;
} leankv_dense_gemv_t;

int leankv_dense_gemv(const leankv_dense_gemv_t* args, void* stream);

/* x = fp32(table[*token]) ; token = argmax of fp32 logits (see leankv_decode_begin / _end), parity flipped. */
int leankv_embed_begin(const void* table, int dtype, const long long* token, float* x, int width, int vocab,
                       int32_t* state, void* stream);
int leankv_greedy_end(const float* logits, int vocab, long long* token, long long* history, int history_cap,
                      int32_t* state, void* stream);

/* Rows of a prompt portion: x_out = x_in + scale * delta (delta NULL: x_out is not written and may be
 * NULL; post_gain given, per column: x_in + post_mult * post_gain * rms(delta), no scale), h = gain * rms(x_out) (gain one
 * number, or one per column; NULL with h: only the sum), and for each of n_mix coefficient vectors mixed[i] = h + (h' - h) * mu[i], h' the row
 * above (row 0: prev_in). h may be NULL. h of the last row goes to prev_out. delta is of type
 * delta_dtype, h and mixed [n_mix][rows][width] of type dtype. prev_in and prev_out must differ. */
typedef struct leankv_stream_norm {
    const float* x_in;
    float* x_out;
    const void* delta;
    const float* scale;
    const float* gain;
    void* h;
    void* mixed;
    const float* mu[LEANKV_MAX_MIX];
    const float* prev_in;
    float* prev_out;
    int dtype, delta_dtype, rows, width, n_mix;
    float eps;
    int gain_per_col;
    const float* post_gain;
    float post_mult;
} leankv_stream_norm_t;

int leankv_stream_norm(const leankv_stream_norm_t* args, void* stream);

/* out = silu(gate) * up; gate_up [rows][2 * inter], gate columns first. */
int leankv_silu_mul(const void* gate_up, void* out, int dtype, int rows, int inter, void* stream);

/* x = cap * tanh(x / cap), in place. */
int leankv_softcap(float* x, long long n, float cap, void* stream);

/* bf16: out [rows][2 n] = {hi, lo} with hi + lo = tanh(in) to 16 bits; fp32: out [rows][n] = tanh(in). */
int leankv_tanh_split(const float* in, void* out, int dtype, int rows, int n, void* stream);

/* Window + pooled-block attention: position i sees the tokens j with 0 <= i - j < size, and one key and
 * value for every block of `pool` tokens that ends at or before i - size. Raw keys / values live in rings of
 * `ring` slots (position p in slot p % ring, [ring][kv_heads][dim_pad]), pooled ones in [block][kv_heads][..].
 * dim_pad / vdim_pad: multiples of 16, padding zero. */
typedef struct leankv_window_pool {
    int dtype, heads, kv_heads, dim, vdim, dim_pad, vdim_pad;
    int size, pool, ring, max_blocks;
    float scale;
    void* k_ring;
    void* v_ring;
    void* k_pool;
    void* v_pool;
    const float* q_norm;      /* [heads * dim], NULL: q is not normed */
    const float* k_norm;      /* [kv_heads * dim] */
    float eps;
    const float* talk;        /* [heads][heads], NULL: weights are not mixed across heads */
} leankv_window_pool_t;

/* Portion of `rows` tokens at positions start..: rows of qkv (fp32 [rows][ld], q | k | v columns; bias
 * (may be NULL) added) -> normed q [rows][heads][dim_pad] of the storage type, k / v into the ring, and the
 * blocks that become complete into the pool. rows + max(size, pool) - 1 <= ring. */
int leankv_window_pool_append(const leankv_window_pool_t* a, const float* qkv, int ld, const float* bias, void* q,
                              int rows, int start, void* stream);
/* out[row][heads * vdim] (storage type, row stride out_ld elements) = out_scale * attention of those rows. */
size_t leankv_window_pool_workspace_bytes(const leankv_window_pool_t* a, int rows, int max_pos);
int leankv_window_pool_attend(const leankv_window_pool_t* a, const void* q, void* out, int out_ld, float out_scale,
                              int rows, int start, void* ws, size_t ws_bytes, void* stream);

/* Time mixing: per head o_t = (S + diag(u) k v^T)^T r, S = diag(w_t) S + k v^T, w = exp(-exp(z + w0)).
 * S fp32 [heads][dim key][dim value]. */
typedef struct leankv_time_mix {
    int dtype, heads, dim;
    float* S;
    const float* u;           /* [heads * dim] */
    const float* w0;          /* [heads * dim] */
    const float* norm;        /* [heads * dim] */
    float eps;
} leankv_time_mix_t;

/* Portion of `rows` tokens. r, k, v, g: storage type [rows][heads * dim]; z fp32 [rows][heads * dim];
 * out[row][heads * dim] (storage type, row stride out_ld) = out_scale * rms(o) * norm * silu(g). */
size_t leankv_time_mix_workspace_bytes(const leankv_time_mix_t* a, int rows);
int leankv_time_mix_rows(const leankv_time_mix_t* a, const void* r, const void* k, const void* v, const void* g,
                         const float* z, void* out, int out_ld, float out_scale, int rows, void* ws, size_t ws_bytes,
                         void* stream);

/* One decode step of both mixers in one launch (either may be NULL). y: fp32 projections of the step's
 * token, q | k | v at qkv_off and r | k | v | g at rkvg_off, low-rank decay input (rank numbers) at w1_off; w2
 * [heads * dim][rank] of the storage type. The position state[0], the rings and the pooled blocks may be read
 * before the launch just ahead of this one has finished: that launch must not write them. out fp32: left at 0, right at right_off, each times its scale. */
typedef struct leankv_mixer_step {
    const float* y;
    int qkv_off, rkvg_off, w1_off, rank;
    const void* w2;
    float* out;
    int right_off;
    float left_scale, right_scale;
    const int32_t* state;
    int max_pos;              /* positions stay below this */
    void* ws;
    size_t ws_bytes;
} leankv_mixer_step_t;

size_t leankv_mixer_step_workspace_bytes(const leankv_window_pool_t* left, int max_pos);
int leankv_mixer_step(const leankv_window_pool_t* left, const leankv_time_mix_t* right,
                      const leankv_mixer_step_t* step, void* stream);

/* ---- causal attention over a ring of keys -------------------------------------------------------------
 * Position i sees the positions j with 0 <= i - j < size. A key is `dim` numbers of its kv head and, after them,
 * shared_dim numbers common to all heads (0: none); query head h reads kv head h / (heads / kv_heads). Position p
 * lies in slot (p - base) % ring. v NULL: the value is the first vdim numbers of the key's own part (a latent).
 * Paddings are multiples of 16 and zero; slots hold finite numbers. */
typedef struct leankv_causal_attn {
    int dtype, heads, kv_heads;
    int dim, shared_dim, vdim, dim_pad, shared_pad, vdim_pad;
    int size;
    float scale;
    void* k;                  /* [k_ring][kv_heads][dim_pad], the first k_rows slots are there */
    void* v;                  /* [k_ring][kv_heads][vdim_pad] */
    int k_base, k_ring, k_rows;
    void* shared;             /* [s_ring][shared_pad], base 0 */
    int s_ring;
} leankv_causal_attn_t;

/* Rows of a portion on their way into operand buffers and rings. Segment: element i < n of head h of row r at
 * src[r * ld + h * head_stride + i] -> dst[slot * dst_ld + h * dst_head_stride + i] (storage type), i in n .. n_pad
 * zero; slot = (start + r) % ring, or r without a ring. gain (heads == 1): RMS-normed over n. rot: coordinates
 * 2i, 2i + 1 < rot of every head turn by (start + r) * rate[i]. */
#define LEANKV_MAX_SEGMENTS 4
typedef struct leankv_row_segment {
    const float* src;
    int ld, heads, head_stride, n;
    void* dst;
    int dst_ld, dst_head_stride, n_pad, ring;
    const float* gain;
    int rot;
} leankv_row_segment_t;
typedef struct leankv_place_rows {
    int dtype, rows, start, n_seg;
    leankv_row_segment_t seg[LEANKV_MAX_SEGMENTS];
    const float* rate;
    float eps;
} leankv_place_rows_t;

int leankv_place_rows(const leankv_place_rows_t* args, void* stream);

/* Attention of `rows` tokens at positions start.., whose keys are in place. q [rows][heads][dim_pad + shared_pad] of the
 * storage type; out [rows][heads * vdim] (storage type, row stride out_ld), times the logistic function of gate (fp32,
 * row stride gate_ld; NULL: none). status: int32 set non-zero if a wait inside the kernel ran out. */
int leankv_causal_attend(const leankv_causal_attn_t* a, const void* q, const float* gate, int gate_ld, void* out,
                         int out_ld, int rows, int start, int32_t* status, void* stream);

/* One decode step at position state[0] < max_pos: rotates the query and the new key, stores the key / value, attends.
 * fp32 inputs: q [heads] x dim numbers (stride q_stride), q_shared [heads] x shared_dim (stride qs_stride), k_new
 * [kv_heads][dim], shared_new [shared_dim], v_new [kv_heads][vdim] (unused if a->v is NULL). k_gain: k_new is RMS-normed
 * over dim (kv_heads == 1). rot_own / rot_shared: rotated coordinates of either part. out fp32 [heads][vdim]; gate
 * fp32 [heads * vdim] or NULL. state[0] and the rings may be read before the launch just ahead has finished: that
 * launch must not write them. ws: leankv_causal_step_workspace_bytes, zeroed once before the first call. */
typedef struct leankv_causal_step {
    const float* q;
    const float* q_shared;
    const float* k_new;
    const float* shared_new;
    const float* v_new;
    int q_stride, qs_stride;
    const float* k_gain;
    float eps;
    const float* rate;
    int rot_own, rot_shared;
    const float* gate;
    float* out;
    const int32_t* state;
    int max_pos;
    void* ws;
    size_t ws_bytes;
} leankv_causal_step_t;

size_t leankv_causal_step_workspace_bytes(const leankv_causal_attn_t* a, int max_pos);
int leankv_causal_step(const leankv_causal_attn_t* a, const leankv_causal_step_t* step, void* stream);

#ifdef __cplusplus
}
#endif

#endif /* LEANKV_MIXERS_H */
