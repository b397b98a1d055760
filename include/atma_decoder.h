/*
 * atma_decoder - C ABI of the B200 (sm_100a) kernels for decoder-only language models that are assembled from a
 * configuration: softmax attention over a paged cache (one or two maps per head, rotary positions from a table or
 * norms over the whole projections, sliding windows with kept first keys, a sink, an output gate), the gated delta
 * rule with per-head decay behind short convolutions, and the row operations around them (fp32 residual stream, RMS
 * norms in front of or behind a sublayer, bigram or learned-position embedding, feed-forward activations).
 *
 * Conventions as in atma_b200.h: plain device pointers, element strides, a CUDA stream passed as void*; nothing
 * allocates or synchronises; every call returns ATMA_OK or a negative atma_status and leaves a message for
 * atma_last_error().  dtype is that of activations, caches and weights: ATMA_F32 or ATMA_BF16.  Residual stream,
 * norms, scores, softmax weights, decays, step sizes, unit norms and recurrent state are fp32 in both.
 *
 * A step's rows are its sequences' new tokens back to back; sequence s owns rows cu_rows[s] .. cu_rows[s+1]-1, its
 * first row stands at position start_pos[s] (a negative start_pos marks a padded sequence of one row: nothing of
 * the caches or states is touched and its outputs are zero).
 */
#ifndef ATMA_DECODER_H_
#define ATMA_DECODER_H_

#include "atma_b200.h"

#ifdef __cplusplus
extern "C" {
#endif

int atma_decoder_abi_version(void);

/* x[row] = embed[ids[row]] + bigram[r], fp32 [rows][D].  r = (prev * mul_prev + id * mul_cur) mod buckets, or
 * `buckets` (the table's last row) where prev[row] < 0.  bigram NULL = no second term. */
int atma_embed_bigram(const int32_t* ids, const int32_t* prev, const void* embed, const void* bigram, float* x, int rows, int D,
                      int vocab, int64_t mul_prev, int64_t mul_cur, int64_t buckets, int dtype, void* stream);

/* x += y (y NULL = nothing to add; x_out receives the sum, may equal x, NULL = not stored), then for each non-NULL
 * h: h = x / sqrt(mean x^2 + eps) * (offset + w).  Two norms of the same sum share one pass. */
int atma_residual_norms(const float* x, const void* y, float* x_out, const void* w1, void* h1, const void* w2, void* h2, int rows,
                        int D, float eps, float offset, int dtype, void* stream);

/* s = embed[ids[row]] * scale + pos[positions[row]] (pos NULL = no second term); x = s / sqrt(mean s^2 + eps) *
 * (offset + w), fp32 [rows][D]; h (NULL = not stored) receives x in the activation dtype. */
int atma_embed_position_norm(const int32_t* ids, const int32_t* positions, const void* embed, const void* pos, const void* w, float* x,
                             void* h, int rows, int D, int vocab, int max_positions, float scale, float eps, float offset, int dtype,
                             void* stream);

/* Norm on a sublayer's output: t = y + bias (bias NULL = none), x += t / sqrt(mean t^2 + eps) * (offset + w); x_out
 * receives the sum (may equal x, NULL = not stored).  h (NULL = not stored) receives the sum in the activation dtype
 * or, with w_next, the sum's own norm times (offset + w_next). */
int atma_residual_post_norm(const float* x, const void* y, const void* bias, const void* w, float* x_out, void* h, const void* w_next,
                            int rows, int D, float eps, float offset, int dtype, void* stream);

/* out = relu(z + bias)^2 (bias NULL = none; out may be z), row strides in elements. */
int atma_bias_squared_relu(const void* z, int64_t z_rs, const void* bias, void* out, int64_t out_rs, int rows, int width, int dtype,
                           void* stream);

/* out = gelu_tanh(gate) * up, row strides in elements. */
int atma_gelu_gate(const void* gate, int64_t gate_rs, const void* up, int64_t up_rs, void* out, int64_t out_rs, int rows, int width,
                   int dtype, void* stream);

/* out[row][h][:] = o[row][h][:] / sqrt(mean o^2 + eps) * w * silu(gate[row][h][:]); o dense, heads of vdim channels. */
int atma_head_norm_silu_gate(const void* o, const void* w, const void* gate, int64_t gate_rs, void* out, int64_t out_rs, int rows,
                             int H, int vdim, float eps, int dtype, void* stream);

/* Rotary positions and cache write in one pass.  z rows hold [q: H*maps*dim | k: G*maps*dim | v: G*vdim].  In every
 * map of every q and k head channels 2i and 2i+1, i < rot_dims/2, are turned by the table's (cos, sin) at the row's
 * position; q goes to q_out (dense), k and v to row slot_mapping[row] of the caches (negative = not stored). */
int atma_rotary_store(const void* z, int64_t z_rs, const int32_t* positions, const int64_t* slot_mapping, const float* cos_sin,
                      int table_rows, void* q_out, void* k_cache, void* v_cache, int rows, int H, int G, int maps, int dim, int vdim,
                      int rot_dims, int dtype, void* stream);

/* Norms over whole projections, value mixing and cache write in one pass.  z rows hold [q: q_width | k: k_width |
 * v: v_width].  q / sqrt(mean q^2 + eps) * wq goes to q_out (dense), k / sqrt(mean k^2 + eps) * wk to row
 * slot_mapping[row] of the k cache (wq, wk NULL = that part as it is), v or, with v_first,
 * (1 - lambda) v + lambda v_first[row] to the same row of the v cache.  A negative slot is not stored. */
int atma_norm_store(const void* z, int64_t z_rs, const int64_t* slot_mapping, const void* wq, const void* wk, const void* v_first,
                    int64_t v_first_rs, float lambda, float eps, void* q_out, void* k_cache, void* v_cache, int rows, int q_width,
                    int k_width, int v_width, int dtype, void* stream);

/* Causal softmax attention of a step's rows over a paged cache that already holds their own keys.
 * q dense [rows][H][maps][dim]; k_cache [num_blocks*block_size][G][maps][dim]; v_cache [..][G][vdim]; query head h
 * reads key/value head h / (H/G).  maps = 1: out = attention.  maps = 2: both maps attend over the same values and
 * o = a1 - lambda * a2 is divided by its root mean square over vdim (eps inside the root) and multiplied by out_scale.
 * Position i sees key j <= i if i - j < window (INT_MAX = every key) or j < keep_first.  sink: the score of an added
 * key that has no value and only enters the denominator (-INFINITY = none).  gate [rows][H*vdim] (NULL = none): the
 * result is multiplied by sigmoid(gate). */
typedef struct {
  const void* q; const void* k_cache; const void* v_cache;
  const int32_t* block_tables; int64_t bt_stride;
  const int32_t* cu_rows;            /* [n_seqs + 1] */
  const int32_t* start_pos;          /* [n_seqs] */
  void* out; int64_t out_rs;         /* [rows][H*vdim] */
  float* scratch;                    /* atma_softmax_decode only: atma_softmax_decode_scratch_floats() */
  const int32_t* tile_seq;           /* atma_softmax_prefill, tensor-core path: sequence and first row (inside the */
  const int32_t* tile_row;           /* sequence) of every 128-row query tile; may be NULL for the other path */
  int n_tiles;
  int n_seqs, max_rows, total_rows;  /* max_rows: the longest sequence of the step */
  int H, G, maps, dim, vdim;
  int num_blocks, block_size, max_blocks, n_splits, dtype;
  float scale, lambda, out_scale, eps;
  const void* gate; int64_t gate_rs;
  int window, keep_first;
  float sink;
} atma_softmax_args;

int atma_softmax_prefill(const atma_softmax_args* args, void* stream);
/* 1 = the tensor-core kernel serves this shape, 0 = the fp32-arithmetic kernel does. */
int atma_softmax_prefill_path(const atma_softmax_args* args);
/* One row per sequence.  n_splits > 1 or a supported 16-bit shape: key ranges side by side, merged afterwards. */
int atma_softmax_decode(const atma_softmax_args* args, void* stream);
int atma_softmax_decode_path(const atma_softmax_args* args);
int64_t atma_softmax_decode_scratch_floats(int n_seqs, int H, int maps, int vdim, int n_splits);

/* Gated delta rule.  z rows hold [q: G*dim | k: G*dim | v: H*vdim | gate: H*vdim | a: H | b: H].  q, k, v pass a
 * causal depthwise convolution of `taps` taps and silu; q and k are made unit vectors (x / sqrt(sum x^2 + unit_eps),
 * q also times q_scale); log decay = -exp(A_log) * softplus(a + dt_bias), beta = sigmoid(b).
 * conv_table [slots][taps][2*G*dim + H*vdim] holds raw inputs by position mod taps; state_table [slots][H][dim][vdim]
 * fp32.  A sequence at position 0 starts from zero whatever its rows hold. */
typedef struct {
  const void* z; int64_t z_rs;
  const void* conv_q; const void* conv_k; const void* conv_v;   /* [channels][taps] */
  const float* A_log; const float* dt_bias;                      /* [H] */
  void* conv_table; int64_t conv_ss;                             /* elements between slots */
  float* state_table; int64_t state_ss;
  const int64_t* slots;                                          /* [n_seqs] */
  const int32_t* cu_rows; const int32_t* start_pos;              /* [n_seqs + 1], [n_seqs] */
  const int32_t* row_seq;                                        /* [rows] sequence of every row (prefill) */
  int n_seqs, total_rows, H, G, dim, vdim, taps, dtype;
  float unit_eps, q_scale;
} atma_delta_args;

/* Convolutions, unit-norm factors and gates of a step's rows: q, k [rows][G][dim], v [rows][H][vdim] (dtype),
 * q_inv, k_inv [rows][G], log_decay, beta [rows][H] fp32; then the convolutions' state. */
int atma_delta_prepare(const atma_delta_args* args, void* q, void* k, void* v, float* q_inv, float* k_inv, float* log_decay,
                       float* beta, void* stream);
/* The recurrence over those rows, state in and out through the slot table; o [rows][H][vdim] (dtype).  scratch:
 * atma_delta_scan_scratch_bytes() bytes (chunk factors of the tensor-core path; 0 for other shapes). */
int atma_delta_scan(const atma_delta_args* args, const void* q, const void* k, const void* v, const float* q_inv, const float* k_inv,
                    const float* log_decay, const float* beta, void* o, void* scratch, void* stream);
int atma_delta_scan_path(const atma_delta_args* args);
int64_t atma_delta_scan_scratch_bytes(const atma_delta_args* args);
/* One token per sequence, everything in one launch: convolutions, gates, recurrence, per-head norm with weight
 * `norm_w` [vdim], silu gate; out [n_seqs][H*vdim]. */
int atma_delta_step(const atma_delta_args* args, const void* norm_w, void* out, int64_t out_rs, float eps, void* stream);

/* Status word of this library's tensor-core kernels (see atma_device_status). */
int atma_decoder_device_status(int* status);

#ifdef __cplusplus
}
#endif
#endif
