/*
 * atoma_hybrid.h — operators and the step executor for models whose layers mix attention with
 * recurrent (state-carrying) mixers, run on MIXED batches: portions of prompts beside single decoded
 * tokens, keys and values in a paged cache, recurrent state in per-sequence slots.
 *
 * The first design served through it is Lilovik: sandwich RMS norms (weights stored as offsets from
 * one), a sinusoidal position signal on the embedding, sigmoid attention (no softmax) with a
 * whole-projection q/k norm, a position-dependent query temperature, a tanh soft cap, a linear
 * distance bias and a talking-heads mix of the attention weights, minGRU layers, and a ReLU-gated
 * feed-forward.  Every constant of those mechanisms is an argument, so that another design can use
 * the operator with other values.
 *
 * The second design is Patadra: a learned position table, pre-norm layers with RMS norms taken over
 * equal consecutive groups of the row, sublayer results gated by a sigmoid of a projection of the
 * sublayer's input before they join the residual stream, latent attention (queries, keys and values
 * expanded from low-rank latents; only the key/value latent is cached) under a sliding window with a
 * per-head softmax sink, a mixture-of-experts feed-forward with a sigmoid router whose score scales the
 * expert's INPUT, a clamped gated activation, an always-on shared expert, a per-layer token input
 * looked up in a side table, and a tanh cap on the logits.  A span of layers may run several times
 * with the same weights; every run is one entry of the layer list with a cache of its own.
 *
 * The third design is Nemasun: a scaled embedding without a position signal, several residual LANES
 * (copies of the residual stream; every sublayer reads a weighted sum of them and writes its result
 * back through a lane-mixing matrix — the arrangement known as hyper-connections), softmax attention
 * with grouped key/value heads whose values are the un-normed key projections, a per-head q/k RMS
 * norm, a learned bias looked up by query-key distance, a sliding window that also keeps the first
 * tokens of the sequence, and a sigmoid gate on the heads' outputs; a clamped gated feed-forward with
 * biases; and a mixture of experts with a softmax router whose choice (not its weights) carries a
 * per-output correction and is restricted to the best groups of neighbouring outputs, with identity
 * experts (router outputs that hand the token's input through) and an ungated shared expert.
 *
 * The fourth design is Surinex: PARALLEL blocks (one RMS norm per layer whose output both the mixer and the
 * feed-forward read, each through its own causal tap filter over time whose last inputs are carried as state;
 * x <- x + mixer + feed-forward), three mixers — gated linear attention (a matrix state per head whose rows decay
 * by a data-dependent factor per key channel), latent attention with one rotated key part shared by all heads
 * beside the cached latent, and a PAIR of mixers on the same input: sigmoid attention with rotary positions on
 * queries, keys AND values (a head's sum is turned back by the query's position) beside a gated delta rule
 * (short causal filters with silu on q / k / v, unit-length q and k, a scalar decay and a write strength per
 * head), each result RMS-normed over the model width before the two are averaged — and a span of layers that
 * runs several times with the embedding added again and a per-pass vector at the start of every pass.
 *
 * The fifth design is Mobunex: POST-NORM blocks (x <- norm(alpha x + sublayer(x)), the sublayer reads the stream itself, a norm's
 * weight is one number), a depth average after every layer (what goes on is a learned weighted sum of the embedding output and of
 * every layer's result so far), grouped softmax attention under a sliding window with projection biases, unweighted per-head q/k
 * norms and a factor per head on the score, a recurrent block with a real-gated linear recurrent unit (short causal filter,
 * block-diagonal gates, a decay per channel and token), latent attention with a rotated key part (YaRN-scaled frequencies) under a
 * sliding window with a sigmoid gate on the heads' outputs, and a mixture of experts whose groups are ranked by the sum of their two
 * best choice scores.
 *
 * The sixth design is Lusalorn: blocks that norm the sublayer's RESULT only (x <- x + m norm(sublayer(x)), the sublayer reads the stream
 * itself), an embedding with a second row looked up by a hash of the pair (token before, token), differential attention (two softmax
 * maps per head over the same values, combined as a1 - lambda a2 at unit root mean square) under a sliding window with projection
 * biases, layers that read an earlier layer's cached keys and values, and a SUM of two mixers on the same input: softmax attention with
 * rotary positions (YaRN-scaled) beside a state-space recurrence (short causal filter, a scalar decay and a step size per head and
 * token, keys and queries shared by groups of heads, a skip term, a gate before a grouped norm).
 *
 * Conventions: row-major; `dtype` is the number format of activations, large weights and the caches:
 * 1 = bfloat16, 2 = float32 (true 32-bit arithmetic: no reduced-precision matrix mode).  Whatever the
 * dtype, the residual stream, norm statistics, attention scores and weights, recurrent state and all
 * small per-channel parameters (norm weights, biases, per-head tables) are float32.  Everything is
 * stream-ordered and allocates nothing (library workspaces excepted).  Errors: atoma_last_status()
 * / atoma_last_error() (atoma_flash.h).
 */
#ifndef ATOMA_HYBRID_H_
#define ATOMA_HYBRID_H_

#include <stdint.h>

#include "atoma_flash.h"

#ifdef __cplusplus
extern "C" {
#endif

#define ATOMA_DTYPE_BF16 1u
#define ATOMA_DTYPE_F32 2u

/* out[t, 2i] = table[tokens[t], 2i] + sin(positions[t] * inv_freq[i]), out[t, 2i+1] = ... + cos(same); the angle is
 * formed and reduced in double precision (inv_freq [ceil(width/2)] is a device table of doubles). */
void atoma_embed_sinusoid(const uint32_t *tokens, const int64_t *positions, const void *table, const double *inv_freq,
                          float *out, int64_t T, int64_t width, int64_t vocab, uint32_t dtype, atoma_stream_t stream);

/* out[r, :] = x[rows ? rows[r] : r, :] / sqrt(mean(x^2) + eps) * (weight_offset + weight); x float32, out `dtype`. */
void atoma_rmsnorm_rows(const float *x, const int32_t *rows, const float *weight, float weight_offset, void *out,
                        int64_t R, int64_t width, float eps, uint32_t dtype, atoma_stream_t stream);

/* Sandwich-norm residual update and the next sublayer's input norm in ONE kernel:
 *   x[t, :] += rms(y[t, :]) * (weight_offset + w_post);   h[t, :] = rms(x[t, :]) * (weight_offset + w_pre)
 * y, h in `dtype`, x float32 in place; w_pre / h may be NULL (no following norm). */
void atoma_postnorm_add_prenorm(const void *y, float *x, const float *w_post, const float *w_pre, void *h, int64_t T,
                                int64_t width, float eps, float weight_offset, uint32_t dtype, atoma_stream_t stream);

/* After the fused q/k/v projection qkv [T, H dim + G dim + G vdim] (+ bias, float32, may be NULL):
 *   q <- rms over the WHOLE q part * q_weight * (1 + temp_coef * ln(floor((pos + 1) / temp_every) + 1)) -> q_out [T, H dim]
 *   k <- rms over the WHOLE k part * k_weight -> key cache row slot_mapping[t];   v -> value cache row
 * caches: [num_blocks * block_size, G, dim] and [.., G, vdim] in `dtype`; slot < 0 is skipped. */
void atoma_qk_norm_cache(const void *qkv, const float *bias, const float *q_weight, const float *k_weight,
                         const int64_t *positions, const int64_t *slot_mapping, void *q_out, void *k_cache, void *v_cache,
                         int64_t T, int64_t H, int64_t G, int64_t dim, int64_t vdim, float eps, float temp_coef,
                         int64_t temp_every, uint32_t dtype, atoma_stream_t stream);

/*
 * Sigmoid attention over a paged cache for a mixed batch.  For query token t of sequence b at position p and every
 * cached key j <= p of that sequence:
 *   s = (q_g . k_j) * scale;  s = softcap * tanh(s / softcap) (softcap > 0);  s -= slopes[g] * (p - j)
 *   a_g = sigmoid(s + head_bias[g]);   a'_h = sum_g talk[h, g] a_g  (talk NULL = identity)
 *   out[t, h, :] = sum_j a'_h(j) v_j[kv head of h, :]
 * Scores, weights and the sums are float32; keys are visited in position order whatever the batch looks like.
 */
typedef struct atoma_sigmoid_attn_args {
    const void *q;                /* [T, H dim] */
    const void *k_cache, *v_cache;
    void *out;                    /* [T, H vdim] */
    const int64_t *positions;     /* [T] */
    const int32_t *token_seq;     /* [T] batch row of every token */
    const int32_t *query_start;   /* [B + 1] first token of every batch row (rows are contiguous, positions ascending) */
    const int32_t *block_tables;  /* [B, max_blocks] */
    const float *slopes, *head_bias, *talk; /* [H] (NULL: no distance term), [H], [H, H] (NULL: the heads do not talk) */
    int64_t T, B, max_blocks, H, G, dim, vdim, block_size;
    float scale, softcap;
    uint32_t dtype;
    int32_t max_query_len;        /* longest portion of the batch (1 = decode only): selects the kernel */
    int32_t max_seq_len;          /* longest sequence (context + portion) of the batch; 0 = unknown (keys are not split) */
} atoma_sigmoid_attn_args;
void atoma_sigmoid_attention_paged(const atoma_sigmoid_attn_args *args, atoma_stream_t stream);

/*
 * minGRU over a mixed batch.  zxg [T, 3 S] = the fused projections (rows: update gate, candidate, output gate) with
 * bias [3 S] (may be NULL) added here.  Per sequence b (tokens query_start[b] .. query_start[b+1]) and channel c:
 *   z = sigmoid(zpre), cand = u >= 0 ? u + 1/2 : sigmoid(u),  s <- (1 - z) s + z cand,  out = s * silu(g)
 * s starts from state[state_slots[b], c] — from zero when context_lens[b] == 0 — and is stored back.  float32 state.
 */
void atoma_mingru_scan(const void *zxg, const float *bias, float *state, const int32_t *state_slots,
                       const int32_t *query_start, const int32_t *context_lens, void *out, int64_t T, int64_t B, int64_t S,
                       int32_t max_query_len, uint32_t dtype, atoma_stream_t stream);

/* out[t, j] = act(gu[t, j]) * gu[t, ff + j]; act: 0 = silu, 1 = relu, 2 = gelu (tanh form). */
void atoma_glu(const void *gu, void *out, int64_t T, int64_t ff, int32_t act, uint32_t dtype, atoma_stream_t stream);

/* y[T, N] = x[T, K] w[N, K]^T.  bfloat16 with 16-byte aligned rows runs the tcgen05 kernels of atoma_gemm_tn;
 * float32 (and whatever those kernels do not take) runs a plain float32-FMA tile kernel. */
void atoma_linear(const void *x, const void *w, void *y, int64_t T, int64_t N, int64_t K, uint32_t dtype,
                  atoma_stream_t stream);

/* logits_f32[r, :] = logits[r, :] * scale and token_out[r] = the last index of the row's maximum. */
void atoma_scale_logits_greedy(const void *logits, float *logits_f32, uint32_t *token_out, int64_t R, int64_t vocab,
                               float scale, uint32_t dtype, atoma_stream_t stream);

/* ------------------------------------------------------------------------------------------ */
/* Pre-norm designs with gated residuals, latent attention and mixtures of experts             */
/* ------------------------------------------------------------------------------------------ */

/* out[t, :] = table[tokens[t], :] + pos_table[positions[t], :] (float32 sum; positions beyond max_positions - 1 are an
 * error the caller must exclude: the kernel clamps). */
void atoma_embed_learned(const uint32_t *tokens, const int64_t *positions, const void *table, const void *pos_table, float *out,
                         int64_t T, int64_t width, int64_t vocab, int64_t max_positions, uint32_t dtype, atoma_stream_t stream);

/* RMS norm in `groups` equal consecutive parts of the row, each divided by its own sqrt(mean(part^2) + eps); the whole
 * row is then multiplied by (weight_offset + weight).  groups = 1 is atoma_rmsnorm_rows.  width % groups == 0. */
void atoma_group_rmsnorm_rows(const float *x, const int32_t *rows, const float *weight, float weight_offset, int64_t groups,
                              void *out, int64_t R, int64_t width, float eps, uint32_t dtype, atoma_stream_t stream);

/*
 * Residual update of a pre-norm layer and the next sublayer's input norm in ONE kernel.  Per token t and channel c:
 *   v = (y ? y[t, c] * (row_scale ? row_scale[t] : 1) : 0) + sum_{k < top} expert_out[pair_row[t top + k], c]
 *   x[t, c] += gate ? v * sigmoid(gate[t, c] + gate_bias[c]) : v
 *   h[t, :]  = group_rmsnorm(x[t, :]) * (weight_offset + w_next)      (w_next NULL: no norm)
 *   x_cast[t, :] = x[t, :] in `dtype`                                  (x_cast NULL: not written)
 * y, gate, expert_out, h, x_cast in `dtype` with row strides ld_y, ld_gate, width, width, width; x float32 in place.
 * The experts' rows are added in the order k = 0 .. top - 1.
 */
typedef struct atoma_gated_residual_args {
    const void *y;
    int64_t ld_y;
    const float *row_scale;       /* [T] or NULL */
    const void *expert_out;       /* [rows, width] or NULL */
    const int32_t *pair_row;      /* [T top] row of expert_out that holds pair (t, k) */
    int64_t top;
    const void *gate;             /* pre-activation of the residual gate, or NULL */
    int64_t ld_gate;
    const float *gate_bias;       /* [width] */
    float *x;                     /* [T, width] */
    const float *w_next;          /* [width] or NULL */
    void *h;                      /* [T, width] */
    void *x_cast;                 /* [T, width] or NULL */
    int64_t T, width, groups;
    float eps, weight_offset;
    uint32_t dtype;
} atoma_gated_residual_args;
void atoma_gated_residual_norm(const atoma_gated_residual_args *args, atoma_stream_t stream);

/* Token side input, gate part: out[t, j] = gelu_tanh(a[t, j]) * side_table[tokens[t], part * dim + j], j < dim.
 * a (row stride ld_a) and out [T, dim] in `dtype`; side_table [vocab, table_width] in `dtype`. */
void atoma_side_gate(const void *a, int64_t ld_a, const uint32_t *tokens, const void *side_table, int64_t table_width, int64_t part,
                     void *out, int64_t T, int64_t dim, int64_t vocab, uint32_t dtype, atoma_stream_t stream);

/* x[t, :] += y[t, :] / sqrt(mean(y^2) + eps) * w_unit;  h[t, :] = group_rmsnorm(x[t, :]) * (weight_offset + w_next) (NULL: none). */
void atoma_unitnorm_add_norm(const void *y, float *x, const float *w_unit, const float *w_next, void *h, int64_t T, int64_t width,
                             int64_t groups, float eps, float weight_offset, uint32_t dtype, atoma_stream_t stream);

/* After the fused down projections proj[t, :] = [c_q (q_rank) | c (kv_rank) | ...] (row stride ld):
 *   cq_out[t, :] = rms(c_q) * q_weight  (q_rank = 0: no query latent)      latent_cache[slot_mapping[t], :] = rms(c) * kv_weight
 * plain weights; cq_out and the cache [num_blocks * block_size, kv_rank] in `dtype`; slot < 0 is skipped. */
void atoma_latent_norm_cache(const void *proj, int64_t ld, const float *q_weight, const float *kv_weight, const int64_t *slot_mapping,
                             void *cq_out, void *latent_cache, int64_t T, int64_t q_rank, int64_t kv_rank, float eps, uint32_t dtype,
                             atoma_stream_t stream);

/* Per-head projection between a head's own space and a shared latent, w [H n, R] (stored [out, in], as the checkpoint has it):
 *   absorb = 1:  out[t, h, r] = sum_j in[t, h n + j] w[h n + j, r]     in [T, H n] `dtype`      -> out [T, H, R] float32
 *   absorb = 0:  out[t, h n + j] = sum_r in[t, h, r] w[h n + j, r]     in [T, H, R] float32    -> out [T, H n] `dtype`
 * The first moves a query into the latent space of the keys (so that q . (W c) = (W^T q) . c needs no expanded keys);
 * the second expands a head's weighted sum of latents into its values. */
void atoma_head_project(const void *in, const void *w, void *out, int64_t T, int64_t H, int64_t n, int64_t R, int32_t absorb,
                        uint32_t dtype, atoma_stream_t stream);

/*
 * Softmax attention of H heads over ONE shared cached latent per token (keys = values = the latent), paged, mixed batch.
 * For query token t of sequence b at position p and keys j with 0 <= p - j < window (window <= 0: every j <= p):
 *   s_h(j) = (q_lat[t, h, :] . c_j) * scale
 *   w_h(j) = exp(s_h(j)) / (sum_j' exp(s_h(j')) + (sink ? exp(sink[h]) : 0))
 *   out[t, h, :] = sum_j w_h(j) c_j
 * q_lat and out float32 [T, H, R]; scores, weights and sums float32.
 */
typedef struct atoma_latent_attn_args {
    const float *q_lat;
    const void *latent_cache;     /* [num_blocks * block_size, R] `dtype` */
    float *out;
    const int64_t *positions;     /* [T] */
    const int32_t *token_seq;     /* [T] */
    const int32_t *query_start;   /* [B + 1] */
    const int32_t *block_tables;  /* [B, max_blocks] */
    const float *sink;            /* [H] or NULL */
    int64_t T, B, max_blocks, H, R, block_size, window;
    float scale;
    uint32_t dtype;
    int32_t max_query_len, max_seq_len;
    int32_t skip_min_q;           /* > 0: sequences with at least this many query tokens in the step are left alone */
    int64_t out_cols;             /* > 0: only the first out_cols entries of every row of `out` are read by the caller (a cached row whose
                                   * tail takes part in the scores only, like a rotated key part); the rest may be left unwritten */
} atoma_latent_attn_args;
void atoma_latent_attention_paged(const atoma_latent_attn_args *args, atoma_stream_t stream);

/*
 * The same attention for LONG prompt portions, on expanded keys and values (bfloat16, values of 64 or 128, keys of up to 64 more
 * entries): for every
 * sequence with at least min_q query tokens in the step, the latents its queries can see (window + portion) are gathered
 * from the paged cache, k = w_uk c and v = w_uv c are formed by two dense products, and softmax attention with the window
 * and the sink runs per head on the 5th-generation tensor cores; out[t, h dim ..] is written for those sequences' tokens
 * only.  A (query, key, head) pair costs 2 (dim + vdim) multiply-adds here instead of 4 kv_rank in the latent space.
 * max_keys: an upper bound of the gathered rows (sum over the long sequences of min(context, window - 1) + tokens).
 * Cached rows with a score-only tail (rot_dim > 0, a rotated key part that all heads share): rows have R + rot_dim entries, query
 * heads dim + rot_dim (their tail already rotated), and w_uk is [H (dim + rot_dim), R + rot_dim] — a head's rows [W_uk_h | 0] and
 * [0 | identity], so that one product makes whole keys; values come from the first R entries.  gate (NULL: none, row stride ld_gate):
 * the result times sigmoid(gate[t, h vdim + j]).
 */
typedef struct atoma_latent_expanded_args {
    const void *q;                /* [T, H dim] */
    const void *latent_cache;
    const void *w_uk, *w_uv;      /* [H dim, R], [H dim, R] */
    void *out;                    /* [T, H dim] */
    const int32_t *query_start;   /* [B + 1] */
    const int32_t *context_lens;  /* [B] */
    const int32_t *block_tables;  /* [B, max_blocks] */
    const float *sink;            /* [H] or NULL */
    int64_t T, B, max_blocks, H, dim, R, block_size, window, max_keys;
    float scale;
    int32_t min_q, max_query_len, max_seq_len;
    int64_t rot_dim, vdim;        /* vdim 0: dim */
    const void *gate;
    int64_t ld_gate;
} atoma_latent_expanded_args;
void atoma_latent_attention_expanded(const atoma_latent_expanded_args *args, atoma_stream_t stream);

/* Router of a mixture of experts, float32: z = w_router h (h [T, width] `dtype`, w_router [experts, width] float32),
 * s = sigmoid(z) (score_fn 0) ; the `top` largest scores (ties: the lower index) -> top_expert [T, top] int32 and
 * top_weight [T, top] float32 = the chosen scores as they are (renormalize 0) or divided by their sum (1).
 * w_row_gate (float32 [width], may be NULL): row_gate[t] = sigmoid(w_row_gate . h[t]) — the shared expert's gate. */
void atoma_moe_route(const void *h, const float *w_router, const float *w_row_gate, int32_t *top_expert, float *top_weight,
                     float *row_gate, int64_t T, int64_t width, int64_t experts, int64_t top, int32_t renormalize, uint32_t dtype,
                     atoma_stream_t stream);

/* y = act(g, u) of a gated feed-forward with clamps: g = min(gu[t, j], limit), u = clamp(gu[t, ff + j], -limit, limit),
 * out[t, j] = g * sigmoid(alpha g) * (u + up_shift).  limit <= 0: no clamp.  gu row stride ld. */
void atoma_glu_clamped(const void *gu, int64_t ld, void *out, int64_t T, int64_t ff, float limit, float alpha, float up_shift,
                       uint32_t dtype, atoma_stream_t stream);

/*
 * The routed experts of a step: every (token, k) pair is sorted by its expert on the device (no host read), its input row
 * h[t] * top_weight[t, k] is gathered (scale_input 1; with 0 the weight multiplies the expert's output instead), and the
 * experts run as two grouped products with the clamped gated activation between them:
 *   expert_out[pair_row[t top + k], :] = w_down[e] act(w_gate_up[e] (weight * h[t]))
 * w_gate_up [experts, 2 ff, width] (gate rows, then up rows), w_down [experts, width, ff], all `dtype`.
 * workspace: atoma_moe_workspace_bytes(T, top, experts, width, ff, dtype) bytes; expert_out and pair_row point into it
 * and are returned through *expert_out / *pair_row for atoma_gated_residual_norm.
 */
typedef struct atoma_moe_args {
    const void *h;                /* [T, width] */
    const int32_t *top_expert;    /* [T, top] */
    const float *top_weight;      /* [T, top] */
    const void *w_gate_up, *w_down;
    void *workspace;
    int64_t workspace_bytes;
    int64_t T, width, experts, top, ff;
    float limit, alpha, up_shift;
    int32_t scale_input;
    uint32_t dtype;
} atoma_moe_args;
int64_t atoma_moe_workspace_bytes(int64_t T, int64_t top, int64_t experts, int64_t width, int64_t ff, uint32_t dtype);
void atoma_moe_experts(const atoma_moe_args *args, const void **expert_out, const int32_t **pair_row, atoma_stream_t stream);

/* logits_f32[r, :] = cap(logits[r, :] * scale), cap(v) = softcap * tanh(v / softcap) (softcap <= 0: identity), and
 * token_out[r] = the last index of the row's maximum. */
void atoma_finish_logits_greedy(const void *logits, float *logits_f32, uint32_t *token_out, int64_t R, int64_t vocab, float scale,
                                float softcap, uint32_t dtype, atoma_stream_t stream);

/* ------------------------------------------------------------------------------------------ */
/* Residual lanes, softmax attention with a distance table, grouped routing                     */
/* ------------------------------------------------------------------------------------------ */

/* x[t, s, :] = table[tokens[t], :] * scale for every lane s < lanes; x float32 [T, lanes, width]. */
void atoma_embed_scaled_lanes(const uint32_t *tokens, const void *table, float scale, float *x, int64_t T, int64_t lanes, int64_t width,
                              int64_t vocab, uint32_t dtype, atoma_stream_t stream);

/* A sublayer's input from the lanes: u = sum_s w_in[s] x[r, s, :] (w_in NULL: the plain sum), r = rows ? rows[i] : i;
 * out[i, :] = u / sqrt(mean(u^2) + eps) * (weight_offset + weight) in `dtype`; sum_out (float32 [R, width], may be NULL) = u. */
void atoma_lanes_read_norm(const float *x, const float *w_in, const int32_t *rows, const float *weight, float weight_offset, void *out,
                           float *sum_out, int64_t R, int64_t lanes, int64_t width, float eps, uint32_t dtype, atoma_stream_t stream);

/*
 * A sublayer's result written back to the lanes, fused with the NEXT sublayer's read and norm.  Per token t, channel c:
 *   v = (y ? y[t, c] : 0) + (y_bias ? y_bias[c] : 0)
 *       + sum_{k < top} (top_expert[t, k] in [0, experts):  expert_out[pair_row[t top + k], c]
 *                        top_expert[t, k] >= experts:        top_weight[t, k] * h_in[t, c]       (identity expert)
 *                        top_expert[t, k] < 0:               nothing)
 *   x'[t, s2, c] = sum_s w_mix[s, s2] x[t, s, c] + w_out[s2] v           (all lanes from the old ones)
 *   u = sum_s w_in_next[s] x'[t, s, c];  h[t, :] = u / sqrt(mean(u^2) + eps) * (weight_offset + w_next)    (w_next NULL: no read)
 *   lane_sum[t, c] = sum_s x'[t, s, c]                                                                    (NULL: not written)
 * y, expert_out, h_in, h in `dtype`; x float32 [T, lanes, width] in place.  h_in and h may be the same buffer.
 * The experts' rows are added in the order k = 0 .. top - 1.
 */
typedef struct atoma_lanes_update_args {
    const void *y;                /* [T, width] or NULL */
    const float *y_bias;          /* [width] or NULL */
    const void *expert_out;       /* rows of the routed experts' results, or NULL */
    const int32_t *pair_row;      /* [T top] */
    const int32_t *top_expert;    /* [T top] */
    const float *top_weight;      /* [T top] */
    const void *h_in;             /* [T, width]: what identity experts hand through */
    int64_t top, experts;
    float *x;                     /* [T, lanes, width] */
    const float *w_mix, *w_out;   /* [lanes, lanes] indexed [from, to]; [lanes] */
    const float *w_in_next;       /* [lanes] or NULL (plain sum) */
    const float *w_next;          /* [width] or NULL */
    void *h;                      /* [T, width] */
    float *lane_sum;              /* [T, width] or NULL */
    int64_t T, lanes, width;
    float eps, weight_offset;
    uint32_t dtype;
} atoma_lanes_update_args;
void atoma_lanes_update_norm(const atoma_lanes_update_args *args, atoma_stream_t stream);

/* After a fused projection proj[t, :] (row stride ld) that holds the queries at column q_off (H heads of dim), the keys at
 * k_off (G heads of dim) and the values at v_off (G heads of vdim; v_off = k_off: the values ARE the key projections):
 *   q_out[t, h, :] = proj_q / sqrt(mean over the head's dim + eps) * (weight_offset + q_weight)     (one weight [dim] for all heads)
 *   k_cache[slot_mapping[t], g, :] = the same with k_weight;   v_cache[slot, g, :] = the values as projected (no norm)
 * caches [num_blocks * block_size, G, dim] / [.., G, vdim] in `dtype`; slot < 0 is skipped. */
void atoma_qk_headnorm_cache(const void *proj, int64_t ld, int64_t q_off, int64_t k_off, int64_t v_off, const float *q_weight,
                             const float *k_weight, float weight_offset, const int64_t *slot_mapping, void *q_out, void *k_cache,
                             void *v_cache, int64_t T, int64_t H, int64_t G, int64_t dim, int64_t vdim, float eps, uint32_t dtype,
                             atoma_stream_t stream);

/*
 * Softmax attention over a paged cache for a mixed batch, grouped key/value heads (head h reads kv head h / (H / G)).
 * Query token t of sequence b at position p sees key j <= p if p - j < window (window <= 0: no limit) or j < keep_first.
 *   s_h(j) = (q_h . k_j) * scale + (dist_bias ? dist_bias[min(p - j, dist_rows - 1), h] : 0)
 *   out[t, h, :] = softmax_j(s_h) v_j * (gate ? sigmoid(gate[t, h vdim ..]) : 1)
 * Scores, weights, maxima and sums are float32.  gate (row stride ld_gate) and out in `dtype`.
 */
typedef struct atoma_softmax_attn_args {
    const void *q;                /* [T, H dim] */
    const void *k_cache, *v_cache;
    void *out;                    /* [T, H vdim] */
    const void *gate;             /* pre-activation of the output gate, [T, >= H vdim], or NULL */
    int64_t ld_gate;
    const float *dist_bias;       /* [dist_rows, H] or NULL */
    int64_t dist_rows;
    const int64_t *positions;     /* [T] */
    const int32_t *token_seq;     /* [T] */
    const int32_t *query_start;   /* [B + 1] */
    const int32_t *block_tables;  /* [B, max_blocks] */
    int64_t T, B, max_blocks, H, G, dim, vdim, block_size, window, keep_first;
    float scale;
    uint32_t dtype;
    int32_t max_query_len, max_seq_len;
    int32_t skip_min_q;           /* > 0: sequences with at least this many query tokens in the step are left alone */
    /* long prompt portions (all zero = none): sequences with at least long_min_q (>= 32) tokens in the step, how many there are,
     * the sum of their tokens and of their contexts.  bfloat16 heads of 64 or 128 with dim = vdim run them on the tensor-memory
     * prefill kernel: the keys and values their queries can see through the window are gathered from the pages, the distance
     * term is added inside that kernel's softmax, the kept first tokens behind the window are a second short pass merged through
     * the log-sum-exp, and the gate is applied in the merge.  Without a table, kept tokens and a gate, dim and vdim may differ (vdim 64
     * or 128, dim a multiple of 8 up to vdim + 64). */
    int32_t long_min_q, long_seqs;
    int64_t long_tokens, long_ctx_sum;
    int64_t ld_out;               /* row stride of out (0: H vdim) */
    int64_t v_share;              /* neighbouring key heads that share one value head (0: 1): the value cache has G / v_share heads per row */
} atoma_softmax_attn_args;
void atoma_softmax_attention_paged(const atoma_softmax_attn_args *args, atoma_stream_t stream);

/* Two softmax maps per head into one result.  maps [T, 2 H vdim] (`dtype`) holds the heads' outputs by groups of rep = H / G query heads:
 * group g's rep outputs under the first map, then its rep outputs under the second.  Per token and head h = g rep + r, in float32:
 *   o = a1 - lambda a2;   out[t, h vdim ..] = o / sqrt(mean(o^2) + eps) * gain
 * out [T, H vdim] in `dtype`. */
void atoma_differential_combine(const void *maps, void *out, int64_t T, int64_t H, int64_t G, int64_t vdim, float lambda, float gain,
                                float eps, uint32_t dtype, atoma_stream_t stream);

/* Router with a restricted choice, float32.  z = w_router h over `outputs` router rows (experts, then identity experts);
 * s = softmax(z) (score_fn 1) or sigmoid(z) (0); choice score c = s + correction (NULL: none).  The outputs form `groups`
 * equal groups of neighbours (groups <= 1: no restriction); a group's score is the sum of its `group_top` largest c (1 or 2; a
 * group of one output has only that one); only outputs of the `keep` best groups can be chosen (ties: the lower group).  The `top` largest c among them (ties: the lower index) ->
 * top_expert [T, top] (an index >= the caller's expert count is an identity expert; -1 where fewer than `top` could be
 * chosen) and top_weight = their s divided by (their sum + 1e-20) (renormalize 1) or as they are (0). */
void atoma_moe_route_grouped(const void *h, const float *w_router, const float *correction, int32_t *top_expert, float *top_weight,
                             int64_t T, int64_t width, int64_t outputs, int64_t top, int64_t groups, int64_t keep, int32_t group_top,
                             int32_t score_fn, int32_t renormalize, uint32_t dtype, atoma_stream_t stream);

/* act_out[T, ff] = clamped gated activation (atoma_glu_clamped_bias) of the projection x [T, K] w_gate_up [2 ff, K]^T (gate rows,
 * then up rows).  Decode-sized bfloat16 steps (T <= 128, K % 64 == 0) run ONE kernel, the activation in the tcgen05 product's
 * epilogue; everything else atoma_linear into proj [T, 2 ff] and atoma_glu_clamped_bias. */
void atoma_linear_glu_clamped(const void *x, const void *w_gate_up, const float *bias, void *proj, void *act_out, int64_t T, int64_t ff,
                              int64_t K, float limit, float alpha, float up_shift, uint32_t dtype, atoma_stream_t stream);

/* atoma_glu_clamped with biases added first: g = gu[t, j] + bias[j], u = gu[t, ff + j] + bias[ff + j] (bias float32 [2 ff]). */
void atoma_glu_clamped_bias(const void *gu, int64_t ld, const float *bias, void *out, int64_t T, int64_t ff, float limit, float alpha,
                            float up_shift, uint32_t dtype, atoma_stream_t stream);

/* ------------------------------------------------------------------------------------------ */
/* Parallel blocks: tap filters with carried inputs, matrix-state recurrences, rotary operators */
/* ------------------------------------------------------------------------------------------ */

/*
 * Residual update of a parallel block fused with what precedes the next layer and with that layer's input norm.
 * Per token t and channel c, all in float32:
 *   a = y_a ? (norm_a ? y_a[t, :] / sqrt(mean(y_a[t, :]^2) + eps) * norm_a : y_a[t, :]) : 0        (b likewise)
 *   x[t, c] += mix_scale * (a[c] + b[c]) + (y_ff ? y_ff[t, c] : 0);     trace[t, c] = x[t, c]          (trace NULL: not written)
 *   x[t, c] += (add_rows ? add_rows[t, c] : 0) + (add_vec ? add_vec[c] : 0)
 *   h[t, :]  = x[t, :] / sqrt(mean(x[t, :]^2) + eps) * (weight_offset + w_next)                       (w_next NULL: no norm)
 * y_a, y_b, y_ff, h in `dtype` [T, width]; x, trace, add_rows float32 [T, width].  With no addends it is the first
 * layer's input norm.
 */
typedef struct atoma_parallel_residual_args {
    const void *y_a, *y_b, *y_ff;
    const float *norm_a, *norm_b; /* [width] or NULL */
    float mix_scale;
    float *x;
    float *trace;
    const float *add_rows, *add_vec;
    const float *w_next;
    void *h;
    int64_t T, width;
    float eps, weight_offset;
    uint32_t dtype;
} atoma_parallel_residual_args;
void atoma_parallel_residual_norm(const atoma_parallel_residual_args *args, atoma_stream_t stream);

/*
 * Causal tap filter over time per channel, on a mixed batch, with the inputs that precede a portion carried as state.
 * in [T, channels] (row stride ld_in, `dtype`); w1, w2 [channels, taps] float32, the LAST column weighs the current token
 * (w2 / out2 may be NULL: one filter).  For token t of sequence b at position p:
 *   f_k(t, c) = sum_{j < taps} w_k[c, j] * in(position p - (taps - 1) + j, c)       zero before the sequence's start
 *   out_k[t, c] = act(residual ? in[t, c] + f_k : f_k)        act: 0 = none, 1 = silu        (`dtype`, row stride ld_out)
 * in_bias [channels] (NULL: none) is part of the input: in(.) above is the stored value plus in_bias for every token of the
 * sequence (zero before its start, without the bias), and the history keeps the sum.  bias1 [channels] (NULL: none) is added to f_1.
 * history [slots, history_stride] float32 holds, at the slot of the sequence, its last taps - 1 inputs as
 * [taps - 1, channels]; it is read for positions before the portion (never when they lie before the sequence's start)
 * and rewritten with the portion's last inputs.  taps <= 16.
 */
typedef struct atoma_tap_filter_args {
    const void *in;
    int64_t ld_in;
    const float *w1, *w2;
    void *out1, *out2;
    int64_t ld_out;
    float *history;
    int64_t history_stride;
    const int32_t *state_slots;   /* [B] */
    const int32_t *token_seq;     /* [T] */
    const int32_t *query_start;   /* [B + 1] */
    const int32_t *context_lens;  /* [B] */
    int64_t T, B, channels, taps;
    int32_t residual, act;
    uint32_t dtype;
    const float *in_bias, *bias1; /* [channels] or NULL */
} atoma_tap_filter_args;
void atoma_tap_filter(const atoma_tap_filter_args *args, atoma_stream_t stream);

/*
 * Matrix-state recurrences on a mixed batch.  Every head keeps S [dim, vdim] float32 at the sequence's state slot
 * (state [slots, state_stride], head h at h dim vdim); it starts from zero when context_lens[b] == 0 and is stored back.
 * Tokens of a sequence are visited in order, so the result does not depend on how the sequence was cut into steps.
 *   kind 0, gated linear attention (q, k [T, H dim], v [T, H vdim]; decay pre-activation z [T, H dim] + z_bias):
 *     alpha = exp(log(sigmoid(z)) / tau);  S <- diag(alpha) S + k v^T;  o = S^T (q * q_scale)
 *   kind 1, gated delta rule (q, k [T, G dim] shared by H / G heads, v [T, H vdim]; per head b_pre, a_pre [T, H]):
 *     q, k <- x / sqrt(sum(x^2) + unit_eps) (q also times q_scale);  beta = sigmoid(b_pre);
 *     g = exp(-exp(a_log[h]) * softplus(a_pre + dt_bias[h]));
 *     S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
 *   kind 2, state-space recurrence (q, k [T, G dim] shared by H / G heads, v [T, H vdim]; per head a_pre [T, H]):
 *     d = softplus(a_pre + dt_bias[h]);  S <- exp(-exp(a_log[h]) d) S + d k v^T;  o = S^T q * q_scale + skip[h] v
 * q, k, v, z, b_pre, a_pre are columns of `dtype` matrices with their own row strides; out float32 [T, H vdim].
 */
typedef struct atoma_state_scan_args {
    int32_t kind;
    const void *q, *k, *v, *z, *b_pre, *a_pre;
    int64_t ld_q, ld_k, ld_v, ld_z, ld_b, ld_a;
    const float *z_bias;          /* [H dim] (kind 0) */
    const float *a_log, *dt_bias; /* [H] (kinds 1, 2) */
    float tau, q_scale, unit_eps;
    float *state;
    int64_t state_stride;
    const int32_t *state_slots, *query_start, *context_lens;
    float *out;
    int64_t T, B, H, G, dim, vdim;
    uint32_t dtype;
    const float *skip;            /* [H] or NULL (kind 2) */
} atoma_state_scan_args;
void atoma_state_scan(const atoma_state_scan_args *args, atoma_stream_t stream);

/* out[t, h vdim + j] = o[t, h, j] / sqrt(mean_j(o[t, h, :]^2) + eps) * weight[j] * silu(gate[t, h vdim + j]);
 * o float32 [T, H vdim], gate (row stride ld_gate) and out [T, H vdim] in `dtype`; gate NULL: no gate. */
void atoma_headnorm_gate(const float *o, const float *weight, const void *gate, int64_t ld_gate, void *out, int64_t T, int64_t H,
                         int64_t vdim, float eps, uint32_t dtype, atoma_stream_t stream);

/* A recurrence's read-out through its gate, then normed: u = o[t, :] * silu(gate[t, :]);
 *   out[t, c] = u[c] / sqrt(mean over c's part of u^2 + eps) * weight[c]        (`parts` equal consecutive parts of the n columns)
 * o float32 [T, n], gate (row stride ld_gate) and out (row stride ld_out) in `dtype`.  The zero_before columns in front of out's and the
 * zero_after columns behind them are set to zero (padding between the parts of a wider row). */
void atoma_gate_groupnorm(const float *o, const void *gate, int64_t ld_gate, const float *weight, void *out, int64_t ld_out, int64_t T,
                          int64_t n, int64_t parts, int64_t zero_before, int64_t zero_after, float eps, uint32_t dtype, atoma_stream_t stream);

/*
 * After a fused projection proj[t, :] (row stride ld): queries at q_off (H heads of dim), keys at k_off (G of dim), values
 * at v_off (G of vdim).  Per head: RMS norm over dim with q_weight / k_weight ([dim], NULL: none), then the first
 * 2 rot_pairs entries are turned by position * qk_freq[i] (float32 angle) in pairs (2i, 2i + 1) (interleaved = 1) or
 * (i, i + rot_pairs) (0); the values' first 2 v_pairs entries likewise by v_freq (v_freq NULL: stored as projected).
 * bias (float32, indexed by the columns of proj; NULL: none) is added to the projections first; unit_norm 1 divides every query
 * and key head by its root mean square also without a weight; q_head_scale [H] (NULL: none) multiplies a normed query head.
 * The q / k angles are formed to twice float32's precision: qk_freq_lo is what float32 drops of the frequencies (NULL: nothing);
 * cos and sin are scaled by qk_amplitude (0: 1).  v_heads: value heads when there are fewer than key heads (0: G).
 * slot_mapping NULL: queries only.
 * q -> q_out [T, H dim]; k, v -> cache rows slot_mapping[t] (slot < 0 is skipped).
 */
typedef struct atoma_qkv_rope_args {
    const void *proj;
    int64_t ld, q_off, k_off, v_off;
    const float *q_weight, *k_weight;
    const float *qk_freq, *v_freq;
    int64_t rot_pairs, v_pairs;
    int32_t interleaved;
    const int64_t *positions, *slot_mapping;
    void *q_out, *k_cache, *v_cache;
    int64_t T, H, G, dim, vdim;
    float eps;
    uint32_t dtype;
    const float *bias, *q_head_scale;
    int32_t unit_norm;
    const float *qk_freq_lo;
    float qk_amplitude;
    int64_t v_heads;
} atoma_qkv_rope_args;
void atoma_qkv_headnorm_rope_cache(const atoma_qkv_rope_args *args, atoma_stream_t stream);

/* In place on x [T, H, n] (`dtype`): the first 2 pairs entries of every head turned by sign * position * (freq[i] + freq_lo[i]) (freq_lo
 * NULL: none) and scaled by `amplitude`. */
void atoma_rotate_heads(void *x, const int64_t *positions, const float *freq, const float *freq_lo, float amplitude, int64_t T, int64_t H,
                        int64_t n, int64_t pairs, int32_t interleaved, float sign, uint32_t dtype, atoma_stream_t stream);

/*
 * Latent attention with a rotated key part.  proj[t, :] (row stride ld) = [c_q (q_rank) | c (kv_rank) | k_rot (rot_dim)]:
 *   cq_out[t, :] = rms(c_q) * q_weight;   cache[slot_mapping[t], :] = [rms(c) * kv_weight | rotate(k_rot, position)]
 * rotation in pairs (i, i + pairs) (interleaved 0) or (2i, 2i + 1) by position * (freq[i] + freq_lo[i]) (freq_lo: what float32 drops
 * of the frequency, NULL: none; the product is formed to twice float32's precision), cos and sin times `amplitude`; cache rows of
 * kv_rank + rot_dim in `dtype`.
 */
void atoma_latent_norm_rope_cache(const void *proj, int64_t ld, const float *q_weight, const float *kv_weight, const float *freq,
                                  const float *freq_lo, float amplitude, int64_t pairs, int32_t interleaved, const int64_t *positions, const int64_t *slot_mapping,
                                  void *cq_out, void *cache, int64_t T, int64_t q_rank, int64_t kv_rank, int64_t rot_dim, float eps,
                                  uint32_t dtype, atoma_stream_t stream);

/* Queries q [T, H, dim + rot_dim] (`dtype`) into the space of the cached rows, q_lat float32 [T, H, kv_rank + rot_dim]:
 *   q_lat[t, h, :kv_rank] = w_uk_h^T q[t, h, :dim]  (w_uk [H dim, kv_rank]);   q_lat[t, h, kv_rank:] = rotate(q[t, h, dim:], position) */
void atoma_latent_query_absorb_rope(const void *q, const void *w_uk, const float *freq, const float *freq_lo, float amplitude, int64_t pairs,
                                    int32_t interleaved, const int64_t *positions, float *q_lat, int64_t T, int64_t H, int64_t dim, int64_t rot_dim,
                                    int64_t kv_rank, uint32_t dtype, atoma_stream_t stream);

/* Values of every head from its weighted sum of cached rows: out[t, h vdim + j] = sum_{r < kv_rank} o_lat[t, h, r] w_uv[h vdim + j, r];
 * o_lat float32 [T, H, row] with row >= kv_rank (what lies behind kv_rank is not read).  gate (row stride ld_gate, `dtype`, NULL:
 * none): the result times sigmoid(gate[t, h vdim + j]). */
void atoma_latent_expand_values(const float *o_lat, const void *w_uv, const void *gate, int64_t ld_gate, void *out, int64_t T, int64_t H,
                                int64_t vdim, int64_t kv_rank, int64_t row, uint32_t dtype, atoma_stream_t stream);

/* ------------------------------------------------------------------------------------------ */
/* Post-norm blocks with a depth average; real-gated linear recurrent unit                      */
/* ------------------------------------------------------------------------------------------ */

/* Embedding rows with a second table looked up by the pair (token before, token), for a mixed batch:
 *   x[t, :] = table[tokens[t], :] + pair_table[row, :],  row = (before * mul_prev + tokens[t] * mul_cur) mod buckets   (64-bit integers)
 * and row = buckets for a sequence's first token.  `before` is tokens[t - 1] inside a sequence's portion and prev_tokens[b] (negative: the
 * portion starts the sequence) at its first token.  pair_table [buckets + 1, width] (NULL: x is the plain row).  x float32;
 * h [T, width] (NULL: not written) = x in `dtype`. */
void atoma_embed_pairs(const uint32_t *tokens, const int32_t *token_seq, const int32_t *query_start, const int32_t *prev_tokens, const void *table,
                       const void *pair_table, int64_t buckets, int64_t mul_prev, int64_t mul_cur, float *x, void *h, int64_t T, int64_t width,
                       int64_t vocab, uint32_t dtype, atoma_stream_t stream);

/*
 * Residual update of a post-norm block, fused with the sum of the token's expert rows and the average over depth.  Per token t:
 *   v = alpha * x[t, :] + (y ? y[t, :] : 0) + sum_{k < top} (top_expert[t, k] >= 0: expert_out[pair_row[t top + k], :])
 *   n = v / sqrt(mean(v^2) + eps) * (weight_offset + w_norm)
 *   x[t, :] = n                                                              (depth_n = 0)
 *   depth[depth_n - 1][t, :] = n;  x[t, :] = sum_{j < depth_n} depth_w[j] depth[j][t, :]   (depth_n > 0; depth_w NULL: x = n)
 *   h[t, :] = x[t, :] in `dtype` (NULL: not written);   trace[t, :] = x[t, :] (NULL: not written)
 * norm_branch = 1 norms the sublayer's result instead of the sum:
 *   v = y_scale * y[t, :] + y_bias + expert rows;   n = alpha * x[t, :] + branch_scale * v / sqrt(mean(v^2) + eps) * (weight_offset + w_norm)
 * (y_bias NULL: none; y_scale and branch_scale are used in this form only).
 * x float32 [T, width] in place; depth float32 [.., T, width] (row j of the average at j T width), rows 0 .. depth_n - 2 written by
 * earlier calls.  y, expert_out, h in `dtype`.  Experts' rows are added in the order of k, depth rows in the order of j.
 */
typedef struct atoma_postnorm_args {
    const void *y;
    const void *expert_out;
    const int32_t *pair_row;      /* [T top] */
    const int32_t *top_expert;    /* [T top] (NULL with expert_out: every pair has a row) */
    int64_t top;
    float *x;
    const float *w_norm;          /* [width] */
    float *depth;
    const float *depth_w;         /* [depth_n] or NULL */
    int64_t depth_n;
    void *h;
    float *trace;
    int64_t T, width;
    float alpha, eps, weight_offset;
    uint32_t dtype;
    int32_t norm_branch;
    const float *y_bias;          /* [width] or NULL */
    float y_scale, branch_scale;
} atoma_postnorm_args;
void atoma_postnorm_residual(const atoma_postnorm_args *args, atoma_stream_t stream);

/*
 * Gates of a real-gated linear recurrent unit with block-diagonal gate matrices.  u [T, channels] (`dtype`, row stride ld_u) in
 * `blocks` equal parts of n = channels / blocks; w [blocks, 2 n, n] `dtype` (a part's first n rows make the recurrence gate r, the next
 * n the input gate i, stored [out, in]); bias_r, bias_i, rate [channels] float32.  Everything behind the products is float32:
 *   r = sigmoid(w_r u + bias_r);  i = sigmoid(w_i u + bias_i);  log a = rate * r  (rate <= 0)
 *   decay[t, c] = exp(log a);     input[t, c] = sqrt(1 - a^2) * i * u[t, c]        (1 - a^2 without cancellation)
 * decay and input float32 [T, channels].
 */
typedef struct atoma_lru_gates_args {
    const void *u;
    int64_t ld_u;
    const void *w;
    const float *bias_r, *bias_i, *rate;
    float *decay, *input;
    int64_t T, channels, blocks;
    uint32_t dtype;
} atoma_lru_gates_args;
void atoma_lru_gates(const atoma_lru_gates_args *args, atoma_stream_t stream);

/*
 * Linear recurrence with one float32 state per channel on a mixed batch: per sequence, in token order,
 *   S <- decay[t, c] S + input[t, c];   out[t, c] = S * act(gate[t, c] + gate_bias[c])        act: 0 silu, 1 relu, 2 gelu (tanh form)
 * S starts from state[state_slots[b], c] — from zero when context_lens[b] == 0 — and is stored back.  decay, input float32
 * [T, channels]; gate (row stride ld_gate) and out [T, channels] in `dtype`; state rows state_stride floats apart.
 */
typedef struct atoma_linear_scan_args {
    const float *decay, *input;
    const void *gate;
    int64_t ld_gate;
    const float *gate_bias;       /* [channels] or NULL */
    float *state;
    int64_t state_stride;
    const int32_t *state_slots, *query_start, *context_lens;
    void *out;
    int64_t T, B, channels;
    int32_t act, max_query_len;
    uint32_t dtype;
} atoma_linear_scan_args;
void atoma_linear_scan(const atoma_linear_scan_args *args, atoma_stream_t stream);

/* ------------------------------------------------------------------------------------------ */
/* Step executor                                                                                */
/* ------------------------------------------------------------------------------------------ */
enum { ATOMA_MIXER_SIGMOID_ATTENTION = 0, ATOMA_MIXER_MINGRU = 1, ATOMA_MIXER_LATENT_ATTENTION = 2, ATOMA_MIXER_SOFTMAX_ATTENTION = 3,
       ATOMA_MIXER_GLA = 4, ATOMA_MIXER_PAIR = 5, ATOMA_MIXER_LRU = 6, ATOMA_MIXER_ATTENTION_SSM = 7 };
enum { ATOMA_BLOCK_SANDWICH = 0, ATOMA_BLOCK_PRENORM = 1, ATOMA_BLOCK_LANES = 2, ATOMA_BLOCK_PARALLEL = 3,
       ATOMA_BLOCK_POSTNORM = 4 };
enum { ATOMA_SCORE_SIGMOID = 0, ATOMA_SCORE_SOFTMAX = 1 };
enum { ATOMA_FF_DENSE = 0, ATOMA_FF_MOE = 1 };
enum { ATOMA_ACT_SILU = 0, ATOMA_ACT_RELU = 1, ATOMA_ACT_GELU_TANH = 2 };

typedef struct atoma_hybrid_layer {
    int32_t mixer, has_mlp;
    const float *norm1, *norm1b, *norm2, *norm2b; /* [width] offsets from one */
    /* attention */
    int64_t heads, kv_heads, dim, vdim, temp_every;
    float scale, softcap, temp_coef;
    const void *w_qkv;      /* [H dim + G dim + G vdim, width] */
    const float *b_qkv;
    const float *q_norm, *k_norm, *talk, *head_bias, *slopes;
    void *k_cache, *v_cache;
    /* minGRU */
    int64_t state_width;
    const void *w_zxg;      /* [3 S, width] */
    const float *b_zxg;
    float *state;           /* [slots, S] */
    /* both mixers */
    const void *w_o;        /* [width, H vdim] or [width, S] */
    /* feed-forward */
    int64_t ff;
    int32_t act;
    const void *w_gate_up;  /* [2 ff, width] */
    const void *w_down;     /* [width, ff] */
    /* ---- pre-norm blocks (model.block_style = ATOMA_BLOCK_PRENORM) ---- */
    /* latent attention (uses heads, dim, vdim, scale above) */
    int64_t q_rank, kv_rank, window;   /* window <= 0: every earlier token is visible */
    const void *w_down_in;  /* [q_rank + kv_rank (+ width with a gated residual), width]: query latent, key/value latent, residual gate */
    const float *dq_norm, *dkv_norm, *sink;
    const void *w_uq, *w_uk, *w_uv;    /* [H dim, q_rank], [H dim, kv_rank], [H vdim, kv_rank] */
    void *latent_cache;     /* [num_blocks * block_size, kv_rank] */
    /* gated residuals: bias of the gate, NULL = the sublayer's result is added as it is */
    const float *gate1_bias, *gate2_bias;
    /* mixture of experts (ff_kind = ATOMA_FF_MOE): ff above = the shared expert's size (0: none) */
    int32_t ff_kind, renormalize;
    int64_t experts, top, expert_ff;
    float expert_limit, shared_limit, act_alpha, act_up_shift;
    const float *w_router;  /* [experts, width] float32 */
    const float *w_shared_gate; /* [width] float32 or NULL */
    const void *w_expert_gate_up, *w_expert_down;
    const void *w_ff_in;    /* [2 ff (+ width with a gated residual), width]: shared gate rows, up rows, residual gate */
    /* token side input after the feed-forward (side_gate NULL: none) */
    int64_t side_part;
    const void *side_gate, *side_proj; /* [side_dim, width], [width, side_dim] */
    const float *side_norm;
    /* ---- blocks on residual lanes (model.block_style = ATOMA_BLOCK_LANES) ---- */
    /* softmax attention (uses heads, kv_heads, dim, vdim, scale, window, q_norm / k_norm [dim], k_cache, v_cache, w_o above;
     * w_qkv = the stacked projections [H dim queries | G dim keys | G vdim values unless values_are_keys | H vdim gate if out_gate]) */
    int64_t keep_first, dist_rows;
    const float *dist_bias; /* [dist_rows, heads] or NULL */
    int32_t values_are_keys, out_gate;
    /* lane weights of the mixer (1) and the feed-forward (2): read [lanes], write [lanes], mix [lanes, lanes] as [from, to] */
    const float *lanes_in1, *lanes_out1, *lanes_mix1, *lanes_in2, *lanes_out2, *lanes_mix2;
    /* feed-forward biases (dense kind; NULL: none) and what the router adds */
    const float *b_gate_up, *b_down; /* [2 ff], [width] */
    const float *router_correction;  /* [experts + identity_experts] or NULL */
    int64_t route_groups, route_keep, identity_experts;
    int32_t score_fn, scale_input;   /* ATOMA_SCORE_*; 1: the router's weight scales the expert's input, 0: its output */
    /* ---- parallel blocks (model.block_style = ATOMA_BLOCK_PARALLEL): x += mixer(f1(h)) + ff(f2(h)), h = norm1(x) ---- */
    /* what precedes the layer: the embedding rows and / or a vector added to the stream (the start of a pass over a looped span) */
    int32_t add_embedding;
    const float *add_vec;            /* [width] or NULL */
    /* tap filters of the two sublayers' inputs (taps <= 0: none); the layer's state row = [input history | mixer state] */
    int64_t taps;
    const float *tap_w1, *tap_w2;    /* [width, taps] */
    float *layer_state;              /* [slots, layer_state_stride] float32 */
    int64_t layer_state_stride;
    /* stacked projection of the mixer: w_qkv [proj_cols, width]; columns of its parts (-1: absent) */
    int64_t proj_cols;
    /* gated linear attention (heads, dim, vdim): q, k, v, g columns, the decay's low-rank projection (w_a1 [a_rank, width] as
     * columns a_off .. of the stacked projection, w_a2 [heads dim, a_rank], bias), head norm weight, tau */
    int64_t q_off, k_off, v_off, g_off, a_off, a_rank;
    const void *w_a2;
    const float *a2_bias, *head_norm;
    float tau;
    /* pair of mixers: left = sigmoid attention with rotary positions (heads, kv_heads, dim, vdim, scale, q_norm, k_norm, head_bias,
     * k_cache, v_cache, w_o above), right = gated delta rule */
    const float *qk_freq, *v_freq;   /* [rot_pairs], [v_pairs] float32 */
    int64_t rot_pairs, v_pairs;
    int32_t rot_interleaved;
    int64_t r_heads, r_kv_heads, r_dim, r_vdim, r_taps;
    int64_t rq_off, rk_off, rv_off, rg_off, rb_off, ra_off;
    const float *r_tap_w;            /* [2 r_kv_heads r_dim + r_heads r_vdim, r_taps] */
    const float *r_a_log, *r_dt_bias, *r_head_norm;
    const void *r_w_o;               /* [width, r_heads r_vdim] */
    const float *out_norm_a, *out_norm_b; /* [width] */
    /* latent attention with a rotated key part (q_rank, kv_rank, dq_norm, dkv_norm, w_uq [heads (dim + rot_dim), q_rank], w_uk, w_uv,
     * latent_cache rows of kv_rank + rot_dim; qk_freq / rot_pairs / rot_interleaved above) */
    int64_t rot_dim;
    /* ---- post-norm blocks (model.block_style = ATOMA_BLOCK_POSTNORM): x <- norm(alpha x + sublayer(x)) ---- */
    /* norm1 / norm2 above follow the sums; b_qkv [proj_cols] = biases of the stacked projection; softmax attention: columns q_off, k_off,
     * v_off; latent attention: [c_q | c | k_rot] at column 0, the output gate's pre-activation at g_off (out_gate); mixture of experts:
     * w_ff_in = the shared expert's gate and up rows */
    const float *depth_w;            /* weights of the embedding output and of every layer's result up to this one, or NULL */
    const float *q_head_scale;       /* [heads] or NULL */
    const float *qk_freq_lo;         /* [rot_pairs] or NULL */
    float rot_amplitude;
    int32_t route_group_top;         /* choice scores of a group that make its score (1 or 2; 0 = 1) */
    /* real-gated linear recurrent unit: width lru_width, gate branch at column q_off, recurrent branch at k_off, filter r_tap_w
     * [lru_width, r_taps] with bias; the layer's state row = [filter history (r_taps - 1) lru_width | state lru_width] */
    int64_t lru_width, lru_blocks;
    const void *lru_w;               /* [lru_blocks, 2 n, n] */
    const float *lru_bias_r, *lru_bias_i, *lru_rate, *r_tap_bias; /* [lru_width] */
    const void *w_uk_rot;            /* [heads (dim + rot_dim), kv_rank + rot_dim]: a cached row -> the heads' whole keys, or NULL */
    /* softmax attention, further: bias of the output projection [width] or NULL (joined in the residual update); v_share key heads per
     * value head (0: 1); v_off < 0: no key and value projections, the caches are an earlier layer's; diff_gain != 0: differential, `heads`
     * counts both maps' heads (laid out by groups, first map then second), w_o reads heads / 2 of them */
    const float *b_o;
    int64_t v_share;
    float diff_lambda, diff_gain;
    /* sum of softmax attention and a state-space recurrence on the same input: attention as above; recurrence of r_heads heads of r_vdim,
     * r_kv_heads groups of r_dim states, filter [r_heads r_vdim + 2 r_kv_heads r_dim, r_taps] with r_tap_bias over the columns [x | B | C] at
     * rv_off, gate at rg_off, step sizes at ra_off, r_a_log, r_dt_bias, r_skip [r_heads], norm weight r_head_norm [r_heads r_vdim] in
     * r_norm_groups parts.  w_o [width, mix_cols] reads [attention | padding | recurrence at column r_mix_off | padding] in one product; the sum
     * is its result times mix_scale.  The layer's state row = [filter history | r_heads r_dim r_vdim] */
    const float *r_skip;
    int64_t r_norm_groups, mix_cols, r_mix_off;
    float mix_scale;
} atoma_hybrid_layer;

typedef struct atoma_hybrid_model {
    int64_t width, vocab, num_layers, block_size;
    float eps, logit_scale, norm_offset;
    uint32_t dtype;
    const void *embed;      /* [vocab, width] */
    const double *inv_freq; /* [ceil(width / 2)] */
    const float *final_norm;
    const void *head;       /* [vocab, width] */
    const atoma_hybrid_layer *layers; /* host array */
    /* ---- pre-norm designs ---- */
    int32_t block_style;    /* ATOMA_BLOCK_* */
    int32_t norm_groups;    /* 0 or 1: whole-row norms */
    const void *pos_table;  /* [max_positions, width] learned positions (then inv_freq may be NULL) */
    int64_t max_positions;
    float logit_softcap;    /* <= 0: none */
    const void *side_table; /* [vocab, side_table_width] */
    int64_t side_dim, side_table_width;
    /* ---- designs on residual lanes ---- */
    int32_t lanes;          /* copies of the residual stream (ATOMA_BLOCK_LANES: >= 1) */
    float embed_scale;      /* the embedding row times this; no position signal is added */
    /* ---- post-norm designs ---- */
    const float *embed_norm; /* [width]: norm of the embedding rows */
    float residual_alpha;   /* the stream's factor in every sum */
    /* embed_norm NULL: the embedding rows as they are; norm_branch 1: the sublayers' results are normed and added times branch_scale */
    float branch_scale;
    int32_t norm_branch;
    const void *pair_table; /* [pair_buckets + 1, width] second embedding table (atoma_embed_pairs) or NULL */
    int64_t pair_buckets, pair_mul_prev, pair_mul_cur;
} atoma_hybrid_model;

typedef struct atoma_hybrid_batch {
    int64_t num_tokens, num_seqs, num_selected, max_blocks;
    int32_t max_query_len, max_seq_len;
    const uint32_t *tokens;       /* [T] */
    const int64_t *positions;     /* [T] */
    const int64_t *slot_mapping;  /* [T] */
    const int32_t *token_seq;     /* [T] */
    const int32_t *query_start;   /* [B + 1] */
    const int32_t *context_lens;  /* [B] tokens already in the cache / state */
    const int32_t *block_tables;  /* [B, max_blocks] */
    const int32_t *state_slots;   /* [B] */
    const int32_t *selected;      /* [num_selected] token rows whose logits are wanted */
    void *scratch;
    int64_t scratch_bytes;
    float *logits;                /* out [num_selected, vocab] */
    uint32_t *next_tokens;        /* out [num_selected] greedy */
    float *residual_trace;        /* optional out [num_layers, T, width]: the residual stream (the sum of the lanes) after every layer */
    /* long prompt portions (pre-norm designs; all zero = none): sequences with at least long_min_q tokens in the step, how many
     * there are, the sum of their tokens and of their contexts (tokens already cached) */
    int32_t long_seqs, long_min_q;
    int64_t long_tokens, long_ctx_sum;
    const int32_t *prev_tokens;   /* [B] token before the portion, -1 at a sequence's start (models with a pair table; else may be NULL) */
} atoma_hybrid_batch;

int64_t atoma_hybrid_abi_sizeof(int which); /* 0 layer, 1 model, 2 batch, 3 attention args, 4 gated residual args, 5 latent attention args, 6 expert args, 7 expanded attention args, 8 lanes update args, 9 softmax attention args, 10 parallel residual args, 11 tap filter args, 12 state scan args, 13 rotary cache args, 14 post-norm args, 15 gate args, 16 linear scan args */
int64_t atoma_hybrid_scratch_bytes(const atoma_hybrid_model *model, int64_t num_tokens, int64_t num_selected);
void atoma_hybrid_step(const atoma_hybrid_model *model, const atoma_hybrid_batch *batch, atoma_stream_t stream);

/* Diagnostics: bit 0 = every projection through the plain float32-FMA kernel; bit 1 = the general attention kernel
 * for every batch (no tensor-core prefill / split decode kernels); bit 2 = the sequential minGRU scan; bit 3 = the routed
 * experts' tensor-memory (tcgen05) products for steps of any size (they normally serve steps of 1024 pairs and more);
 * bit 4 = the matrix-state scans with many rows per lane whatever the step's size (they normally take 8 rows per lane when a
 * step has few CTAs; both add in the same order). */
void atoma_debug_hybrid(int flags);

/* CTAs of the tensor-memory prefill attention kernel that gave up a wait since the library was loaded (0 unless something is broken;
 * -1: the device could not be asked).  Synchronises the device. */
int atoma_prefill_timeouts(void);

#ifdef __cplusplus
}
#endif
#endif /* ATOMA_HYBRID_H_ */
