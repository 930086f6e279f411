/*
 * peregrine_b200 -- C ABI of the layer mechanisms that the bf16 / f32 language models are put together from
 * (libperegrine_b200_lm.so).  Contexts, graphs, device memory and the greedy choice are those of peregrine_b200.h; the
 * library carries them too, so that a program which serves one of these models builds and loads this library only.
 *
 * Conventions (beyond those of peregrine_b200.h)
 *   - A step runs the rows (tokens) of one or more sequences, all rows of a sequence next to each other; pg_batch says
 *     which row is which position of which sequence, and in which slot that sequence keeps its cache or state.
 *   - A step starts with pg_embed_norm or pg_embed_prenorm (or with a copy), which wait for everything before them.  The
 *     kernels behind may read the batch's arrays, and what earlier steps left in caches and states, while the kernel in
 *     front of them still runs.
 *   - Activations that enter a product are [rows, K] in the step's type (PG_F32 or PG_BF16) with K a multiple of 64:
 *     columns behind a matrix's true width are zero in the weights and zero in the activations.
 *   - The residual stream, norms, routers, scores, decays and recurrent states are f32 in both types.
 *   - PG_F32 is true f32 throughout (bf16 weights are widened exactly; FFMA, no reduced-precision matrix mode).
 */
#ifndef PEREGRINE_B200_LM_H
#define PEREGRINE_B200_LM_H

#include "peregrine_b200.h"

#ifdef __cplusplus
extern "C" {
#endif

typedef struct pg_linear pg_linear; /* bf16 weights [experts][N][K] on the device */
typedef struct pg_route pg_route;   /* which token goes to which expert, rebuilt in every step */

typedef enum pg_dtype { PG_F32 = 0, PG_BF16 = 1 } pg_dtype;

/* What a product does with its output columns.  The two gated forms take weights whose rows alternate in blocks of
 * eight -- eight gate rows, eight up rows -- and write N / 2 columns. */
typedef enum pg_act {
    PG_ACT_NONE = 0,
    PG_ACT_GELU_TANH_GLU = 1,    /* gelu_tanh(g) * u */
    PG_ACT_CLAMPED_SWISH_GLU = 2 /* g' = min(g, limit), u' = clamp(u, -limit, limit): g' * sigmoid(1.702 g') * (u' + 1) */
} pg_act;

typedef struct pg_batch {
    int32_t rows, seqs, max_len;    /* tokens, sequences, longest sequence of this step */
    const int32_t *d_tokens;        /* [rows] */
    const int32_t *d_pos;           /* [rows] position in the sequence */
    const int32_t *d_row_seq;       /* [rows] index of the sequence (0 .. seqs - 1) */
    const int32_t *d_seq_row0;      /* [seqs + 1] first row of each sequence */
    const int32_t *d_seq_slot;      /* [seqs] cache / state slot */
} pg_batch;

/* ---- products: y = a W^T ---- */
PG_API int32_t pg_linear_wrap(pg_ctx *ctx, const void *d_w_bf16, int64_t n, int64_t k, int64_t experts, pg_linear **out);
PG_API int32_t pg_linear_free(pg_ctx *ctx, pg_linear *lin);
/* a [m, K]; y [m, ldy] of N (or N / 2) columns in y_dtype (gated forms: y_dtype == dtype) */
PG_API int32_t pg_linear_run(pg_ctx *ctx, pg_linear *lin, const void *d_a, int32_t dtype, int64_t m, int32_t act, float limit, void *d_y,
                             int32_t y_dtype, int64_t ldy);
/* The same with rows of a `lda` (>= K, a multiple of 8) elements apart */
PG_API int32_t pg_linear_run_ld(pg_ctx *ctx, pg_linear *lin, const void *d_a, int64_t lda, int32_t dtype, int64_t m, int32_t act, float limit, void *d_y,
                                int32_t y_dtype, int64_t ldy);
/* The same for the rows of a route, each with its expert's weights.  by_token: row r of the route reads row
 * (its token) of a, else row r; y has one row per row of the route. */
PG_API int32_t pg_linear_run_routed(pg_ctx *ctx, pg_linear *lin, pg_route *route, const void *d_a, int32_t dtype, int32_t by_token, int32_t act,
                                    float limit, void *d_y, int32_t y_dtype, int64_t ldy);

/* ---- mixture of experts: softmax scores, corrected choice, groups, identity experts ---- */
PG_API int32_t pg_route_create(pg_ctx *ctx, int64_t max_tokens, int64_t experts, int64_t identity, int64_t top, pg_route **out);
PG_API int32_t pg_route_free(pg_ctx *ctx, pg_route *route);
PG_API int64_t pg_route_max_rows(const pg_route *route); /* rows a routed output can have */
/* logits [m, ld] of experts + identity columns; correction [experts + identity] is added to the scores for the choice
 * only; only the best `keep` of `groups` groups of neighbours can be chosen (groups <= 1: no limit). */
PG_API int32_t pg_route_run(pg_ctx *ctx, pg_route *route, int32_t dtype, const float *d_logits, int64_t ld, int64_t m, const float *d_correction,
                            int32_t groups, int32_t keep);
/* copies of the chosen ids [m, top] and weights [m, top] (device -> host, blocking) */
PG_API int32_t pg_route_read(pg_ctx *ctx, const pg_route *route, int32_t *ids, float *weights);

/* ---- rows of the residual stream ---- */
/* x = rms_norm(table[token] + pos_table[pos]) * w; h = x in the step's type */
PG_API int32_t pg_embed_norm(pg_ctx *ctx, const pg_batch *batch, const void *d_table_bf16, const void *d_pos_table_bf16, int64_t width,
                             const float *d_w, float eps, float *d_x, void *d_h, int32_t dtype, int64_t ldh);
/* x += scale * (rms_norm(y) * w); h = x */
PG_API int32_t pg_norm_add(pg_ctx *ctx, const float *d_y, int64_t ldy, float *d_x, const float *d_w, const float *d_scale, int64_t rows, int64_t width,
                           float eps, void *d_h, int32_t dtype, int64_t ldh);
/* The forms of a model with norms in front of its sublayers too.  x = table[token]; h = rms_norm(x) * next */
PG_API int32_t pg_embed_prenorm(pg_ctx *ctx, const pg_batch *batch, const void *d_table_bf16, int64_t width, const float *d_next, float eps, float *d_x,
                                void *d_h, int32_t dtype, int64_t ldh);
/* x += rms_norm(y) * w; h = rms_norm(x) * next (x itself where next is null) */
PG_API int32_t pg_norm_add_prenorm(pg_ctx *ctx, const float *d_y, int64_t ldy, float *d_x, const float *d_w, const float *d_next, int64_t rows,
                                   int64_t width, float eps, void *d_h, int32_t dtype, int64_t ldh);
/* pg_norm_add with y = the weighted sum of a token's expert outputs (identity experts: x itself) */
PG_API int32_t pg_routed_norm_add(pg_ctx *ctx, const pg_route *route, const void *d_out, int64_t ldo, float *d_x, const float *d_w,
                                  const float *d_scale, int64_t rows, int64_t width, float eps, void *d_h, int32_t dtype, int64_t ldh);
/* h[i] = rms_norm(x[row i]) * w for the rows named by d_rows [m] */
PG_API int32_t pg_norm_rows(pg_ctx *ctx, const float *d_x, const int32_t *d_rows, int64_t m, int64_t width, const float *d_w, float eps, void *d_h,
                            int32_t dtype, int64_t ldh);

/* ---- gated delta rule with short convolutions ----
 * proj row: [q G*D | k G*D | v H*V | gate H*V | b H | a H] (f32).  ring [slot][taps][2 G D + H V]: the last inputs of
 * the convolutions, position p in entry p mod taps.  state [slot][H][D][vs], vs = V rounded up to 4. */
typedef struct pg_delta {
    int32_t heads, kv_heads, dim, vdim, taps;
    float eps, unit_eps;
    const float *d_conv;    /* [taps][2 G D + H V], last for the current token */
    const float *d_a_log;   /* [H] */
    const float *d_dt_bias; /* [H] */
    const float *d_norm;    /* [V] */
    float *d_work;          /* pg_delta_work_floats(...) */
} pg_delta;
PG_API int64_t pg_delta_work_floats(const pg_delta *p, int64_t max_rows);
PG_API int32_t pg_delta_run(pg_ctx *ctx, const pg_delta *p, const pg_batch *batch, const float *d_proj, int64_t ldp, float *d_ring, float *d_state,
                            void *d_out, int32_t dtype, int64_t ldo);

/* ---- attention; each of these is there or not: per-head query / key norms, a query temperature that grows with the
 * position, a sink, a distance bias, chunks ----
 * proj row: [q H*D | k G*D | v G*V] (f32).  Caches [slot][G][cap][dp] and [slot][G][cap][vp] in the step's type, dp and
 * vp = D and V rounded up to 16.  In a chunked layer (chunk > 0) position i sees the positions j <= i of its own chunk,
 * floor(j / chunk) = floor(i / chunk); cap is then a multiple of chunk, position p lies in row p mod cap, and a step's tokens
 * of one sequence must not touch more chunks than cap has. */
typedef struct pg_attention {
    int32_t heads, kv_heads, dim, vdim, cap, slots; /* slots: of the caches */
    float eps, scale;
    float temp_coef, temp_every; /* temp_every == 0: none; else q *= 1 + coef * ln(floor((p + 1) / every) + 1) */
    int32_t sink;                /* 1: one is added to the softmax denominator */
    int32_t chunk;               /* 0: a position sees all positions up to its own */
    int32_t positions;           /* most positions of a sequence (0: cap) */
    const float *d_q_norm;       /* [D], null: no norm */
    const float *d_k_norm;       /* [D], null: no norm */
    const float *d_slopes;       /* [H], null: none; else slope * (i - j) is taken off the scaled score */
    void *d_q;                   /* [max_rows][H][dp] in the step's type */
    float *d_part;               /* pg_attention_part_floats(...) */
    int32_t *d_tickets;          /* [max_seqs * G * 16], zero before the first call */
} pg_attention;
PG_API int64_t pg_attention_part_floats(pg_ctx *ctx, const pg_attention *p, int64_t max_seqs);
PG_API int32_t pg_attention_run(pg_ctx *ctx, const pg_attention *p, const pg_batch *batch, const float *d_proj, int64_t ldp, void *d_kcache,
                                void *d_vcache, void *d_out, int32_t dtype, int64_t ldo);

/* ---- latent attention ----
 * A position's cache row is [c | rotated key part]: C = kv_rank columns padded to a multiple of 64, and rot_dim columns padded
 * to a multiple of 16, in the step's type: [slot][cap][cp + rp].
 * proj row: [q H*(dim + rot_dim) | latent C, key part rot_dim | gate H*vdim] (f32); the second part is there if `own` is 1 --
 * else the layer reads a cache that another layer has written in the same step.  The heads' outputs are multiplied by the
 * sigmoid of the gate. */
typedef struct pg_latent {
    int32_t heads, dim, rot_dim, vdim, kv_rank, cap, slots, own;
    float eps, scale;
    const float *d_rot;  /* [cap][rot_dim / 2][2]: cosine and sine of the angle of every position and pair of dimensions */
    const float *d_norm; /* [C]; null without a latent of its own */
    const void *d_uk;    /* bf16 [H][cp][dim up to 32]: W_uk transposed per head, zero where padded */
    const void *d_uv;    /* bf16 [H * vdim + 7][cp], zero where padded */
    void *d_q;           /* [max_rows][H][max(cp + rp, dim up to 64 + rot_dim up to 64)] in the step's type */
    float *d_part;
    int64_t part_floats; /* of d_part: pg_latent_part_floats(...) */
} pg_latent;
PG_API int64_t pg_latent_part_floats(pg_ctx *ctx, const pg_latent *p, int32_t dtype, int64_t max_rows, int64_t max_seqs);
/* The sequences with fewer than long_from tokens in this step: short_rows tokens in all, at most short_len of one sequence. */
PG_API int32_t pg_latent_run(pg_ctx *ctx, const pg_latent *p, const pg_batch *batch, int64_t long_from, int64_t short_rows, int64_t short_len,
                             const float *d_proj, int64_t ldp, void *d_cache, void *d_out, int32_t dtype, int64_t ldo);
/* A longer portion of one sequence (bf16), in three calls: pg_latent_prompt_prep appends its positions; a product with
 * [W_uk, heads padded to a multiple of 16 rows | W_uv, the same] unfolds the cache rows of all positions into kv
 * [positions][ldkv]; pg_latent_prompt attends. */
PG_API int32_t pg_latent_prompt_supports(const pg_latent *p);
PG_API int32_t pg_latent_prompt_prep(pg_ctx *ctx, const pg_latent *p, const pg_batch *batch, int64_t row0, int64_t len, int64_t slot, const float *d_proj,
                                     int64_t ldp, void *d_cache);
PG_API int32_t pg_latent_prompt(pg_ctx *ctx, const pg_latent *p, const pg_batch *batch, int64_t seq, int64_t len, int64_t positions, int64_t slot,
                                const float *d_proj, int64_t ldp, const void *d_cache, const void *d_kv, int64_t ldkv, void *d_out, int64_t ldo);

/* ---- selective scan (one decay per channel and state) with a short convolution ----
 * proj row: [x inner | z inner] (f32).  ring [slot][taps][inner]: the last inputs of the convolution, position p in entry
 * p mod taps.  state [slot][inner][ss], ss = `state` rounded up to 4.  low row: [dt | B | C] (f32), the first part padded to a
 * multiple of 64 columns. */
typedef struct pg_scan {
    int32_t inner, state, dt_rank, taps;
    const float *d_conv;      /* [taps][inner], last for the current token */
    const float *d_conv_bias; /* [inner] */
    const float *d_a;         /* [inner][ss]: A * log2(e), zero where padded */
    const float *d_d;         /* [inner] */
    const float *d_dt_bias;   /* [inner] */
    const void *d_dt;         /* bf16 [inner][dt_rank up to 64]: W_dt, zero where padded */
} pg_scan;
/* x [rows, ldx] = silu(convolution) in the step's type.  Where every sequence has one token the ring takes it here, else in
 * pg_scan_run. */
PG_API int32_t pg_scan_conv(pg_ctx *ctx, const pg_scan *p, const pg_batch *batch, const float *d_proj, int64_t ldp, float *d_ring, void *d_x, int32_t dtype,
                            int64_t ldx);
/* One token per sequence: step sizes (W_dt inside), state update, read-out, gate silu(z). */
PG_API int32_t pg_scan_step(pg_ctx *ctx, const pg_scan *p, const pg_batch *batch, const float *d_proj, int64_t ldp, const void *d_x, int64_t ldx,
                            const float *d_low, int64_t ldl, float *d_state, void *d_out, int32_t dtype, int64_t ldo);
/* Portions of any length; dt [rows, ldt]: the product with W_dt, before bias and softplus; bc [rows, ldb]: [B | C]. */
PG_API int32_t pg_scan_run(pg_ctx *ctx, const pg_scan *p, const pg_batch *batch, const float *d_proj, int64_t ldp, float *d_ring, const void *d_x, int64_t ldx,
                           const float *d_dt, int64_t ldt, const float *d_bc, int64_t ldb, float *d_state, void *d_out, int32_t dtype, int64_t ldo);

#ifdef __cplusplus
}
#endif
#endif
