// What the two attention files share.
#pragma once

#include "pg_lm.cuh"

struct AttnShape {
    int H, G, rep, D, V, dp, vp, sink;   // dp, vp: row widths of the caches (D and V rounded up to 16)
    int cap;                             // rows of a slot's and head's part of the cache
    int limit;                           // positions of a sequence
    int chunk;                           // 0: a position sees all before it; else those of its chunk, and cap is a multiple of chunk
    float eps, scale, coef, every;
    const float *qn, *kn;                // null: no norm
    const float *slopes;                 // [H], null: no distance bias
};

#ifdef __CUDACC__
// A chunked layer keeps whole chunks only, position p in row p mod cap: the rows of a chunk lie next to each other.
__device__ __forceinline__ int attn_low(const AttnShape &s, int pos) { return s.chunk ? pos - pos % s.chunk : 0; }
__device__ __forceinline__ int attn_row(const AttnShape &s, int pos) { return s.chunk ? pos % s.cap : pos; }
#endif

// pg_attention.cu: out [rows][H V] f32; every head's query is a row of s.dp floats
int32_t pgk_attention_f32(pg_ctx *ctx, const AttnShape &s, const pg_batch *bt, const float *q, const float *kc, const float *vc, float *out, int64_t ldo);

// pg_attention_tc.cu
// Keys and values that a latent layer made from its latents for one sequence (csrc/pg_latent.cu): every head has its own, and
// a key has a second part that all heads share and that lies in the layer's cache.
struct AttnSplitKeys {
    const bf16 *q;          // [rows][H][qd]: the part for `k`, zero up to a multiple of 64, then the part for `shared`, the same
    int qd;
    const bf16 *k;          // [positions][H][kd], rows ldk elements apart
    int kd;
    const bf16 *v;          // [positions][H][vd], rows ldk elements apart
    int vd;
    int64_t ldk;
    const bf16 *shared;     // [positions][sd] of the sequence's slot, rows lds elements apart
    int sd;
    int64_t lds;
    const float *gate;      // [rows][H V], rows ldg elements apart: the output is multiplied by its sigmoid
    int64_t ldg;
    int seq, len, positions;   // the sequence, its tokens in this step and its positions with them
};
bool pgk_attention_split_supports(int kd, int sd, int V);
int32_t pgk_attention_split_tc(pg_ctx *ctx, const AttnShape &s, const pg_batch *bt, const AttnSplitKeys &k, bf16 *out, int64_t ldo);

bool pgk_attention_prompt_tc_supports(const AttnShape &s, const pg_batch *bt, int64_t slots, int64_t ldo, const void *out);
int32_t pgk_attention_prompt_tc(pg_ctx *ctx, const AttnShape &s, const pg_batch *bt, int64_t slots, const bf16 *q, const bf16 *kc, const bf16 *vc, bf16 *out,
                                int64_t ldo);
