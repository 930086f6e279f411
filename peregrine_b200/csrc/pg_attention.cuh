// What the two attention files share.
#pragma once

#include "pg_lm.cuh"

struct AttnShape {
    int H, G, rep, D, V, dp, vp, cap, sink;   // dp, vp: row widths of the caches (D and V rounded up to 16)
    float eps, scale, coef, every;
    const float *qn, *kn;
};

// pg_attention_tc.cu
bool pgk_attention_prompt_tc_supports(const AttnShape &s, const pg_batch *bt, int64_t slots, int64_t ldo, const void *out);
int32_t pgk_attention_prompt_tc(pg_ctx *ctx, const AttnShape &s, const pg_batch *bt, int64_t slots, const bf16 *q, const bf16 *kc, const bf16 *vc, bf16 *out,
                                int64_t ldo);
