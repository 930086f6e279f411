// Products with bf16 weights: the handle and the choice of kernel (include/peregrine_b200_lm.h).
#include <algorithm>
#include <new>

#include "pg_lm.cuh"

extern "C" {

PG_API int32_t pg_linear_wrap(pg_ctx *ctx, const void *d_w_bf16, int64_t n, int64_t k, int64_t experts, pg_linear **out)
{
    PG_ENTER(ctx);
    PG_REQUIRE(out != nullptr, "linear_wrap: out is null");
    *out = nullptr;
    PG_REQUIRE(d_w_bf16 && n > 0 && k > 0 && experts > 0, "linear_wrap: bad arguments");
    PG_REQUIRE(k % 64 == 0 && ((uintptr_t)d_w_bf16 & 15) == 0, "linear_wrap: K must be a multiple of 64 (K = %lld) and the weights 16-byte aligned",
               (long long)k);
    PG_REQUIRE(n < (1 << 30) && k < (1 << 30), "linear_wrap: shape too large");
    // now, since the workspace cannot grow while a step is being recorded
    const int32_t rc = pg_splitk_reserve(ctx, std::max(pgk_linear_gemv_workspace(n, k), PG_LM_TICKET_BYTES + (size_t)ctx->sm_count * 128 * 128 * sizeof(float)));
    if (rc != PG_OK) return rc;
    pg_linear *l = new (std::nothrow) pg_linear();
    if (!l) PG_FAIL(PG_ERR_NOMEM, "out of host memory");
    l->w = (const bf16 *)d_w_bf16;
    l->n = n;
    l->k = k;
    l->experts = experts;
    *out = l;
    return PG_OK;
}

PG_API int32_t pg_linear_free(pg_ctx *ctx, pg_linear *lin)
{
    (void)ctx;
    delete lin;
    return PG_OK;
}

PG_API int32_t pg_linear_run(pg_ctx *ctx, pg_linear *lin, const void *d_a, int32_t dtype, int64_t m, int32_t act, float limit, void *d_y,
                             int32_t y_dtype, int64_t ldy)
{
    return pg_linear_run_ld(ctx, lin, d_a, lin ? lin->k : 0, dtype, m, act, limit, d_y, y_dtype, ldy);
}

PG_API int32_t pg_linear_run_ld(pg_ctx *ctx, pg_linear *lin, const void *d_a, int64_t lda, int32_t dtype, int64_t m, int32_t act, float limit, void *d_y,
                                int32_t y_dtype, int64_t ldy)
{
    PG_ENTER(ctx);
    PG_REQUIRE(lin && d_a && d_y && m >= 0, "linear: bad arguments");
    PG_REQUIRE(lda >= lin->k && lda % 8 == 0, "linear: rows of a are %lld apart, K is %lld (and a multiple of 8 is wanted)", (long long)lda, (long long)lin->k);
    PG_REQUIRE(act >= PG_ACT_NONE && act <= PG_ACT_CLAMPED_SWISH_GLU && (act == PG_ACT_NONE || (lin->n % 16 == 0 && y_dtype == dtype)),
               "linear: bad activation");
    PG_REQUIRE(ldy >= (act == PG_ACT_NONE ? lin->n : lin->n / 2) && ((uintptr_t)d_a & 15) == 0, "linear: output rows too short or operand not aligned");
    if (m == 0) return PG_OK;
    if (dtype == PG_F32) return pgk_linear_f32(ctx, lin, (const float *)d_a, lda, m, act, limit, d_y, y_dtype, ldy, nullptr);
    if (pgk_linear_gemv_supports(lin, m)) return pgk_linear_gemv(ctx, lin, (const bf16 *)d_a, lda, m, act, limit, d_y, y_dtype, ldy, nullptr, 1);
    return pgk_linear_tc(ctx, lin, (const bf16 *)d_a, lda, m, act, limit, d_y, y_dtype, ldy, nullptr);
}

PG_API int32_t pg_linear_run_routed(pg_ctx *ctx, pg_linear *lin, pg_route *route, const void *d_a, int32_t dtype, int32_t by_token, int32_t act,
                                    float limit, void *d_y, int32_t y_dtype, int64_t ldy)
{
    PG_ENTER(ctx);
    PG_REQUIRE(lin && route && d_a && d_y && lin->experts == route->experts, "linear: bad arguments");
    PG_REQUIRE(act >= PG_ACT_NONE && act <= PG_ACT_CLAMPED_SWISH_GLU && (act == PG_ACT_NONE || (lin->n % 16 == 0 && y_dtype == dtype)),
               "linear: bad activation");
    PG_REQUIRE(ldy >= (act == PG_ACT_NONE ? lin->n : lin->n / 2) && ((uintptr_t)d_a & 15) == 0, "linear: output rows too short or operand not aligned");
    if (route->m == 0) return PG_OK;
    const PgRouted rt = {route->blocks, route->block_expert, route->row_pair, (int)route->top, by_token};
    if (route->block == PG_ROUTE_SMALL) {
        PG_REQUIRE(dtype == PG_BF16 && pgk_linear_gemv_supports(lin, 1), "linear: the route was made for the streaming form");
        const int64_t pairs = route->m * route->top;
        return pgk_linear_gemv(ctx, lin, (const bf16 *)d_a, lin->k, route->m, act, limit, d_y, y_dtype, ldy, &rt, pairs < route->experts ? pairs : route->experts);
    }
    // rows the route can have for this many tokens
    const int64_t pairs = route->m * route->top;
    const int64_t rows = pg_up(pairs + (pairs < route->experts ? pairs : route->experts) * (PG_ROUTE_BLOCK - 1), PG_ROUTE_BLOCK);
    PG_REQUIRE(rows <= route->max_rows, "linear: the route is larger than it was created for");
    const void *a = d_a;
    if (by_token) {
        // the tokens' rows in the order of the route
        const size_t row_bytes = (size_t)lin->k * (dtype == PG_F32 ? 4 : 2);
        const int32_t rr = pg_scratch_reserve(ctx, (size_t)rows * row_bytes);
        if (rr != PG_OK) return rr;
        const int32_t rc = pgk_route_gather(ctx, route, d_a, row_bytes, ctx->scratch);
        if (rc != PG_OK) return rc;
        a = ctx->scratch;
    }
    if (dtype == PG_F32) return pgk_linear_f32(ctx, lin, (const float *)a, lin->k, rows, act, limit, d_y, y_dtype, ldy, &rt);
    return pgk_linear_tc(ctx, lin, (const bf16 *)a, lin->k, rows, act, limit, d_y, y_dtype, ldy, &rt);
}

}  // extern "C"
