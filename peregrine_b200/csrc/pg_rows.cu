// Row kernels of the f32 residual stream: a row is normalised (x / sqrt(mean(x^2) + eps) * w) and
//
//   EMBED   becomes the residual row, from the token's and, if there are any, the position's embedding (and is not
//           normalised where the model has no norm there)
//   ADD     is added to the residual row, scaled per channel (norm on a sublayer's output)
//   ROUTED  the same, the row being the weighted sum of the token's expert outputs (identity experts: the residual row)
//   PICK    is written out for the product behind it (the rows whose logits are wanted)
//
// and, except for PICK, the new residual row is written again in the type of the products that read it, normalised once
// more with the weights of the next sublayer's norm where the model has one in front of it.  A cluster of up to 8 CTAs
// shares a row when there are few rows.  The row lives in shared memory between the passes.
#include "pg_lm.cuh"

namespace {

constexpr int RW_T = 256;
enum { SRC_EMBED, SRC_ADD, SRC_ROUTED, SRC_PICK };

struct RowArgs {
    const int32_t *tokens, *pos, *rows;
    const bf16 *table, *pos_table;
    const float *y;
    int64_t ldy;
    const void *out;            // routed: expert outputs, rows of ldy
    const int32_t *ids, *pair_row;
    const float *weights;
    int top, experts;
    float *x;
    const float *w, *scale;     // EMBED: w null, no norm; scale null, 1
    const float *next;          // weights of the norm in front of the next sublayer, or null
    float eps;
    int width;
    void *h;
    int64_t ldh;
};

template <typename T, int V>
__device__ __forceinline__ void load_v(const T *p, float (&v)[V])
{
    if constexpr (V == 4 && sizeof(T) == 4) {
        const float4 q = __ldcg(reinterpret_cast<const float4 *>(p));
        v[0] = q.x, v[1] = q.y, v[2] = q.z, v[3] = q.w;
    } else if constexpr (V == 4) {
        const uint2 q = __ldcg(reinterpret_cast<const uint2 *>(p));
        v[0] = pg_bf16_lo(q.x), v[1] = pg_bf16_hi(q.x), v[2] = pg_bf16_lo(q.y), v[3] = pg_bf16_hi(q.y);
    } else {
        v[0] = pg_get(p);
    }
}
template <typename T, int V>
__device__ __forceinline__ void store_v(T *p, const float (&v)[V])
{
    if constexpr (V == 4 && sizeof(T) == 4) {
        *reinterpret_cast<float4 *>(p) = make_float4(v[0], v[1], v[2], v[3]);
    } else if constexpr (V == 4) {
        *reinterpret_cast<uint2 *>(p) = make_uint2(pg_pack_bf16(v[0], v[1]), pg_pack_bf16(v[2], v[3]));
    } else {
        pg_put(p, v[0]);
    }
}

template <int SRC, int V, typename TA>
__global__ void __launch_bounds__(RW_T) row_norm_kernel(const RowArgs a)
{
    extern __shared__ __align__(16) float row[];   // this CTA's segment
    __shared__ float red[32];
    __shared__ float xs[8], xs2[8];
    const uint32_t cs = cl_size(), rank = cl_rank();
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    if (cs > 1) cl_sync();   // every CTA of the cluster runs before anyone stores into it
    asm volatile("griddepcontrol.wait;" ::: "memory");
    const int64_t r = blockIdx.x / cs;
    const int units = a.width / V, seg = (units + (int)cs - 1) / (int)cs;
    const int u0 = (int)rank * seg, u1 = min(units, u0 + seg);
    const int64_t src_row = SRC == SRC_PICK ? __ldcg(a.rows + r) : r;
    float *x = a.x + src_row * a.width;
    const bf16 *tok = nullptr, *ptab = nullptr;
    if (SRC == SRC_EMBED) {
        tok = a.table + (int64_t)__ldcg(a.tokens + r) * a.width;
        if (a.pos_table) ptab = a.pos_table + (int64_t)__ldcg(a.pos + r) * a.width;
    }
    float ss = 0.0f;
    for (int u = u0 + threadIdx.x; u < u1; u += RW_T) {
        float v[V];
        if (SRC == SRC_EMBED) {
            load_v<bf16, V>(tok + (int64_t)u * V, v);
            if (ptab) {
                float p[V];
                load_v<bf16, V>(ptab + (int64_t)u * V, p);
#pragma unroll
                for (int i = 0; i < V; i++) v[i] += p[i];
            }
        } else if (SRC == SRC_ADD) {
            load_v<float, V>(a.y + r * a.ldy + (int64_t)u * V, v);
        } else if (SRC == SRC_PICK) {
            load_v<float, V>(x + (int64_t)u * V, v);
        } else {
#pragma unroll
            for (int i = 0; i < V; i++) v[i] = 0.0f;
            for (int k = 0; k < a.top; k++) {
                const int64_t p = r * a.top + k;
                const float w = __ldcg(a.weights + p);
                const int at = __ldcg(a.pair_row + p);
                float o[V];
                if (at >= 0) {
                    load_v<TA, V>(reinterpret_cast<const TA *>(a.out) + (int64_t)at * a.ldy + (int64_t)u * V, o);
                } else if (__ldcg(a.ids + p) >= a.experts) {
                    load_v<float, V>(x + (int64_t)u * V, o);
                } else {
                    continue;
                }
#pragma unroll
                for (int i = 0; i < V; i++) v[i] = fmaf(w, o[i], v[i]);
            }
        }
        store_v<float, V>(row + (size_t)(u - u0) * V, v);
#pragma unroll
        for (int i = 0; i < V; i++) ss += v[i] * v[i];
    }
    const bool plain = SRC == SRC_EMBED && !a.w;
    float inv = 1.0f, ss2 = 0.0f;
    if (!plain) {
        ss = cl_allreduce<false>(pg_block_sum(ss, red), xs, cs, rank);
        inv = __fdiv_rn(1.0f, sqrtf(__fdiv_rn(ss, (float)a.width) + a.eps));
    }
    TA *h = reinterpret_cast<TA *>(a.h) + r * a.ldh;
    for (int u = u0 + threadIdx.x; u < u1; u += RW_T) {
        float v[V];
#pragma unroll
        for (int i = 0; i < V; i++) v[i] = row[(size_t)(u - u0) * V + i];
        if (SRC == SRC_ADD || SRC == SRC_ROUTED) {
            float b[V];
            load_v<float, V>(x + (int64_t)u * V, b);
#pragma unroll
            for (int i = 0; i < V; i++) {
                const float n = v[i] * inv * __ldg(a.w + u * V + i);
                v[i] = b[i] + (a.scale ? n * __ldg(a.scale + u * V + i) : n);
            }
        } else if (!plain) {
#pragma unroll
            for (int i = 0; i < V; i++) v[i] = v[i] * inv * __ldg(a.w + u * V + i);
        }
        if (SRC != SRC_PICK) store_v<float, V>(x + (int64_t)u * V, v);
        if (SRC == SRC_PICK || !a.next) {
            store_v<TA, V>(h + (int64_t)u * V, v);
        } else {
            store_v<float, V>(row + (size_t)(u - u0) * V, v);   // (read back by the same thread)
#pragma unroll
            for (int i = 0; i < V; i++) ss2 += v[i] * v[i];
        }
    }
    if (SRC == SRC_PICK || !a.next) return;
    ss2 = cl_allreduce<false>(pg_block_sum(ss2, red), xs2, cs, rank);
    const float inv2 = __fdiv_rn(1.0f, sqrtf(__fdiv_rn(ss2, (float)a.width) + a.eps));
    for (int u = u0 + threadIdx.x; u < u1; u += RW_T) {
        float v[V];
#pragma unroll
        for (int i = 0; i < V; i++) v[i] = row[(size_t)(u - u0) * V + i] * inv2 * __ldg(a.next + u * V + i);
        store_v<TA, V>(h + (int64_t)u * V, v);
    }
}

template <int SRC>
int32_t run_rows(pg_ctx *ctx, const RowArgs &a, int64_t rows, int32_t dtype, bool vec)
{
    PG_REQUIRE(a.width > 0 && a.width <= 32768 && a.ldh >= a.width && a.h && a.x && (a.w || SRC == SRC_EMBED), "row norm: bad arguments");
    if (rows == 0) return PG_OK;
    vec = vec && a.width % 4 == 0 && a.ldh % 4 == 0;
    const int V = vec ? 4 : 1;
    int cs = 8;
    while (cs > 1 && (rows * cs > 2 * (int64_t)ctx->sm_count || a.width / cs < 512)) cs >>= 1;
    const int units = a.width / V;
    const size_t smem = (size_t)((units + cs - 1) / cs) * V * 4;
    const dim3 g((unsigned)(rows * cs));
#define PG_ROW_CASE(VV, T)                                                                              \
    {                                                                                                   \
        static std::atomic<uint64_t> set{0};                                                            \
        PG_CUDA(pg_max_smem_once(row_norm_kernel<SRC, VV, T>, 132 * 1024, ctx->device, set));           \
        if (SRC == SRC_EMBED) return launch_whole_cluster(ctx, row_norm_kernel<SRC, VV, T>, g, dim3(RW_T), smem, cs, a); \
        return launch_pdl_cluster(ctx, row_norm_kernel<SRC, VV, T>, g, dim3(RW_T), smem, cs, a);        \
    }
    if (dtype == PG_BF16) {
        if (vec) PG_ROW_CASE(4, bf16)
        PG_ROW_CASE(1, bf16)
    }
    if (vec) PG_ROW_CASE(4, float)
    PG_ROW_CASE(1, float)
#undef PG_ROW_CASE
}

}  // namespace

extern "C" {

PG_API int32_t pg_embed_norm(pg_ctx *ctx, const pg_batch *batch, const void *d_table_bf16, const void *d_pos_table_bf16, int64_t width,
                             const float *d_w, float eps, float *d_x, void *d_h, int32_t dtype, int64_t ldh)
{
    PG_ENTER(ctx);
    PG_REQUIRE(batch && d_table_bf16 && d_pos_table_bf16 && batch->d_tokens && batch->d_pos, "embed_norm: null pointer");
    RowArgs a = {};
    a.tokens = batch->d_tokens;
    a.pos = batch->d_pos;
    a.table = (const bf16 *)d_table_bf16;
    a.pos_table = (const bf16 *)d_pos_table_bf16;
    a.x = d_x, a.w = d_w, a.eps = eps, a.width = (int)width, a.h = d_h, a.ldh = ldh;
    return run_rows<SRC_EMBED>(ctx, a, batch->rows, dtype, true);
}

PG_API int32_t pg_embed_prenorm(pg_ctx *ctx, const pg_batch *batch, const void *d_table_bf16, int64_t width, const float *d_next, float eps, float *d_x,
                                void *d_h, int32_t dtype, int64_t ldh)
{
    PG_ENTER(ctx);
    PG_REQUIRE(batch && d_table_bf16 && d_next && batch->d_tokens, "embed_prenorm: null pointer");
    RowArgs a = {};
    a.tokens = batch->d_tokens;
    a.table = (const bf16 *)d_table_bf16;
    a.x = d_x, a.next = d_next, a.eps = eps, a.width = (int)width, a.h = d_h, a.ldh = ldh;
    return run_rows<SRC_EMBED>(ctx, a, batch->rows, dtype, true);
}

PG_API int32_t pg_norm_add_prenorm(pg_ctx *ctx, const float *d_y, int64_t ldy, float *d_x, const float *d_w, const float *d_next, int64_t rows,
                                   int64_t width, float eps, void *d_h, int32_t dtype, int64_t ldh)
{
    PG_ENTER(ctx);
    PG_REQUIRE(d_y && d_w && ldy >= width, "norm_add_prenorm: bad arguments");
    RowArgs a = {};
    a.y = d_y, a.ldy = ldy, a.next = d_next;
    a.x = d_x, a.w = d_w, a.eps = eps, a.width = (int)width, a.h = d_h, a.ldh = ldh;
    return run_rows<SRC_ADD>(ctx, a, rows, dtype, ldy % 4 == 0);
}

PG_API int32_t pg_norm_add(pg_ctx *ctx, const float *d_y, int64_t ldy, float *d_x, const float *d_w, const float *d_scale, int64_t rows, int64_t width,
                           float eps, void *d_h, int32_t dtype, int64_t ldh)
{
    PG_ENTER(ctx);
    PG_REQUIRE(d_y && d_scale && ldy >= width, "norm_add: bad arguments");
    RowArgs a = {};
    a.y = d_y, a.ldy = ldy, a.scale = d_scale;
    a.x = d_x, a.w = d_w, a.eps = eps, a.width = (int)width, a.h = d_h, a.ldh = ldh;
    return run_rows<SRC_ADD>(ctx, a, rows, dtype, ldy % 4 == 0);
}

PG_API int32_t pg_routed_norm_add(pg_ctx *ctx, const pg_route *route, const void *d_out, int64_t ldo, float *d_x, const float *d_w,
                                  const float *d_scale, int64_t rows, int64_t width, float eps, void *d_h, int32_t dtype, int64_t ldh)
{
    PG_ENTER(ctx);
    PG_REQUIRE(route && d_out && d_scale && ldo >= width && rows == route->m, "routed_norm_add: bad arguments");
    RowArgs a = {};
    a.out = d_out, a.ldy = ldo, a.scale = d_scale;
    a.ids = route->ids, a.pair_row = route->pair_row, a.weights = route->weights, a.top = (int)route->top, a.experts = (int)route->experts;
    a.x = d_x, a.w = d_w, a.eps = eps, a.width = (int)width, a.h = d_h, a.ldh = ldh;
    return run_rows<SRC_ROUTED>(ctx, a, rows, dtype, ldo % 4 == 0);
}

PG_API int32_t pg_norm_rows(pg_ctx *ctx, const float *d_x, const int32_t *d_rows, int64_t m, int64_t width, const float *d_w, float eps, void *d_h,
                            int32_t dtype, int64_t ldh)
{
    PG_ENTER(ctx);
    PG_REQUIRE(d_rows, "norm_rows: null pointer");
    RowArgs a = {};
    a.rows = d_rows;
    a.x = const_cast<float *>(d_x), a.w = d_w, a.eps = eps, a.width = (int)width, a.h = d_h, a.ldh = ldh;
    return run_rows<SRC_PICK>(ctx, a, m, dtype, true);
}

}  // extern "C"
