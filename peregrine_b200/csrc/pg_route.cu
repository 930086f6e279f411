// Mixture-of-experts routing: softmax scores over all router outputs, choice by score + correction among the best
// groups of neighbours, weights = the chosen scores as they are; then the (token, choice) pairs ordered by expert.
//
//   up to 16 tokens      one CTA: a warp chooses for each token, then the CTA writes one 16-row block per expert in use
//   more                 a warp per token counts per expert; one CTA lays out 128-row blocks; pairs take their rows.
//                        (Which row of its expert a pair gets is left to the order of arrival: rows do not meet in any
//                        sum, and a token adds its own pairs up in the order of its choices.)
#include <math.h>

#include <new>

#include "pg_lm.cuh"

namespace {

constexpr int RT_MAX = 1024;   // most router outputs

struct Choice {
    int n, top, groups, keep;
};

__device__ __forceinline__ void warp_argmax(float &v, int &i)
{
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        const float ov = __shfl_xor_sync(0xffffffffu, v, o);
        const int oi = __shfl_xor_sync(0xffffffffu, i, o);
        if (ov > v || (ov == v && oi < i)) {
            v = ov;
            i = oi;
        }
    }
}

// One warp, one token: z = its n logits; c (shared, n floats) and gs (shared, `groups` floats) are scratch of the warp.
__device__ __forceinline__ void choose(const float *z, const float *__restrict__ correction, const Choice ch, float *c, float *gs, int32_t *ids,
                                       float *weights, int lane)
{
    float mx = -INFINITY;
    for (int i = lane; i < ch.n; i += 32) mx = fmaxf(mx, __ldcg(z + i));
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
    float sum = 0.0f;
    for (int i = lane; i < ch.n; i += 32) sum += expf(__ldcg(z + i) - mx);
    sum = pg_warp_sum(sum);
    for (int i = lane; i < ch.n; i += 32) c[i] = __fdiv_rn(expf(__ldcg(z + i) - mx), sum) + __ldg(correction + i);
    __syncwarp();
    if (ch.groups > 1) {
        const int per = ch.n / ch.groups;
        for (int g = lane; g < ch.groups; g += 32) {
            float b = -INFINITY;
            for (int i = 0; i < per; i++) b = fmaxf(b, c[g * per + i]);
            gs[g] = b;
        }
        __syncwarp();
        // the best `keep` groups are marked with +inf, one after the other
        for (int k = 0; k < ch.keep; k++) {
            float v = -INFINITY;
            int idx = RT_MAX;
            for (int g = lane; g < ch.groups; g += 32) {
                const float x = gs[g];
                if (x != INFINITY && (x > v || (x == v && g < idx))) {
                    v = x;
                    idx = g;
                }
            }
            warp_argmax(v, idx);
            __syncwarp();
            if (lane == 0 && idx < ch.groups) gs[idx] = INFINITY;
            __syncwarp();
        }
        for (int i = lane; i < ch.n; i += 32)
            if (gs[i / per] != INFINITY) c[i] = -INFINITY;
        __syncwarp();
    }
    for (int k = 0; k < ch.top; k++) {
        float v = -INFINITY;
        int idx = RT_MAX;
        for (int i = lane; i < ch.n; i += 32) {
            const float x = c[i];
            if (x > v || (x == v && x != -INFINITY && i < idx)) {
                v = x;
                idx = i;
            }
        }
        warp_argmax(v, idx);
        const bool found = idx < ch.n;                    // not-a-number scores choose nothing: weight 0
        if (!found) idx = ch.n - 1;
        __syncwarp();
        if (lane == 0) {
            ids[k] = idx;
            weights[k] = found ? __fdiv_rn(expf(__ldcg(z + idx) - mx), sum) : 0.0f;
            if (found) c[idx] = -INFINITY;
        }
        __syncwarp();
    }
}

__global__ void __launch_bounds__(512)
    route_small_kernel(const float *__restrict__ logits, int64_t ld, int m, int experts, const float *__restrict__ correction, const Choice ch,
                       int32_t *ids, float *weights, int32_t *pair_row, int32_t *row_pair, int32_t *block_expert, int32_t *blocks)
{
    extern __shared__ float sm[];      // [16][n + groups] scratch, then [m * top] ids
    __shared__ int chunk[32];
    pg_pdl_begin();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    float *c = sm + (size_t)warp * (ch.n + ch.groups);
    int32_t *sid = reinterpret_cast<int32_t *>(sm + 16 * (size_t)(ch.n + ch.groups));
    if (warp < m) {
        choose(logits + (int64_t)warp * ld, correction, ch, c, c + ch.n, sid + warp * ch.top, weights + warp * ch.top, lane);
        for (int k = lane; k < ch.top; k += 32) {
            const int id = sid[warp * ch.top + k];
            ids[warp * ch.top + k] = id;
            if (id >= experts) pair_row[warp * ch.top + k] = -1;
        }
    }
    __syncthreads();
    const int pairs = m * ch.top;
    // a block of 16 rows per expert in use, in the order of the experts
    int base = 0;
    for (int e0 = 0; e0 < experts; e0 += 512) {
        const int e = e0 + threadIdx.x;
        bool used = false;
        if (e < experts)
            for (int p = 0; p < pairs && !used; p++) used = sid[p] == e;
        const unsigned ballot = __ballot_sync(0xffffffffu, used);
        if (lane == 0) chunk[warp] = __popc(ballot);
        __syncthreads();
        int at = base + __popc(ballot & ((1u << lane) - 1u)), all = 0;
        for (int w = 0; w < 16; w++) {
            if (w < warp) at += chunk[w];
            all += chunk[w];
        }
        if (used) {
            block_expert[at] = e;
            int r = 0;
            for (int p = 0; p < pairs; p++)
                if (sid[p] == e) {
                    pair_row[p] = r < PG_ROUTE_SMALL ? at * PG_ROUTE_SMALL + r : -1;
                    if (r < PG_ROUTE_SMALL) row_pair[at * PG_ROUTE_SMALL + r] = p;
                    r++;
                }
            for (; r < PG_ROUTE_SMALL; r++) row_pair[at * PG_ROUTE_SMALL + r] = -1;
        }
        base += all;
        __syncthreads();
    }
    if (threadIdx.x == 0) *blocks = base;
}

__global__ void __launch_bounds__(128)
    route_choose_kernel(const float *__restrict__ logits, int64_t ld, int m, int experts, const float *__restrict__ correction, const Choice ch,
                        int32_t *ids, float *weights, int32_t *count)
{
    extern __shared__ float sm[];
    pg_pdl_begin();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int t = blockIdx.x * 4 + warp;
    if (t >= m) return;
    float *c = sm + (size_t)warp * (ch.n + ch.groups);
    choose(logits + (int64_t)t * ld, correction, ch, c, c + ch.n, ids + (int64_t)t * ch.top, weights + (int64_t)t * ch.top, lane);
    __syncwarp();
    if (lane == 0)
        for (int k = 0; k < ch.top; k++) {
            const int id = ids[(int64_t)t * ch.top + k];
            if (id < experts) atomicAdd(count + id, 1);
        }
}

// count -> first row of every expert (in cursor), the experts of the row blocks, the number of row blocks; count back to 0
__global__ void __launch_bounds__(1024) route_layout_kernel(int experts, int32_t *count, int32_t *cursor, int32_t *block_expert, int32_t *blocks)
{
    __shared__ int part[32];
    pg_pdl_begin();
    const int e = threadIdx.x, warp = e >> 5, lane = e & 31;
    const int nb = e < experts ? (__ldcg(count + e) + PG_ROUTE_BLOCK - 1) / PG_ROUTE_BLOCK : 0;
    int inc = nb;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
        const int v = __shfl_up_sync(0xffffffffu, inc, o);
        if (lane >= o) inc += v;
    }
    if (lane == 31) part[warp] = inc;
    __syncthreads();
    int at = inc - nb, all = 0;
    for (int w = 0; w < 32; w++) {
        if (w < warp) at += part[w];
        all += part[w];
    }
    if (e < experts) {
        count[e] = 0;
        cursor[e] = at * PG_ROUTE_BLOCK;
        for (int i = 0; i < nb; i++) block_expert[at + i] = e;
    }
    if (e == 0) *blocks = all;
}

__global__ void __launch_bounds__(256) route_place_kernel(int pairs, int experts, const int32_t *ids, int32_t *cursor, int32_t *pair_row, int32_t *row_pair)
{
    pg_pdl_begin();
    const int p = blockIdx.x * 256 + threadIdx.x;
    if (p >= pairs) return;
    const int e = __ldcg(ids + p);
    int row = -1;
    if (e < experts) {
        row = atomicAdd(cursor + e, 1);
        row_pair[row] = p;
    }
    pair_row[p] = row;
}

// one CTA per token: its row of h to the rows of its pairs (16-byte words)
__global__ void __launch_bounds__(256) route_gather_kernel(const uint4 *__restrict__ h, int words, int top, const int32_t *pair_row, uint4 *__restrict__ out)
{
    pg_pdl_begin();
    const int64_t t = blockIdx.x;
    for (int i = threadIdx.x; i < words; i += 256) {
        const uint4 v = __ldcg(h + t * words + i);
        for (int k = 0; k < top; k++) {
            const int row = __ldcg(pair_row + t * top + k);
            if (row >= 0) out[(int64_t)row * words + i] = v;
        }
    }
}

}  // namespace

int32_t pgk_route_gather(pg_ctx *ctx, const pg_route *route, const void *h, size_t row_bytes, void *out)
{
    return launch_pdl(ctx, route_gather_kernel, dim3((unsigned)route->m), dim3(256), 0, (const uint4 *)h, (int)(row_bytes / 16), (int)route->top,
                      (const int32_t *)route->pair_row, (uint4 *)out);
}

extern "C" {

PG_API int32_t pg_route_create(pg_ctx *ctx, int64_t max_tokens, int64_t experts, int64_t identity, int64_t top, pg_route **out)
{
    PG_ENTER(ctx);
    PG_REQUIRE(out != nullptr, "route_create: out is null");
    *out = nullptr;
    PG_REQUIRE(max_tokens > 0 && experts > 0 && identity >= 0 && experts + identity <= RT_MAX && top > 0 && top <= experts + identity,
               "route_create: bad arguments (at most %d router outputs)", RT_MAX);
    pg_route *r = new (std::nothrow) pg_route();
    if (!r) PG_FAIL(PG_ERR_NOMEM, "out of host memory");
    r->max_tokens = max_tokens;
    r->experts = experts;
    r->identity = identity;
    r->top = top;
    const int64_t pairs = max_tokens * top, used = pairs < experts ? pairs : experts;
    r->max_rows = pg_up(pairs + used * (PG_ROUTE_BLOCK - 1), PG_ROUTE_BLOCK);
    const int64_t nblk = r->max_rows / PG_ROUTE_SMALL;
    const int64_t words = 3 * pg_up(pairs, 32) + pg_up(r->max_rows, 32) + 2 * pg_up(experts, 32) + pg_up(nblk, 32) + 32;
    const cudaError_t e = cudaMalloc(&r->mem, (size_t)words * 4);
    if (e != cudaSuccess) {
        delete r;
        PG_FAIL(e == cudaErrorMemoryAllocation ? PG_ERR_NOMEM : PG_ERR_CUDA, "route_create: %s", cudaGetErrorString(e));
    }
    int32_t *p = (int32_t *)r->mem;
    r->ids = p, p += pg_up(pairs, 32);
    r->weights = (float *)p, p += pg_up(pairs, 32);
    r->pair_row = p, p += pg_up(pairs, 32);
    r->row_pair = p, p += pg_up(r->max_rows, 32);
    r->count = p, p += pg_up(experts, 32);
    r->cursor = p, p += pg_up(experts, 32);
    r->block_expert = p, p += pg_up(nblk, 32);
    r->blocks = p;
    const cudaError_t z = cudaMemsetAsync(r->mem, 0, (size_t)words * 4, ctx->stream);
    if (z != cudaSuccess) {
        cudaFree(r->mem);
        delete r;
        PG_FAIL(PG_ERR_CUDA, "route_create: %s", cudaGetErrorString(z));
    }
    *out = r;
    return PG_OK;
}

PG_API int32_t pg_route_free(pg_ctx *ctx, pg_route *route)
{
    if (!route) return PG_OK;
    PG_ENTER(ctx);
    PG_CUDA(cudaStreamSynchronize(ctx->stream));
    cudaFree(route->mem);
    delete route;
    return PG_OK;
}

PG_API int64_t pg_route_max_rows(const pg_route *route) { return route ? route->max_rows : 0; }

PG_API int32_t pg_route_run(pg_ctx *ctx, pg_route *route, int32_t dtype, const float *d_logits, int64_t ld, int64_t m, const float *d_correction,
                            int32_t groups, int32_t keep)
{
    PG_ENTER(ctx);
    PG_REQUIRE(route && d_logits && d_correction && m >= 0 && m <= route->max_tokens, "route: bad arguments");
    const int n = (int)(route->experts + route->identity);
    if (groups < 1) groups = 1;
    PG_REQUIRE(groups == 1 || (n % groups == 0 && keep >= 1 && keep <= groups && (int64_t)keep * (n / groups) >= route->top),
               "route: %d groups of %d outputs, keep %d, top %d", groups, n, keep, (int)route->top);
    PG_REQUIRE(ld >= n, "route: logit rows too short");
    route->m = m;
    const bool small = dtype == PG_BF16 && m <= PG_ROUTE_SMALL;
    route->block = small ? PG_ROUTE_SMALL : PG_ROUTE_BLOCK;
    if (m == 0) return PG_OK;
    const Choice ch = {n, (int)route->top, groups, keep};
    if (small) {
        const size_t smem = (size_t)16 * (n + groups) * 4 + (size_t)m * route->top * 4;
        PG_REQUIRE(smem <= 200 * 1024, "route: too many router outputs");
        static std::atomic<uint64_t> set{0};
        PG_CUDA(pg_max_smem_once(route_small_kernel, 200 * 1024, ctx->device, set));
        return launch_pdl(ctx, route_small_kernel, dim3(1), dim3(512), smem, d_logits, ld, (int)m, (int)route->experts, d_correction, ch, route->ids,
                          route->weights, route->pair_row, route->row_pair, route->block_expert, route->blocks);
    }
    int32_t rc = launch_pdl(ctx, route_choose_kernel, dim3((unsigned)((m + 3) / 4)), dim3(128), (size_t)4 * (n + groups) * 4, d_logits, ld, (int)m,
                            (int)route->experts, d_correction, ch, route->ids, route->weights, route->count);
    if (rc != PG_OK) return rc;
    rc = launch_pdl(ctx, route_layout_kernel, dim3(1), dim3(1024), 0, (int)route->experts, route->count, route->cursor, route->block_expert, route->blocks);
    if (rc != PG_OK) return rc;
    const int64_t pairs = m * route->top;
    return launch_pdl(ctx, route_place_kernel, dim3((unsigned)((pairs + 255) / 256)), dim3(256), 0, (int)pairs, (int)route->experts,
                      (const int32_t *)route->ids, route->cursor, route->pair_row, route->row_pair);
}

PG_API int32_t pg_route_read(pg_ctx *ctx, const pg_route *route, int32_t *ids, float *weights)
{
    PG_ENTER(ctx);
    PG_REQUIRE(route && ids && weights, "route_read: null pointer");
    const size_t bytes = (size_t)(route->m * route->top) * 4;
    if (bytes) {
        PG_CUDA(cudaMemcpyAsync(ids, route->ids, bytes, cudaMemcpyDeviceToHost, ctx->stream));
        PG_CUDA(cudaMemcpyAsync(weights, route->weights, bytes, cudaMemcpyDeviceToHost, ctx->stream));
    }
    PG_CUDA(cudaStreamSynchronize(ctx->stream));
    return PG_OK;
}

}  // extern "C"
