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

// f32 -> u32 of the same order (not-a-number becomes 0, below every number)
__device__ __forceinline__ uint32_t order_key(float v)
{
    const uint32_t b = __float_as_uint(v);
    return v != v ? 0u : (b & 0x80000000u) ? ~b : (b | 0x80000000u);
}
// the largest key of the warp and the lowest index that has it; key 0 means none
__device__ __forceinline__ void warp_best(uint32_t &key, int &idx)
{
    const uint32_t k = __reduce_max_sync(0xffffffffu, key);
    idx = (int)__reduce_min_sync(0xffffffffu, key == k && k != 0u ? (unsigned)idx : (unsigned)RT_MAX);
    key = k;
}

// One warp, one token: z = its n <= 32 NV logits; lane l keeps the choice scores of outputs l + 32 i in registers.
// gs: shared, `groups` words, scratch of the warp.
template <int NV>
__device__ __forceinline__ void choose(const float *z, const float *__restrict__ correction, const Choice ch, uint32_t *gs, int32_t *ids, float *weights, int lane)
{
    float e[NV], mx = -INFINITY, sum = 0.0f;
#pragma unroll
    for (int i = 0; i < NV; i++) {
        e[i] = lane + 32 * i < ch.n ? __ldcg(z + lane + 32 * i) : -INFINITY;
        mx = fmaxf(mx, e[i]);
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
#pragma unroll
    for (int i = 0; i < NV; i++) {
        e[i] = expf(e[i] - mx);
        sum += e[i];
    }
    sum = pg_warp_sum(sum);
    uint32_t key[NV];
#pragma unroll
    for (int i = 0; i < NV; i++) {
        e[i] = __fdiv_rn(e[i], sum);
        key[i] = lane + 32 * i < ch.n ? order_key(e[i] + __ldg(correction + lane + 32 * i)) : 0u;
    }
    if (ch.groups > 1) {
        const int per = ch.n / ch.groups;
        for (int g = lane; g < ch.groups; g += 32) gs[g] = 0u;
        __syncwarp();
#pragma unroll
        for (int i = 0; i < NV; i++)
            if (lane + 32 * i < ch.n) atomicMax(gs + (lane + 32 * i) / per, key[i]);
        __syncwarp();
        // the best `keep` groups are marked with all ones (no score has that key), one after the other
        for (int k = 0; k < ch.keep; k++) {
            uint32_t best = 0u;
            int idx = RT_MAX;
            for (int g = lane; g < ch.groups; g += 32) {
                const uint32_t x = gs[g];
                if (x != 0xffffffffu && x > best) best = x, idx = g;
            }
            warp_best(best, idx);
            if (lane == 0 && idx < ch.groups) gs[idx] = 0xffffffffu;
            __syncwarp();
        }
#pragma unroll
        for (int i = 0; i < NV; i++)
            if (lane + 32 * i < ch.n && gs[(lane + 32 * i) / per] != 0xffffffffu) key[i] = 0u;
    }
    for (int k = 0; k < ch.top; k++) {
        uint32_t best = 0u;
        int idx = RT_MAX;
        float w = 0.0f;
#pragma unroll
        for (int i = 0; i < NV; i++)
            if (key[i] > best) best = key[i], idx = lane + 32 * i, w = e[i];
        warp_best(best, idx);
        if (idx >= ch.n) {                                // not-a-number scores choose nothing: weight 0
            if (lane == 0) ids[k] = ch.n - 1, weights[k] = 0.0f;
            continue;
        }
        if ((idx & 31) == lane) {
            ids[k] = idx;
            weights[k] = w;
#pragma unroll
            for (int i = 0; i < NV; i++)
                if (lane + 32 * i == idx) key[i] = 0u;
        }
    }
    __syncwarp();
}

template <int NV>
__global__ void __launch_bounds__(512)
    route_small_kernel(const float *__restrict__ logits, int64_t ld, int m, int experts, const float *__restrict__ correction, const Choice ch,
                       int32_t *ids, float *weights, int32_t *pair_row, int32_t *row_pair, int32_t *block_expert, int32_t *blocks)
{
    extern __shared__ uint32_t sm[];   // groups [16][ch.groups] | ids [m * top] | rank of each pair [m * top] | count, then block, per expert
    __shared__ int chunk[16];
    uint32_t *gs = sm;
    int32_t *sid = reinterpret_cast<int32_t *>(sm + 16 * ch.groups), *rank = sid + m * ch.top, *count = rank + m * ch.top;
    for (int e = threadIdx.x; e < experts; e += 512) count[e] = 0;
    pg_pdl_begin();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, pairs = m * ch.top;
    if (warp < m) choose<NV>(logits + (int64_t)warp * ld, correction, ch, gs + warp * ch.groups, sid + warp * ch.top, weights + warp * ch.top, lane);
    __syncthreads();
    for (int p = threadIdx.x; p < pairs; p += 512) {
        const int id = sid[p];
        ids[p] = id;
        rank[p] = id < experts ? atomicAdd(count + id, 1) : -1;
    }
    __syncthreads();
    // a block of 16 rows per expert in use, in the order of the experts
    int base = 0;
    for (int e0 = 0; e0 < experts; e0 += 512) {
        const int e = e0 + threadIdx.x;
        const bool used = e < experts && count[e] > 0;
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
            for (int r = count[e]; r < PG_ROUTE_SMALL; r++) row_pair[at * PG_ROUTE_SMALL + r] = -1;
            count[e] = at;
        }
        base += all;
        __syncthreads();
    }
    if (threadIdx.x == 0) *blocks = base;
    for (int p = threadIdx.x; p < pairs; p += 512) {
        const int r = rank[p];
        const int row = r >= 0 && r < PG_ROUTE_SMALL ? count[sid[p]] * PG_ROUTE_SMALL + r : -1;
        pair_row[p] = row;
        if (row >= 0) row_pair[row] = p;
    }
}

template <int NV>
__global__ void __launch_bounds__(128)
    route_choose_kernel(const float *__restrict__ logits, int64_t ld, int m, int experts, const float *__restrict__ correction, const Choice ch,
                        int32_t *ids, float *weights, int32_t *count)
{
    extern __shared__ uint32_t sm[];
    pg_pdl_begin();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int t = blockIdx.x * 4 + warp;
    if (t >= m) return;
    choose<NV>(logits + (int64_t)t * ld, correction, ch, sm + warp * ch.groups, ids + (int64_t)t * ch.top, weights + (int64_t)t * ch.top, lane);
    for (int k = lane; k < ch.top; k += 32) {
        const int id = __ldcg(ids + (int64_t)t * ch.top + k);
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
#define PG_RT_SMALL(NV)                                                                                                                                  \
    do {                                                                                                                                                 \
        static std::atomic<uint64_t> set{0};                                                                                                             \
        PG_CUDA(pg_max_smem_once(route_small_kernel<NV>, 220 * 1024, ctx->device, set));                                                                 \
        return launch_pdl(ctx, route_small_kernel<NV>, dim3(1), dim3(512), smem, d_logits, ld, (int)m, (int)route->experts, d_correction, ch, route->ids, \
                          route->weights, route->pair_row, route->row_pair, route->block_expert, route->blocks);                                         \
    } while (0)
#define PG_RT_CHOOSE(NV)                                                                                                                                 \
    launch_pdl(ctx, route_choose_kernel<NV>, dim3((unsigned)((m + 3) / 4)), dim3(128), (size_t)4 * groups * 4, d_logits, ld, (int)m, (int)route->experts, \
               d_correction, ch, route->ids, route->weights, route->count)
    if (small) {
        const size_t smem = ((size_t)16 * groups + 2 * m * route->top + route->experts) * 4;
        PG_REQUIRE(smem <= 220 * 1024, "route: too many choices for the one-CTA form");
        if (n <= 32) PG_RT_SMALL(1);
        if (n <= 128) PG_RT_SMALL(4);
        if (n <= 256) PG_RT_SMALL(8);
        PG_RT_SMALL(32);
    }
    int32_t rc;
    if (n <= 32)
        rc = PG_RT_CHOOSE(1);
    else if (n <= 128)
        rc = PG_RT_CHOOSE(4);
    else if (n <= 256)
        rc = PG_RT_CHOOSE(8);
    else
        rc = PG_RT_CHOOSE(32);
#undef PG_RT_SMALL
#undef PG_RT_CHOOSE
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
