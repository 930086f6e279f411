// Greedy choice of the next tokens (examples/llama/main.rs:15-26: the first maximum wins), for one vocabulary per GPU
// and for a vocabulary sharded by column.
#include <math.h>

#include "pg_internal.cuh"
#include "pg_launch.cuh"

namespace {

// a cluster of cs CTAs per row, each scanning V / cs logits; the first maximum wins (examples/llama/main.rs:15-26).
// The first CTA of row 0 also advances the position; with row_pos every row has a position of its own, which its first
// CTA advances.
// PEER (po.world > 0): `logits` holds this rank's V columns of a vocabulary sharded by column; the row's local
// (maximum, index + v0) pair goes to slot [b][rank] of every rank's exchange buffer instead of tokens[b], and
// pick_embed_kernel chooses among the ranks' pairs.
__global__ void __launch_bounds__(1024) argmax_kernel(const float *__restrict__ logits, int V, int *__restrict__ tokens, int *pos_ptr,
                                                       int pos_limit, int row_pos, int v0, const PgPeerOut po)
{
    __shared__ float bv[32];
    __shared__ int bi[32];
    __shared__ float xv[8];
    __shared__ int xi[8];
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    asm volatile("griddepcontrol.wait;" ::: "memory");
    const uint32_t cs = cl_size(), rank = cl_rank();
    const int b = blockIdx.x / cs;
    const float *row = logits + (int64_t)b * V;
    const int seg = (V + (int)cs - 1) / (int)cs;
    const int i0 = (int)rank * seg, i1 = min(V, i0 + seg);
    float best = -INFINITY;
    int idx = 0x7fffffff;
    for (int i = i0 + threadIdx.x; i < i1; i += blockDim.x) {
        const float v = pg_ld_fresh(row + i);
        if (v > best || (v == best && i < idx)) {
            best = v;
            idx = i;
        }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        const float ov = __shfl_xor_sync(0xffffffffu, best, o);
        const int oi = __shfl_xor_sync(0xffffffffu, idx, o);
        if (ov > best || (ov == best && oi < idx)) {
            best = ov;
            idx = oi;
        }
    }
    if ((threadIdx.x & 31) == 0) {
        bv[threadIdx.x >> 5] = best;
        bi[threadIdx.x >> 5] = idx;
    }
    __syncthreads();
    if (threadIdx.x == 0) {
        for (int w = 1; w < (int)(blockDim.x >> 5); w++)
            if (bv[w] > best || (bv[w] == best && bi[w] < idx)) {
                best = bv[w];
                idx = bi[w];
            }
        if (cs > 1) {
            cl_store_f32(xv + rank, 0, best);     // everything meets in the first CTA of the cluster
            cl_store_s32(xi + rank, 0, idx);
        }
    }
    if (cs > 1) cl_sync();
    if (threadIdx.x == 0 && rank == 0) {
        for (uint32_t c = 1; c < cs; c++)
            if (xv[c] > best || (xv[c] == best && xi[c] < idx)) {
                best = xv[c];
                idx = xi[c];
            }
        if (po.world > 0) {
            // an all-NaN (or empty) slice never wins: -inf with the slice's first index
            pg_cell_store2(po, pg_cell_seq(po), b, 0, (idx == 0x7fffffff) ? -INFINITY : best,
                           __int_as_float((idx == 0x7fffffff) ? v0 : idx + v0));
        } else {
            tokens[b] = (idx == 0x7fffffff) ? 0 : idx;   // all-NaN row: the reference keeps index 0
            if (pos_ptr && (b == 0 || row_pos)) {
                int *pp = pos_ptr + (row_pos ? b : 0);
                const int p = pg_ld_fresh(pp);
                if (pos_limit <= 0 || p < pos_limit) *pp = p + 1;   // never past the end of the cache
            }
        }
    }
    if (po.world > 0) pg_cell_finish(po, pg_cell_seq(po), threadIdx.x);
}

}  // namespace

static const PgPeerOut NO_PEER_OUT = {};

// tokens[b] = argmax(logits[b, :]) (first maximum); d_pos (nullable) is advanced by one, but never beyond pos_limit
// (pass the KV capacity; 0 = no limit): a decode loop that runs off the end of its cache stops advancing instead of
// writing behind it.
extern "C" PG_API int32_t pg_argmax_advance(pg_ctx *ctx, const float *d_logits, int64_t B, int64_t V, int32_t *d_tokens, int32_t *d_pos, int64_t pos_limit)
{
    PG_ENTER(ctx);
    PG_REQUIRE(d_logits && d_tokens && V > 0 && V <= 0x7fffffff, "argmax: bad arguments");
    if (B == 0) return PG_OK;
    const int cs = row_cluster(ctx, B, V, 4096);
    return launch_pdl_cluster(ctx, argmax_kernel, dim3((unsigned)(B * cs)), dim3(1024), 0, cs, d_logits, (int)V, (int *)d_tokens, (int *)d_pos,
                              (int)pos_limit, 0, 0, NO_PEER_OUT);
}

// The same with one position per row (sequences of different lengths): d_pos [B].
extern "C" PG_API int32_t pg_argmax_rows(pg_ctx *ctx, const float *d_logits, int64_t B, int64_t V, int32_t *d_tokens, int32_t *d_pos, int64_t pos_limit)
{
    PG_ENTER(ctx);
    PG_REQUIRE(d_logits && d_tokens && V > 0 && V <= 0x7fffffff, "argmax: bad arguments");
    if (B == 0) return PG_OK;
    const int cs = row_cluster(ctx, B, V, 4096);
    return launch_pdl_cluster(ctx, argmax_kernel, dim3((unsigned)(B * cs)), dim3(1024), 0, cs, d_logits, (int)V, (int *)d_tokens, (int *)d_pos,
                              (int)pos_limit, 1, 0, NO_PEER_OUT);
}

int32_t pgk_argmax_peer(pg_ctx *ctx, const float *d_logits, int64_t B, int64_t V, int v0, const PgPeerOut &out)
{
    const int cs = row_cluster(ctx, B, V, 1024);
    return launch_pdl_cluster(ctx, argmax_kernel, dim3((unsigned)(B * cs)), dim3(1024), 0, cs, d_logits, (int)V, (int *)nullptr, (int *)nullptr,
                              0, 0, v0, out);
}
