// Internal declarations of libperegrine_b200_lm: objects, small conversions and the launchers that cross files.
#pragma once

#include <cuda.h>
#include <cuda_bf16.h>

#include "peregrine_b200_lm.h"
#include "pg_internal.cuh"
#include "pg_launch.cuh"

typedef __nv_bfloat16 bf16;

struct pg_linear {
    const bf16 *w = nullptr;   // [experts][n][k]
    int64_t n = 0, k = 0, experts = 1;
    alignas(64) unsigned char tmap[2][128];   // TMA descriptors of w, one per tile height in use
    int tmap_rows[2] = {0, 0};
};

constexpr int PG_ROUTE_SMALL = 16;    // most tokens of the one-CTA form, and its row block
constexpr int PG_ROUTE_BLOCK = 128;   // row block of the other form

// A route orders the (token, choice) pairs by expert.  Every expert's rows start at a multiple of `block`, so a block
// of rows has one expert; identity pairs have no row.
struct pg_route {
    int64_t max_tokens = 0, experts = 0, identity = 0, top = 0, max_rows = 0, m = 0;
    int block = PG_ROUTE_BLOCK;
    void *mem = nullptr;
    int32_t *ids = nullptr;        // [m * top] expert of each pair (>= experts: identity)
    float *weights = nullptr;      // [m * top]
    int32_t *pair_row = nullptr;   // [m * top] row of the pair, -1 for identity
    int32_t *row_pair = nullptr;   // [max_rows] pair of the row, -1 for padding
    int32_t *count = nullptr;      // [experts] (zero between steps in the many-token form)
    int32_t *cursor = nullptr;     // [experts]
    int32_t *block_expert = nullptr;   // [max_rows / block]
    int32_t *blocks = nullptr;     // [1] row blocks in use
};

inline int64_t pg_up(int64_t v, int64_t to) { return (v + to - 1) / to * to; }

// what a routed product needs of a route
struct PgRouted {
    const int32_t *blocks, *block_expert, *row_pair;
    int top, by_token;
};

// The context's split-K workspace: tickets, zero between calls, then slabs.
constexpr size_t PG_LM_TICKET_BYTES = 64 * 1024;
// what pg_linear_wrap reserves for the streaming form of a matrix, and for the tensor-core form (a tile of 128 x 128 per SM)
size_t pgk_linear_gemv_workspace(int64_t n, int64_t k);

// pg_linear_gemv.cu: m <= 16 rows (or row blocks of 16) against streamed weights
bool pgk_linear_gemv_supports(const pg_linear *lin, int64_t m);
int32_t pgk_linear_gemv(pg_ctx *ctx, const pg_linear *lin, const bf16 *a, int64_t lda, int64_t m, int act, float limit, void *y, int y_dtype, int64_t ldy,
                        const PgRouted *routed, int64_t max_blocks);
// pg_linear_tc.cu
int32_t pgk_linear_tc(pg_ctx *ctx, pg_linear *lin, const bf16 *a, int64_t lda, int64_t m, int act, float limit, void *y, int y_dtype, int64_t ldy,
                      const PgRouted *routed);
// pg_linear_f32.cu
int32_t pgk_linear_f32(pg_ctx *ctx, const pg_linear *lin, const float *a, int64_t lda, int64_t m, int act, float limit, void *y, int y_dtype, int64_t ldy,
                       const PgRouted *routed);
// pg_route.cu: rows of h in the order of the route (many-token form)
int32_t pgk_route_gather(pg_ctx *ctx, const pg_route *route, const void *h, size_t row_bytes, void *out);

#ifdef __CUDACC__
__device__ __forceinline__ void pg_put(float *p, float v) { *p = v; }
__device__ __forceinline__ void pg_put(bf16 *p, float v) { *p = __float2bfloat16_rn(v); }
__device__ __forceinline__ float pg_get(const float *p) { return __ldcg(p); }
__device__ __forceinline__ float pg_get(const bf16 *p)
{
    const unsigned short b = __ldcg(reinterpret_cast<const unsigned short *>(p));
    return __uint_as_float((uint32_t)b << 16);
}
__device__ __forceinline__ float pg_get_plain(const float *p) { return *p; }   // (shared memory)
__device__ __forceinline__ float pg_get_plain(const bf16 *p) { return __uint_as_float((uint32_t)*reinterpret_cast<const unsigned short *>(p) << 16); }
__device__ __forceinline__ uint32_t pg_pack_bf16(float lo, float hi)
{
    const __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<const uint32_t *>(&v);
}
__device__ __forceinline__ float pg_bf16_lo(uint32_t v) { return __uint_as_float(v << 16); }
__device__ __forceinline__ float pg_bf16_hi(uint32_t v) { return __uint_as_float(v & 0xffff0000u); }

__device__ __forceinline__ void pg_pdl_begin()
{
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    asm volatile("griddepcontrol.wait;" ::: "memory");
}

// (the quick division is within two units in the last place, and 0 where the denominator is beyond 2^126)
__device__ __forceinline__ float pg_sigmoid(float z) { return __fdividef(1.0f, 1.0f + expf(-z)); }
__device__ __forceinline__ float pg_silu(float z) { return __fdividef(z, 1.0f + expf(-z)); }
__device__ __forceinline__ float pg_gelu_tanh(float z)
{
    const float c = 0.7978845608028654f;   // sqrt(2 / pi)
    return 0.5f * z * (1.0f + tanhf(c * (z + 0.044715f * z * z * z)));
}
// one gated output of a product (pg_act)
template <int ACT>
__device__ __forceinline__ float pg_glu(float g, float u, float limit)
{
    if (ACT == PG_ACT_GELU_TANH_GLU) return pg_gelu_tanh(g) * u;
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit);
    return g * pg_sigmoid(1.702f * g) * (u + 1.0f);
}
// 2^x, within two units in the last place (results below 2^-126 become 0)
__device__ __forceinline__ float pg_ex2(float x)
{
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ float pg_warp_sum(float v)
{
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
// sum over a CTA of at most 1024 threads; red: 32 floats not in use by anything else in flight
__device__ __forceinline__ float pg_block_sum(float v, float *red)
{
    v = pg_warp_sum(v);
    __syncthreads();
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    float r = 0.0f;
    for (int i = 0; i < (int)(blockDim.x >> 5); i++) r += red[i];
    return r;
}
#endif
