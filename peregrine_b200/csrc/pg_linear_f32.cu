// y = a W^T in true f32: bf16 weights widened exactly, FFMA sums.  64 x 64 tiles, 4 x 4 outputs per thread; the tile
// edges are masked on load and store.  Also the routed form (a row block of 128 has one expert).
#include "pg_lm.cuh"

namespace {

constexpr int FM = 64, FN = 64, FK = 16;

template <int ACT, typename TY>
__global__ void __launch_bounds__(256)
    linear_f32_kernel(const float *__restrict__ a, int64_t lda, const bf16 *__restrict__ w, int M, int N, int K, float limit, TY *__restrict__ y, int64_t ldy,
                      const PgRouted rt)
{
    __shared__ float sa[FK][FM + 4];
    __shared__ float sw[FK][FN + 4];
    pg_pdl_begin();
    const int m0 = blockIdx.x * FM, n0 = blockIdx.y * FN;
    if (rt.blocks) {
        if (m0 >= __ldcg(rt.blocks) * PG_ROUTE_BLOCK) return;
        w += (int64_t)__ldcg(rt.block_expert + m0 / PG_ROUTE_BLOCK) * N * K;
    }
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    const int lr = threadIdx.x >> 2, lk = (threadIdx.x & 3) * 4;   // one row, four k per thread and tile
    float acc[4][4] = {};
    for (int k0 = 0; k0 < K; k0 += FK) {
        float4 va = make_float4(0.f, 0.f, 0.f, 0.f);
        uint2 vw = make_uint2(0u, 0u);
        if (m0 + lr < M) va = __ldcg(reinterpret_cast<const float4 *>(a + (m0 + lr) * lda + k0 + lk));
        if (n0 + lr < N) vw = __ldg(reinterpret_cast<const uint2 *>(w + (int64_t)(n0 + lr) * K + k0 + lk));
        __syncthreads();
        sa[lk][lr] = va.x, sa[lk + 1][lr] = va.y, sa[lk + 2][lr] = va.z, sa[lk + 3][lr] = va.w;
        sw[lk][lr] = pg_bf16_lo(vw.x), sw[lk + 1][lr] = pg_bf16_hi(vw.x), sw[lk + 2][lr] = pg_bf16_lo(vw.y), sw[lk + 3][lr] = pg_bf16_hi(vw.y);
        __syncthreads();
        float sub[4][4] = {};                              // sums of 16 terms meet in acc: shorter chains, smaller error
#pragma unroll
        for (int k = 0; k < FK; k++) {
            float x[4], b[4];
#pragma unroll
            for (int i = 0; i < 4; i++) x[i] = sa[k][ty * 4 + i];
#pragma unroll
            for (int j = 0; j < 4; j++) b[j] = sw[k][ACT == PG_ACT_NONE ? tx * 4 + j : (tx >> 2) * 16 + (tx & 3) * 2 + (j & 1) + (j >> 1) * 8];
#pragma unroll
            for (int i = 0; i < 4; i++)
#pragma unroll
                for (int j = 0; j < 4; j++) sub[i][j] = fmaf(x[i], b[j], sub[i][j]);
        }
#pragma unroll
        for (int i = 0; i < 4; i++)
#pragma unroll
            for (int j = 0; j < 4; j++) acc[i][j] += sub[i][j];
    }
#pragma unroll
    for (int i = 0; i < 4; i++) {
        const int m = m0 + ty * 4 + i;
        if (m >= M) continue;
        if (ACT == PG_ACT_NONE) {
#pragma unroll
            for (int j = 0; j < 4; j++)
                if (n0 + tx * 4 + j < N) pg_put(y + m * ldy + n0 + tx * 4 + j, acc[i][j]);
        } else {
            // this thread's columns: two gates and, eight rows of W further, their ups
#pragma unroll
            for (int j = 0; j < 2; j++) {
                const int n = n0 / 2 + (tx >> 2) * 8 + (tx & 3) * 2 + j;
                if (n < N / 2) pg_put(y + m * ldy + n, pg_glu<ACT>(acc[i][j], acc[i][j + 2], limit));
            }
        }
    }
}

}  // namespace

int32_t pgk_linear_f32(pg_ctx *ctx, const pg_linear *lin, const float *a, int64_t lda, int64_t m, int act, float limit, void *y, int y_dtype, int64_t ldy,
                       const PgRouted *routed)
{
    PG_REQUIRE(y_dtype == PG_F32, "linear: an f32 step has f32 outputs");
    const PgRouted none = {};
    const PgRouted rt = routed ? *routed : none;
    const dim3 grid((unsigned)((m + FM - 1) / FM), (unsigned)((lin->n + FN - 1) / FN));
    PG_REQUIRE(grid.y <= 65535, "linear: too many output columns for the f32 form");
#define PG_F32_CASE(A) \
    return launch_pdl(ctx, linear_f32_kernel<A, float>, grid, dim3(256), 0, a, lda, lin->w, (int)m, (int)lin->n, (int)lin->k, limit, (float *)y, ldy, rt)
    if (act == PG_ACT_NONE) PG_F32_CASE(PG_ACT_NONE);
    if (act == PG_ACT_GELU_TANH_GLU) PG_F32_CASE(PG_ACT_GELU_TANH_GLU);
    PG_F32_CASE(PG_ACT_CLAMPED_SWISH_GLU);
#undef PG_F32_CASE
}
