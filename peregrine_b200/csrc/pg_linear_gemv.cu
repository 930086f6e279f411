// Decode-size product y = a W^T with bf16 operands and f32 sums, for at most 16 rows: one pass over W [N][K].
//
//   * One persistent CTA of 16 warps per SM.  `kw` warps (1 .. 16) share a tile of output columns, each with one part of
//     K of at most 256 elements.  A warp keeps its part of the activations in registers, as MMA fragments, for as long as
//     it works on the same rows: the activations are read once per CTA and never pass through shared memory.
//   * A fill is 8 rows of W: a warp's 8 row segments (up to 512 bytes each) come by bulk asynchronous copies into a private
//     two-slot ring, completion on an mbarrier.  A plain tile is one fill; a tile of a gated product is two, eight gate
//     rows and the eight up rows behind them, whose sums land in the same lanes, so the gate is applied in registers.
//   * Products run on mma.sync m16n8k16 with a permuted K (a lane's 16 contiguous bytes of a weight row and of an
//     activation row feed two MMAs).  The parts of a tile meet in shared memory, added in a fixed order.
//   * K beyond 16 x 256 elements (SPLIT): sp CTAs take the same tiles, each with its part of K, and write their raw sums to
//     slabs of their own; the last of them to finish (a ticket per group) adds the slabs in a fixed order and writes the
//     outputs of all the group's tiles.  Nobody waits for anybody.
//   * ROUTED: the rows come in blocks of 16 that share an expert; the tiles of all blocks form one list, of which a CTA
//     takes a contiguous stretch.
//
// Weights do not depend on the preceding kernel: without a route the ring is filled before griddepcontrol.wait.  Every
// mbarrier wait is bounded; a warp that gave up goes on through the remaining barriers without computing.
#include <algorithm>

#include "pg_async.cuh"
#include "pg_lm.cuh"

namespace {

constexpr int GV_WARPS = 16;
constexpr int GV_THREADS = GV_WARPS * 32;
constexpr int GV_SLOTS = 2;
constexpr int GV_KSTEPS = 8;                              // 32-element steps of one warp's part of K
constexpr int GV_KW_MAX = GV_KSTEPS * 32;
constexpr int GV_STRIDE = GV_KW_MAX * 2 + 64;             // bytes per ring row: 64 mod 128, free of bank conflicts
constexpr int GV_SLOT = 8 * GV_STRIDE;
constexpr int GV_RING = GV_WARPS * GV_SLOTS * GV_SLOT;

// shared memory: ring | partial sums [2][16 warps][32 lanes][4 NT] | barriers
// slabs (SPLIT): [sp][items][32 lanes][4 NT]
template <int ACT, bool HI, bool ROUTED, bool SPLIT, typename TY>
__global__ void __launch_bounds__(GV_THREADS, 1)
    linear_gemv_kernel(const bf16 *__restrict__ a, int64_t lda, int M, const bf16 *__restrict__ w, int N, int K, int kw, int KW, int KH, float limit,
                       TY *__restrict__ y, int64_t ldy, const PgRouted rt, int sp, float *slabs, unsigned int *tickets, int32_t *status,
                       unsigned long long limit_ns)
{
    constexpr int NT = ACT == PG_ACT_NONE ? 1 : 2;
    constexpr int CELL = 4 * NT;                          // floats per lane
    extern __shared__ __align__(128) unsigned char smem[];
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, r = lane >> 2, t = lane & 3;
    const int my_part = SPLIT ? (int)blockIdx.x % sp : 0;
    const int groups = GV_WARPS / kw, slot_idx = warp / kw, kpart = warp - slot_idx * kw;
    float *part = reinterpret_cast<float *>(smem + GV_RING);
    unsigned char *tail = reinterpret_cast<unsigned char *>(part + 2 * GV_WARPS * 32 * CELL);
    const uint32_t bars = pg_smem(tail), my_bar = bars + (uint32_t)warp * (GV_SLOTS * 8);
    volatile int *abort_flag = reinterpret_cast<volatile int *>(tail + GV_WARPS * GV_SLOTS * 8);
    const uint32_t ring = pg_smem(smem) + (uint32_t)warp * (GV_SLOTS * GV_SLOT);
    if (threadIdx.x == 0) {
        for (int i = 0; i < GV_WARPS * GV_SLOTS; i++) pg_mbar_init(bars + 8 * i, 1);
        *abort_flag = 0;
        pg_mbar_fence();
    }
    __syncthreads();

    const int ka0 = my_part * KH;
    const int k0 = ka0 + kpart * KW;
    const int klen = max(0, min(KW, min(K, ka0 + KH) - k0));   // a multiple of 32; 0 only in a short last range
    const int tiles = (N + 8 * NT - 1) / (8 * NT);
    const int64_t unit = SPLIT ? blockIdx.x / sp : blockIdx.x, units = SPLIT ? gridDim.x / sp : gridDim.x;
    if (ROUTED) asm volatile("griddepcontrol.wait;" ::: "memory");
    const int nblk = ROUTED ? __ldcg(rt.blocks) : 1;
    const int64_t items = (int64_t)nblk * tiles, per = (items + units * groups - 1) / (units * groups);
    const int64_t first = (unit * groups + slot_idx) * per;
    const int mine = (int)max((int64_t)0, min(per, items - first));
    const int total = klen > 0 ? mine * NT : 0;

    // fill f: item f / NT, half f % NT
    auto issue = [&](int f) {
        const int64_t it = first + f / NT;
        const int blk = ROUTED ? (int)(it / tiles) : 0, tile = (int)(it - (int64_t)blk * tiles);
        const uint32_t bar = my_bar + (uint32_t)(f % GV_SLOTS) * 8;
        if (lane == 0) pg_mbar_expect(bar, 8u * (uint32_t)klen * 2u);
        __syncwarp();
        if (lane < 8) {
            int64_t n = (int64_t)tile * (8 * NT) + (f % NT) * 8 + lane;
            if (n >= N) n = N - 1;                        // rows past the edge repeat the last one; their sums are dropped
            const int64_t e = ROUTED ? __ldcg(rt.block_expert + blk) : 0;
            pg_bulk_load(ring + (uint32_t)(f % GV_SLOTS) * GV_SLOT + (uint32_t)lane * GV_STRIDE, w + (e * N + n) * K + k0, (uint32_t)klen * 2u, bar);
        }
    };
#pragma unroll
    for (int f = 0; f < GV_SLOTS; f++)
        if (f < total) issue(f);
    if (!ROUTED) asm volatile("griddepcontrol.wait;" ::: "memory");

    // outputs of a tile; lane: rows r and r + 8, columns 2t and 2t + 1
    auto finish = [&](const float (&acc)[NT][4], int blk, int tile) {
#pragma unroll
        for (int h = 0; h < (HI ? 2 : 1); h++) {
            const int m = (ROUTED ? blk * PG_ROUTE_SMALL : 0) + r + 8 * h;
            if (ROUTED ? (__ldcg(rt.row_pair + m) < 0) : (m >= M)) continue;
            const int n = tile * 8 + 2 * t, nmax = N / NT;
            float v0 = acc[0][2 * h], v1 = acc[0][2 * h + 1];
            if (ACT != PG_ACT_NONE) {
                v0 = pg_glu<ACT>(v0, acc[NT - 1][2 * h], limit);
                v1 = pg_glu<ACT>(v1, acc[NT - 1][2 * h + 1], limit);
            }
            if (n < nmax) pg_put(y + m * ldy + n, v0);
            if (n + 1 < nmax) pg_put(y + m * ldy + n + 1, v1);
        }
    };

    uint4 lo[GV_KSTEPS], hi[GV_KSTEPS];
    const int steps = klen >> 5;
    int have = -1;                                        // the row block whose activations the registers hold
    bool ok = true;
    int f = 0;
    for (int j = 0; j < mine; j++) {
        float acc[NT][4];
#pragma unroll
        for (int h = 0; h < NT; h++)
#pragma unroll
            for (int i = 0; i < 4; i++) acc[h][i] = 0.0f;
        const int64_t it = first + j;
        const int blk = ROUTED ? (int)(it / tiles) : 0, tile = (int)(it - (int64_t)blk * tiles);
        if (klen > 0) {
            if (blk != have) {
                have = blk;
                int64_t r0 = r, r1 = r + 8;
                bool v0 = r < M, v1 = HI && r + 8 < M;
                if (ROUTED) {
                    const int p0 = __ldcg(rt.row_pair + blk * PG_ROUTE_SMALL + r), p1 = __ldcg(rt.row_pair + blk * PG_ROUTE_SMALL + r + 8);
                    v0 = p0 >= 0;
                    v1 = HI && p1 >= 0;
                    r0 = rt.by_token ? p0 / rt.top : blk * PG_ROUTE_SMALL + r;
                    r1 = rt.by_token ? p1 / rt.top : blk * PG_ROUTE_SMALL + r + 8;
                }
                const bf16 *a0 = a + r0 * lda + k0 + t * 8, *a1 = a + r1 * lda + k0 + t * 8;
#pragma unroll
                for (int s = 0; s < GV_KSTEPS; s++) {
                    lo[s] = hi[s] = make_uint4(0u, 0u, 0u, 0u);
                    if (s < steps && v0) lo[s] = __ldcg(reinterpret_cast<const uint4 *>(a0 + s * 32));
                    if (HI && s < steps && v1) hi[s] = __ldcg(reinterpret_cast<const uint4 *>(a1 + s * 32));
                }
            }
#pragma unroll
            for (int h = 0; h < NT; h++, f++) {
                ok = ok && pg_mbar_wait(my_bar + (uint32_t)(f % GV_SLOTS) * 8, (uint32_t)(f / GV_SLOTS) & 1u, abort_flag, status, limit_ns);
                ok = __all_sync(0xffffffffu, ok);
                if (ok) {
                    const uint32_t row = ring + (uint32_t)(f % GV_SLOTS) * GV_SLOT + (uint32_t)r * GV_STRIDE + t * 16;
#pragma unroll
                    for (int s = 0; s < GV_KSTEPS; s++) {
                        if (s < steps) {
                            const uint4 b = pg_lds128(row + s * 64);
                            pg_mma_bf16(acc[h], lo[s].x, hi[s].x, lo[s].y, hi[s].y, b.x, b.y);
                            pg_mma_bf16(acc[h], lo[s].z, hi[s].z, lo[s].w, hi[s].w, b.z, b.w);
                        }
                    }
                    __syncwarp();                         // every lane has read the slot
                    if (f + GV_SLOTS < total) issue(f + GV_SLOTS);
                }
            }
        }
        if (kw > 1) {
            float *mine_at = part + ((size_t)((j & 1) * GV_WARPS + warp) * 32 + lane) * CELL;
            if (kpart != 0) {
#pragma unroll
                for (int h = 0; h < NT; h++) reinterpret_cast<float4 *>(mine_at)[h] = make_float4(acc[h][0], acc[h][1], acc[h][2], acc[h][3]);
            }
            asm volatile("bar.sync %0, %1;" ::"r"(1 + slot_idx), "r"(kw * 32) : "memory");
            if (kpart == 0) {
                for (int p = 1; p < kw; p++) {
#pragma unroll
                    for (int h = 0; h < NT; h++) {
                        const float4 v = reinterpret_cast<const float4 *>(mine_at + (size_t)p * 32 * CELL)[h];
                        acc[h][0] += v.x;
                        acc[h][1] += v.y;
                        acc[h][2] += v.z;
                        acc[h][3] += v.w;
                    }
                }
            }
        }
        if (SPLIT) {
            if (kpart == 0) {
                float4 *dst = reinterpret_cast<float4 *>(slabs + (((int64_t)my_part * items + it) * 32 + lane) * CELL);
#pragma unroll
                for (int h = 0; h < NT; h++) dst[h] = make_float4(acc[h][0], acc[h][1], acc[h][2], acc[h][3]);
            }
        } else if (kpart == 0 && ok) {
            finish(acc, blk, tile);
        }
    }
    if (SPLIT) {
        __shared__ int last_in;
        __threadfence();
        __syncthreads();
        if (threadIdx.x == 0) {
            __threadfence();
            last_in = atomicAdd(tickets + unit, 1u) == (unsigned)(sp - 1);
            if (last_in) tickets[unit] = 0;
        }
        __syncthreads();
        if (last_in) {
            __threadfence();
            const int64_t i0 = unit * groups * per, i1 = min(items, i0 + (int64_t)groups * per);
            for (int64_t it = i0 + warp; it < i1; it += GV_WARPS) {
                float acc[NT][4];
#pragma unroll
                for (int h = 0; h < NT; h++)
#pragma unroll
                    for (int i = 0; i < 4; i++) acc[h][i] = 0.0f;
                for (int q = 0; q < sp; q++) {
                    const float4 *src = reinterpret_cast<const float4 *>(slabs + (((int64_t)q * items + it) * 32 + lane) * CELL);
#pragma unroll
                    for (int h = 0; h < NT; h++) {
                        const float4 v = __ldcg(src + h);
                        acc[h][0] += v.x;
                        acc[h][1] += v.y;
                        acc[h][2] += v.z;
                        acc[h][3] += v.w;
                    }
                }
                const int blk = ROUTED ? (int)(it / tiles) : 0;
                finish(acc, blk, (int)(it - (int64_t)blk * tiles));
            }
        }
    }
    if (!ok) {
        // copies that are still in flight get a bounded time to land before the shared memory goes
        const unsigned long long t0 = pg_globaltimer_ns();
        while (pg_globaltimer_ns() - t0 < 2000000ull) {
        }
    }
}


template <int ACT, bool HI, bool ROUTED, bool SPLIT, typename TY>
int32_t gv_launch(pg_ctx *ctx, const pg_linear *lin, const bf16 *a, int64_t lda, int M, int kw, int KW, int KH, int grid, int sp, float limit, TY *y, int64_t ldy,
                  const PgRouted &rt)
{
    constexpr int NT = ACT == PG_ACT_NONE ? 1 : 2;
    auto kern = linear_gemv_kernel<ACT, HI, ROUTED, SPLIT, TY>;
    const int smem = GV_RING + 2 * GV_WARPS * 32 * 4 * NT * 4 + GV_WARPS * GV_SLOTS * 8 + 16;
    static_assert(GV_RING + 2 * GV_WARPS * 32 * 8 * 4 + GV_WARPS * GV_SLOTS * 8 + 16 <= 226 * 1024, "shared memory of the streaming form");
    static std::atomic<uint64_t> smem_set{0};
    PG_CUDA(pg_max_smem_once(kern, 226 * 1024, ctx->device, smem_set));
    unsigned int *tickets = reinterpret_cast<unsigned int *>(ctx->splitk);
    float *slabs = SPLIT ? reinterpret_cast<float *>(reinterpret_cast<unsigned char *>(ctx->splitk) + PG_LM_TICKET_BYTES) : nullptr;
    return launch_pdl(ctx, kern, dim3((unsigned)grid), dim3(GV_THREADS), (size_t)smem, a, lda, M, lin->w, (int)lin->n, (int)lin->k, kw, KW, KH, limit, y, ldy, rt,
                      sp, slabs, tickets, ctx->d_status, ctx->wait_limit_ns);
}

// parts of K that CTAs share
inline int gv_parts(int64_t k) { return (int)((k + GV_WARPS * GV_KW_MAX - 1) / (GV_WARPS * GV_KW_MAX)); }

}  // namespace

size_t pgk_linear_gemv_workspace(int64_t n, int64_t k)
{
    // plain and gated forms alike: 64 floats of slab per eight columns and part
    return gv_parts(k) > 1 ? PG_LM_TICKET_BYTES + (size_t)gv_parts(k) * (size_t)(n + 16) * 64 : 0;
}

bool pgk_linear_gemv_supports(const pg_linear *lin, int64_t m) { return m >= 1 && m <= 16 && gv_parts(lin->k) <= 16 && lin->n < (1 << 30); }

int32_t pgk_linear_gemv(pg_ctx *ctx, const pg_linear *lin, const bf16 *a, int64_t lda, int64_t m, int act, float limit, void *y, int y_dtype, int64_t ldy,
                        const PgRouted *routed, int64_t max_blocks)
{
    const int K = (int)lin->k, nt = act == PG_ACT_NONE ? 1 : 2;
    const int64_t items = ((lin->n + 8 * nt - 1) / (8 * nt)) * (routed ? max_blocks : 1);
    const int sp = gv_parts(K);
    const int KH = sp > 1 ? (int)pg_up((K + sp - 1) / sp, 32) : K;
    const int64_t units = ctx->sm_count / sp;
    if (sp > 1) {
        const int32_t rc = pg_splitk_reserve(ctx, PG_LM_TICKET_BYTES + (size_t)sp * (size_t)items * 32 * 4 * nt * sizeof(float));
        if (rc != PG_OK) return rc;
    }
    // parts of a CTA's K: as few as registers allow, more while every (tile, part) still finds a warp of its own
    int kw = 1;
    while (kw < GV_WARPS && (KH + kw - 1) / kw > GV_KW_MAX) kw *= 2;
    while (kw < GV_WARPS && KH / (kw * 2) >= 64 && items * (kw * 2) <= units * GV_WARPS) kw *= 2;
    const int KW = (int)pg_up((KH + kw - 1) / kw, 32);
    PG_REQUIRE(KW <= GV_KW_MAX, "linear: K part too long");
    const int groups = GV_WARPS / kw;
    const int grid = (int)std::min<int64_t>(units, (items + groups - 1) / groups) * sp;
    static const PgRouted no_route = {};
    const PgRouted &rt = routed ? *routed : no_route;
    const bool hi = m > 8 || routed;
    const int M = (int)m;
#define PG_GV(ACT, HI, RT, SP, TY) return gv_launch<ACT, HI, RT, SP, TY>(ctx, lin, a, lda, M, kw, KW, KH, grid, sp, limit, (TY *)y, ldy, rt)
#define PG_GV_SP(ACT, HI, RT, TY)                 \
    do {                                          \
        if (sp > 1) PG_GV(ACT, HI, RT, true, TY); \
        PG_GV(ACT, HI, RT, false, TY);            \
    } while (0)
#define PG_GV_ACT(ACT, TY)                           \
    do {                                             \
        if (routed) PG_GV_SP(ACT, true, true, TY);   \
        if (hi) PG_GV_SP(ACT, true, false, TY);      \
        PG_GV_SP(ACT, false, false, TY);             \
    } while (0)
    if (act == PG_ACT_GELU_TANH_GLU) PG_GV_ACT(PG_ACT_GELU_TANH_GLU, bf16);
    if (act == PG_ACT_CLAMPED_SWISH_GLU) PG_GV_ACT(PG_ACT_CLAMPED_SWISH_GLU, bf16);
    if (y_dtype == PG_BF16) PG_GV_ACT(PG_ACT_NONE, bf16);
    PG_GV_ACT(PG_ACT_NONE, float);
#undef PG_GV
#undef PG_GV_SP
#undef PG_GV_ACT
}
