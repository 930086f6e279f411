// Prefill-size product y = a W^T, bf16 operands and f32 sums, on the 5th-generation tensor cores: the structure of
// gemm_i8_tcgen05_kernel (one persistent CTA per SM; TMA producer warp, one issuing lane, four epilogue warps, two TMEM
// accumulators) for kind::f16, with three more things in it:
//
//   * gated products: W's rows alternate eight gate / eight up rows, so a lane's 32 accumulator columns hold complete
//     pairs and the epilogue writes the gated bf16 activations (half the columns, a quarter of the bytes of the raw sums);
//   * products with fewer tiles than SMs: K is divided over `sp` CTAs.  Each writes its raw sums to a slab; the last warp of a
//     32-row band to finish (a ticket per band) adds the slabs in a fixed order and writes the outputs.  Nobody waits;
//   * routed products: an A tile of 128 rows belongs to one expert, whose weights start at row expert * N of the
//     stacked [experts * N][K] matrix.  Number and experts of the tiles are read on the device.
//
// Every mbarrier wait is bounded (pg_async.cuh).
#include <algorithm>

#include "pg_async.cuh"
#include "pg_lm.cuh"
#include "pg_tc_epilogue.cuh"
#include "pg_tcgen05.cuh"

namespace {

constexpr int BM = 128;
constexpr int BK = 64;                 // elements of K per stage = one 128-byte swizzle span
constexpr int BKB = BK * 2;
constexpr int UMMA_KB = 32;            // bytes of K per instruction
constexpr int TC_THREADS = 192;

template <int BN>
struct Cfg {
    static constexpr int STAGE_A = BM * BKB;
    static constexpr int STAGE_B = BN * BKB;
    static constexpr int STAGE = STAGE_A + STAGE_B;
    static constexpr int ROOM = 232448 - (1024 + 256 + 4 * PG_EPI_WARP_BYTES);
    static constexpr int STAGES = ROOM / STAGE > 10 ? 10 : ROOM / STAGE;
    static constexpr int TMEM_COLS = (2 * BN < 32) ? 32 : 2 * BN;
    static constexpr size_t SMEM = (size_t)STAGES * STAGE + 1024 + 256 + 4 * PG_EPI_WARP_BYTES;
};

// How K is divided: parts of `blocks` 64-element blocks; slab of (unit, quarter): [BN][32 rows]
struct KParts {
    int parts, blocks;
    float *slabs;
    unsigned int *tickets;   // one per (tile, quarter), zero between calls
};

// Writes a lane's row of a block of 32 accumulator columns; n0: first column, N: columns of the product.
template <int ACT, typename TY>
__device__ __forceinline__ void store_row(TY *y, int64_t ldy, int row, int n0, int N, const uint32_t (&v)[32], float limit)
{
    if constexpr (ACT != PG_ACT_NONE) {
        // columns n0 .. n0 + 31 = [8 gates | 8 ups] twice; N is a multiple of 16
        bf16 *dst = reinterpret_cast<bf16 *>(y) + (int64_t)row * ldy + n0 / 2;
#pragma unroll
        for (int h = 0; h < 2; h++) {
            if (n0 + 16 * h >= N) break;
            uint32_t o[4];
#pragma unroll
            for (int i = 0; i < 4; i++)
                o[i] = pg_pack_bf16(pg_glu<ACT>(__uint_as_float(v[16 * h + 2 * i]), __uint_as_float(v[16 * h + 8 + 2 * i]), limit),
                                    pg_glu<ACT>(__uint_as_float(v[16 * h + 2 * i + 1]), __uint_as_float(v[16 * h + 9 + 2 * i]), limit));
            *reinterpret_cast<uint4 *>(dst + 8 * h) = make_uint4(o[0], o[1], o[2], o[3]);
        }
    } else if constexpr (sizeof(TY) == 2) {
        bf16 *dst = reinterpret_cast<bf16 *>(y) + (int64_t)row * ldy + n0;
#pragma unroll
        for (int h = 0; h < 4; h++) {
            if (n0 + 8 * h + 8 <= N) {
                uint32_t o[4];
#pragma unroll
                for (int i = 0; i < 4; i++) o[i] = pg_pack_bf16(__uint_as_float(v[8 * h + 2 * i]), __uint_as_float(v[8 * h + 2 * i + 1]));
                *reinterpret_cast<uint4 *>(dst + 8 * h) = make_uint4(o[0], o[1], o[2], o[3]);
            } else {
#pragma unroll
                for (int i = 0; i < 8; i++)
                    if (n0 + 8 * h + i < N) pg_put(dst + 8 * h + i, __uint_as_float(v[8 * h + i]));
            }
        }
    } else {
        float *dst = reinterpret_cast<float *>(y) + (int64_t)row * ldy + n0;
#pragma unroll
        for (int j = 0; j < 32; j++)
            if (n0 + j < N) dst[j] = __uint_as_float(v[j]);
    }
}

template <int BN, int ACT, typename TY>
__global__ void __launch_bounds__(TC_THREADS, 1)
    linear_tc_kernel(const __grid_constant__ CUtensorMap tmap_a, const __grid_constant__ CUtensorMap tmap_b, int M, int N, int K, float limit,
                     TY *__restrict__ y, int64_t ldy, const PgRouted rt, const KParts kp, int32_t *status, unsigned long long limit_ns)
{
    using C = Cfg<BN>;
    constexpr int STAGES = C::STAGES;
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    extern __shared__ uint8_t smem_raw[];
    const uint32_t raw_addr = pg_smem(smem_raw);
    const uint32_t base = (raw_addr + 1023u) & ~1023u;
    uint8_t *smem = smem_raw + (base - raw_addr);
    uint64_t *bars = reinterpret_cast<uint64_t *>(smem + (size_t)STAGES * C::STAGE);
    const uint32_t bar_full = pg_smem(bars);
    const uint32_t bar_empty = bar_full + 8 * STAGES;
    const uint32_t bar_tfull = bar_empty + 8 * STAGES;
    const uint32_t bar_tempty = bar_tfull + 16;
    uint32_t *tmem_slot = reinterpret_cast<uint32_t *>(bars + 2 * STAGES + 4);
    volatile int *abort_flag = reinterpret_cast<volatile int *>(tmem_slot + 1);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;

    if (threadIdx.x == 0) {
        for (int s = 0; s < STAGES; s++) {
            pg_mbar_init(bar_full + 8 * s, 1);
            pg_mbar_init(bar_empty + 8 * s, 1);
        }
        for (int i = 0; i < 2; i++) {
            pg_mbar_init(bar_tfull + 8 * i, 1);
            pg_mbar_init(bar_tempty + 8 * i, 4);   // one arrival per epilogue warp
        }
        *abort_flag = 0;
        pg_mbar_fence();
    }
    if (warp == 1) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(pg_smem(tmem_slot)), "r"(C::TMEM_COLS) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem_base = *tmem_slot;
    const bool routed = rt.blocks != nullptr;
    if (routed) asm volatile("griddepcontrol.wait;" ::: "memory");   // the list of tiles comes from the preceding kernels
    const int tiles_m = routed ? __ldcg(rt.blocks) : (M + BM - 1) / BM;
    const int tiles_n = (N + BN - 1) / BN;
    const int sp = kp.parts, total = tiles_m * tiles_n * sp;   // unit u: part u % sp of tile u / sp
    const int kblocks = K / BK;
    auto k_first = [&](int u) { return (u % sp) * kp.blocks; };
    auto k_end = [&](int u) { return min(kblocks, (u % sp + 1) * kp.blocks); };
    const int rows = routed ? tiles_m * BM : M;

    if (warp == 0) {
        // ---------------------------------------------------------------- producer
        if (lane == 0) {
            uint32_t stage = 0, phase = 0;
            bool ok = true;
            // without a route the weight tiles of the first stages are requested before the predecessor has finished
            int early = 0;
            if (!routed) {
                if ((int)blockIdx.x < total) {
                    const int n0 = ((int)blockIdx.x / sp / tiles_m) * BN, first = k_first(blockIdx.x);
                    early = min(k_end(blockIdx.x) - first, STAGES);
                    for (int i = 0; i < early; i++) {
                        pg_mbar_expect(bar_full + 8 * i, C::STAGE);
                        tma_load_2d(base + i * C::STAGE + C::STAGE_A, &tmap_b, bar_full + 8 * i, (first + i) * BK, n0);
                    }
                }
                asm volatile("griddepcontrol.wait;" ::: "memory");
            }
            for (int u = blockIdx.x; ok && u < total; u += gridDim.x) {
                const int tile = u / sp;
                const int m0 = (tile % tiles_m) * BM;
                const int n0 = (tile / tiles_m) * BN;
                const int b0 = routed ? __ldcg(rt.block_expert + tile % tiles_m) * N + n0 : n0;
                for (int kb = k_first(u), end = k_end(u); kb < end; kb++) {
                    if (!(ok = pg_mbar_wait(bar_empty + 8 * stage, phase ^ 1, abort_flag, status, limit_ns))) break;
                    const uint32_t sa = base + stage * C::STAGE;
                    if (early > 0) {
                        early--;                            // announced and half filled above
                    } else {
                        pg_mbar_expect(bar_full + 8 * stage, C::STAGE);
                        tma_load_2d(sa + C::STAGE_A, &tmap_b, bar_full + 8 * stage, kb * BK, b0);
                    }
                    tma_load_2d(sa, &tmap_a, bar_full + 8 * stage, kb * BK, m0);
                    if (++stage == STAGES) {
                        stage = 0;
                        phase ^= 1;
                    }
                }
            }
            if (!ok) {
                // give copies that are still in flight a bounded time to land before the CTA exits
                const unsigned long long t0 = pg_globaltimer_ns();
                while (pg_globaltimer_ns() - t0 < 2000000ull) {
                }
            }
        }
    } else if (warp == 1) {
        // ---------------------------------------------------------------- MMA issuer (the whole warp; one lane's products count)
        {
            const uint32_t on = pg_elect();
            constexpr uint32_t idesc = make_idesc(BM, BN);
            uint32_t stage = 0, phase = 0, acc = 0, acc_phase = 0;
            bool ok = true;
            for (int u = blockIdx.x; ok && u < total; u += gridDim.x) {
                if (!(ok = __all_sync(0xffffffffu, pg_mbar_wait(bar_tempty + 8 * acc, acc_phase ^ 1, abort_flag, status, limit_ns)))) break;
                tc_fence_after();
                const uint32_t d_tmem = tmem_base + acc * BN;
                const int first = k_first(u), end = k_end(u);
                for (int kb = first; kb < end; kb++) {
                    if (!(ok = __all_sync(0xffffffffu, pg_mbar_wait(bar_full + 8 * stage, phase, abort_flag, status, limit_ns)))) break;
                    tc_fence_after();
                    const uint32_t sa = base + stage * C::STAGE;
                    const uint64_t da = make_smem_desc(sa), db = make_smem_desc(sa + C::STAGE_A);
#pragma unroll
                    for (int j = 0; j < BKB / UMMA_KB; j++)
                        umma_f16(d_tmem, da + (uint64_t)(j * (UMMA_KB >> 4)), db + (uint64_t)(j * (UMMA_KB >> 4)), idesc, kb != first || j != 0 ? 1u : 0u, on);
                    umma_commit(bar_empty + 8 * stage, on);   // stage reusable once these MMAs have read it
                    if (++stage == STAGES) {
                        stage = 0;
                        phase ^= 1;
                    }
                }
                if (!ok) break;
                umma_commit(bar_tfull + 8 * acc, on);         // accumulator complete
                if (++acc == 2) {
                    acc = 0;
                    acc_phase ^= 1;
                }
            }
        }
    } else {
        // ---------------------------------------------------------------- epilogue
        const int q = warp & 3;                           // TMEM lane quarter this warp may read
        if (!routed) asm volatile("griddepcontrol.wait;" ::: "memory");   // y may still be read by the predecessor
        uint32_t acc = 0, acc_phase = 0;
        const bool vec_ok = ACT == PG_ACT_NONE && sizeof(TY) == 4 && ((N & 3) == 0) && ((ldy & 3) == 0) && (((uintptr_t)y & 15) == 0);
        bool ok = true;
        for (int u = blockIdx.x; ok && u < total; u += gridDim.x) {
            const int tile = u / sp;
            const int m0 = (tile % tiles_m) * BM;
            const int n0 = (tile / tiles_m) * BN;
            ok = pg_mbar_wait(bar_tfull + 8 * acc, acc_phase, abort_flag, status, limit_ns);
            ok = __all_sync(0xffffffffu, ok);
            if (!ok) break;
            tc_fence_after();
            const int row_base = m0 + q * 32, row = row_base + lane;
            const uint32_t taddr = tmem_base + ((uint32_t)(q * 32) << 16) + acc * BN;
            const uint32_t stage_buf = base + (uint32_t)((size_t)STAGES * C::STAGE) + 256u + (uint32_t)q * PG_EPI_WARP_BYTES;
            auto put = [&](const uint32_t (&v)[32], int c) {
                if (vec_ok)
                    pg_store_block_32x32(reinterpret_cast<uint32_t *>(y) + (int64_t)row_base * ldy + n0 + c, ldy, rows - row_base, N - (n0 + c), stage_buf,
                                         lane, v);
                else if (row < rows)
                    store_row<ACT, TY>(y, ldy, row, n0 + c, N, v, limit);
            };
#pragma unroll 1
            for (int c = 0; c < BN; c += 32) {
                if (row_base >= rows || n0 + c >= N) break;   // uniform over the warp
                uint32_t v[32];
                tmem_ld32(taddr + c, v);
                if (sp > 1) {
                    float *slab = kp.slabs + (((int64_t)u * 4 + q) * BN + c) * 32 + lane;
#pragma unroll
                    for (int j = 0; j < 32; j++) __stcg(slab + j * 32, __uint_as_float(v[j]));
                } else {
                    put(v, c);
                }
            }
            tc_fence_before();
            __syncwarp();
            if (lane == 0) pg_mbar_arrive(bar_tempty + 8 * acc);
            if (sp > 1 && row_base < rows) {
                unsigned int *ticket = kp.tickets + tile * 4 + q;
                __threadfence();
                __syncwarp();
                const unsigned int before = __shfl_sync(0xffffffffu, lane == 0 ? atomicAdd(ticket, 1u) : 0u, 0);
                if (before == (unsigned)(sp - 1)) {
                    __threadfence();
                    if (lane == 0) *ticket = 0;
#pragma unroll 1
                    for (int c = 0; c < BN; c += 32) {
                        if (n0 + c >= N) break;
                        const float *slab = kp.slabs + (((int64_t)tile * sp * 4 + q) * BN + c) * 32 + lane;
                        float sum[32];
#pragma unroll
                        for (int j = 0; j < 32; j++) sum[j] = __ldcg(slab + j * 32);
                        for (int p = 1; p < sp; p += 2) {  // (two slabs at a time: twice the loads in flight)
                            const float *at = slab + (int64_t)p * 4 * BN * 32, *at2 = at + (p + 1 < sp ? (int64_t)4 * BN * 32 : 0);
                            const float on = p + 1 < sp ? 1.0f : 0.0f;
                            float a[32], b[32];
#pragma unroll
                            for (int j = 0; j < 32; j++) a[j] = __ldcg(at + j * 32);
#pragma unroll
                            for (int j = 0; j < 32; j++) b[j] = __ldcg(at2 + j * 32);
#pragma unroll
                            for (int j = 0; j < 32; j++) sum[j] = fmaf(on, b[j], sum[j] + a[j]);
                        }
                        uint32_t v[32];
#pragma unroll
                        for (int j = 0; j < 32; j++) v[j] = __float_as_uint(sum[j]);
                        put(v, c);
                    }
                }
            }
            if (++acc == 2) {
                acc = 0;
                acc_phase ^= 1;
            }
        }
    }

    __syncwarp();
    tc_fence_before();
    __syncthreads();
    if (warp == 1) {
        tc_fence_after();
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_base), "r"(C::TMEM_COLS) : "memory");
    }
}

// ---------------------------------------------------------------- host side ----
// [rows, k] bf16, rows ld elements apart; box = 64 elements of K x box_rows rows
int32_t encode_kmajor(CUtensorMap *map, const void *ptr, int64_t rows, int64_t k, int64_t ld, int box_rows)
{
    const cuuint64_t dims[2] = {(cuuint64_t)k, (cuuint64_t)rows}, strides[1] = {(cuuint64_t)ld * 2};
    const cuuint32_t box[2] = {(cuuint32_t)BK, (cuuint32_t)box_rows};
    return pg_encode_bf16(map, ptr, 2, dims, strides, box);
}

template <int BN, int ACT, typename TY>
int32_t launch(pg_ctx *ctx, pg_linear *lin, const bf16 *a, int64_t lda, int64_t m, float limit, TY *y, int64_t ldy, const PgRouted &rt,
               KParts kp)
{
    using C = Cfg<BN>;
    CUtensorMap ta;
    int32_t rc = encode_kmajor(&ta, a, m, lin->k, lda, BM);
    if (rc) return rc;
    const int at = BN == 128 || BN == 32 ? 0 : 1;
    if (lin->tmap_rows[at] != BN) {
        rc = encode_kmajor(reinterpret_cast<CUtensorMap *>(lin->tmap[at]), lin->w, lin->experts * lin->n, lin->k, lin->k, BN);
        if (rc) return rc;
        lin->tmap_rows[at] = BN;
    }
    auto kern = linear_tc_kernel<BN, ACT, TY>;
    static std::atomic<uint64_t> smem_set{0};
    PG_CUDA(pg_max_smem_once(kern, (int)C::SMEM, ctx->device, smem_set));
    const int64_t tiles = ((m + BM - 1) / BM) * ((lin->n + BN - 1) / BN) * kp.parts;
    kp.tickets = reinterpret_cast<unsigned int *>(ctx->splitk);
    kp.slabs = reinterpret_cast<float *>(reinterpret_cast<unsigned char *>(ctx->splitk) + PG_LM_TICKET_BYTES);
    return launch_pdl(ctx, kern, dim3((unsigned)std::min<int64_t>(tiles, ctx->sm_count)), dim3(TC_THREADS), C::SMEM, ta,
                      *reinterpret_cast<CUtensorMap *>(lin->tmap[at]), (int)m, (int)lin->n, (int)lin->k, limit, y, ldy, rt, kp, ctx->d_status,
                      ctx->wait_limit_ns);
}

template <int ACT, typename TY>
int32_t dispatch(pg_ctx *ctx, pg_linear *lin, const bf16 *a, int64_t lda, int64_t m, float limit, TY *y, int64_t ldy, const PgRouted &rt)
{
    // the widest tile that still gives every SM one
    const int64_t tiles_m = (m + BM - 1) / BM;
    auto tiles = [&](int w) { return tiles_m * ((lin->n + w - 1) / w); };
    int bn = 32;
    for (int cand = 64; cand <= 256; cand *= 2)
        if (tiles(cand) >= ctx->sm_count) bn = cand;
    const int kblocks = (int)(lin->k / BK);
    KParts kp = {1, kblocks, nullptr, nullptr};
    if (bn < 128 && rt.blocks == nullptr) {
        // narrow tiles read the rows of a over and over: K in parts of at least four blocks instead, if that fills the GPU too
        // -- the widest tile that does, else the one with the most parts in all
        int64_t best = std::min<int64_t>(tiles(bn), ctx->sm_count);
        for (int cand = lin->n > 64 ? 128 : lin->n > 32 ? 64 : 32; cand >= 32; cand /= 2) {
            const int64_t most = std::min<int64_t>({ctx->sm_count / std::max<int64_t>(1, tiles(cand)), kblocks / 4, 16});
            if (most < 2 || (tiles(cand) * most < ctx->sm_count * 3 / 4 && tiles(cand) * most <= best)) continue;
            best = tiles(cand) * most;
            bn = cand;
            kp.blocks = (kblocks + (int)most - 1) / (int)most;
            kp.parts = (kblocks + kp.blocks - 1) / kp.blocks;
            if (best >= ctx->sm_count * 3 / 4) break;
        }
        const size_t need = PG_LM_TICKET_BYTES + (size_t)tiles(bn) * kp.parts * BM * bn * sizeof(float);
        if (kp.parts > 1 && need > ctx->splitk_bytes) {
            const int32_t rc = pg_splitk_reserve(ctx, need);
            if (rc != PG_OK) return rc;
        }
    }
    if (bn == 256) return launch<256, ACT, TY>(ctx, lin, a, lda, m, limit, y, ldy, rt, kp);
    if (bn == 128) return launch<128, ACT, TY>(ctx, lin, a, lda, m, limit, y, ldy, rt, kp);
    if (bn == 64) return launch<64, ACT, TY>(ctx, lin, a, lda, m, limit, y, ldy, rt, kp);
    return launch<32, ACT, TY>(ctx, lin, a, lda, m, limit, y, ldy, rt, kp);
}

}  // namespace

int32_t pgk_linear_tc(pg_ctx *ctx, pg_linear *lin, const bf16 *a, int64_t lda, int64_t m, int act, float limit, void *y, int y_dtype, int64_t ldy,
                      const PgRouted *routed)
{
    static const PgRouted no_route = {};
    const PgRouted &rt = routed ? *routed : no_route;
    PG_REQUIRE(m < (1ll << 31) - 256 && lin->experts * lin->n < (1ll << 31) - 256, "linear: too many rows");
    PG_REQUIRE(act == PG_ACT_NONE || lin->n % 16 == 0, "linear: a gated product has a multiple of 16 columns");
    PG_REQUIRE(y_dtype == PG_F32 || (ldy % 8 == 0 && ((uintptr_t)y & 15) == 0), "linear: bf16 output rows start on 16-byte boundaries");
    if (act == PG_ACT_GELU_TANH_GLU) return dispatch<PG_ACT_GELU_TANH_GLU, bf16>(ctx, lin, a, lda, m, limit, (bf16 *)y, ldy, rt);
    if (act == PG_ACT_CLAMPED_SWISH_GLU) return dispatch<PG_ACT_CLAMPED_SWISH_GLU, bf16>(ctx, lin, a, lda, m, limit, (bf16 *)y, ldy, rt);
    if (y_dtype == PG_BF16) return dispatch<PG_ACT_NONE, bf16>(ctx, lin, a, lda, m, limit, (bf16 *)y, ldy, rt);
    return dispatch<PG_ACT_NONE, float>(ctx, lin, a, lda, m, limit, (float *)y, ldy, rt);
}
