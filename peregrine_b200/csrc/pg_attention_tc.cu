// Attention of a prompt's portion on the 5th-generation tensor cores, for key and value widths up to 128 and a power of two
// of query heads per key/value head (csrc/pg_attention.cu has the other shapes, and short portions), and for the keys and
// values that a latent layer unfolds: a key of up to 128 and up to 64 dimensions, the second part shared by all heads.
//
// Widths are filled up to 64 or 128 by the copies, which read zeros behind the true width.
//
// A CTA has 256 rows -- two tiles of 128 (token, head of the group) pairs that share keys and values -- of one sequence and
// key/value head, and walks the keys in tiles of 128:
//   warp 8     TMA: the queries once, then key and value tiles through one ring of five 128-row slots (two where keys have
//              192 columns)
//   warp 9     MMA: S_t = Q_t K^T into TMEM, O_t += P_t V with P_t taken from TMEM.  While one tile's softmax runs, the other
//              tile's products do: after O_t's product comes S_t's of the next keys.
//   warps 0-3, 4-7   softmax of tile 0 and 1: a thread owns a row.  It reads its 128 scores, keeps a running maximum, writes
//              exp2(s - m) as bf16 over the scores' own TMEM columns, and adds them up in f32.  The maximum is only replaced
//              when it falls behind by more than 2^8 -- then the row's sums in TMEM are rescaled -- so that this is rare.
// TMEM: S_0 | S_1 | O_0 | O_1, 128 columns each.  Every mbarrier wait is bounded.
//
// In a chunked layer the key tiles start anew at every chunk, so that none passes the end of the ring; rows whose chunk is
// another one see nothing of a tile.
#include <math.h>

#include "pg_attention.cuh"
#include "pg_tcgen05.cuh"

namespace {

constexpr int TQ = 128, TKEYS = 128;
constexpr int AT_THREADS = 320;
constexpr float LOG2E = 1.4426950408889634f;
constexpr int BLOCK = 128 * 128;                        // bytes of 128 rows x 64 elements

template <int DK, int DV>
struct AtCfg {
    static constexpr int Q_BYTES = (DK / 64) * BLOCK;   // per tile
    static constexpr int SLOT = (DK > DV ? DK : DV) / 64 * BLOCK;
    static constexpr int SLOTS = DK > 128 ? 2 : 5;
    static constexpr int SMEM = 2 * Q_BYTES + SLOTS * SLOT + 1024 + 256;
};

// what the split form has beyond the plain one
struct SplitArgs {
    int seq0, k_blocks;      // 64-column blocks of a key that come from map_k; the others come from map_s
    const float *gate;
    int64_t ldg;
};

// BIAS: a distance bias and / or chunks; SPLIT: AttnSplitKeys
template <int DK, int DV, bool BIAS, bool SPLIT>
__global__ void __launch_bounds__(AT_THREADS, 1)
    attn_prompt_tc_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k, const __grid_constant__ CUtensorMap map_v,
                          const __grid_constant__ CUtensorMap map_s, const AttnShape s, const pg_batch bt, const SplitArgs sp, bf16 *__restrict__ out,
                          int64_t ldo, int32_t *status, unsigned long long limit_ns)
{
    using C = AtCfg<DK, DV>;
    constexpr int SLOTS = C::SLOTS;
    extern __shared__ uint8_t smem_raw[];
    const uint32_t raw = pg_smem(smem_raw), base = (raw + 1023u) & ~1023u;
    uint64_t *bars = reinterpret_cast<uint64_t *>(smem_raw + (base - raw) + 2 * C::Q_BYTES + SLOTS * C::SLOT);
    const uint32_t sq = base, ring = base + 2 * C::Q_BYTES;
    const uint32_t bar_q = pg_smem(bars), bar_full = bar_q + 8, bar_empty = bar_full + 8 * SLOTS, bar_s = bar_empty + 8 * SLOTS, bar_p = bar_s + 16, bar_o = bar_p + 16;
    uint32_t *tmem_slot = reinterpret_cast<uint32_t *>(bars + 1 + 2 * SLOTS + 6);
    volatile int *abort_flag = reinterpret_cast<volatile int *>(tmem_slot + 1);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    if (threadIdx.x == 0) {
        pg_mbar_init(bar_q, 1);
        for (int i = 0; i < SLOTS; i++) {
            pg_mbar_init(bar_full + 8 * i, 1);
            pg_mbar_init(bar_empty + 8 * i, 1);
        }
        for (int i = 0; i < 2; i++) {
            pg_mbar_init(bar_s + 8 * i, 1);
            pg_mbar_init(bar_p + 8 * i, 4);             // one arrival per softmax warp of the tile
            pg_mbar_init(bar_o + 8 * i, 1);
        }
        *abort_flag = 0;
        pg_mbar_fence();
    }
    if (warp == 9) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(pg_smem(tmem_slot)), "r"(512) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = *tmem_slot;
    asm volatile("griddepcontrol.wait;" ::: "memory");

    const int g = blockIdx.y, seq = SPLIT ? sp.seq0 : blockIdx.z;
    const int row0 = __ldcg(bt.d_seq_row0 + seq), T = __ldcg(bt.d_seq_row0 + seq + 1) - row0;
    const int total = T * s.rep, rr0 = (int)(gridDim.x - 1 - blockIdx.x) * 2 * TQ;   // long tiles first
    const int pos0 = T > 0 ? __ldcg(bt.d_pos + row0) : 0;
    const int64_t slot = __ldcg(bt.d_seq_slot + seq);
    // key tiles of the two row tiles (0: no rows, or positions outside the cache, which attn_prep_kernel has recorded)
    const int chunk = BIAS && s.chunk ? s.chunk : 1 << 30, per_chunk = (chunk + TKEYS - 1) / TKEYS;
    const int chunk0 = (pos0 + rr0 / s.rep) / chunk;    // of the first row
    int tiles[2];
#pragma unroll
    for (int t = 0; t < 2; t++) {
        const int first = rr0 + t * TQ, last = min(first + TQ, total) - 1;
        const int pos = pos0 + last / s.rep;
        tiles[t] = first < total && pos < s.limit ? (pos / chunk - chunk0) * per_chunk + pos % chunk / TKEYS + 1 : 0;
    }
    const int most = max(tiles[0], tiles[1]);
    // position of the first key of tile j
    auto key0_of = [&](int j) { return BIAS ? (chunk0 + j / per_chunk) * chunk + j % per_chunk * TKEYS : j * TKEYS; };

    if (warp == 8) {
        // ---------------------------------------------------------------- producer
        if (lane == 0 && most > 0) {
            pg_mbar_expect(bar_q, 2 * C::Q_BYTES);
            for (int t = 0; t < 2; t++)
                for (int b = 0; b < DK / 64; b++)
                    tma_load_3d(sq + t * C::Q_BYTES + b * BLOCK, &map_q, bar_q, b * 64, g * s.rep, row0 + (rr0 + t * TQ) / s.rep);
            const int region = SPLIT ? g : (int)(slot * s.G + g);
            bool ok = true;
            int at = 0, phase = 0;
            for (int j = 0; ok && j < most; j++) {
                const int row = BIAS ? attn_row(s, key0_of(j)) : j * TKEYS;
                for (int kv = 0; kv < 2; kv++) {
                    if (!(ok = pg_mbar_wait(bar_empty + 8 * at, phase ^ 1, abort_flag, status, limit_ns))) break;
                    const int blocks = (kv ? DV : DK) / 64;
                    pg_mbar_expect(bar_full + 8 * at, blocks * BLOCK);
                    for (int b = 0; b < blocks; b++) {
                        if (SPLIT && !kv && b >= sp.k_blocks)
                            tma_load_3d(ring + at * C::SLOT + b * BLOCK, &map_s, bar_full + 8 * at, (b - sp.k_blocks) * 64, row, 0);
                        else
                            tma_load_3d(ring + at * C::SLOT + b * BLOCK, kv ? &map_v : &map_k, bar_full + 8 * at, b * 64, row, region);
                    }
                    if (++at == SLOTS) {
                        at = 0;
                        phase ^= 1;
                    }
                }
            }
            if (!ok) {
                // give copies that are still in flight a bounded time to land before the CTA exits
                const unsigned long long w0 = pg_globaltimer_ns();
                while (pg_globaltimer_ns() - w0 < 2000000ull) {
                }
            }
        }
    } else if (warp == 9) {
        // ---------------------------------------------------------------- MMA issuer (the whole warp; one lane's products count)
        if (most > 0) {
            const uint32_t on = pg_elect();
            constexpr uint32_t idesc_s = make_idesc(TQ, TKEYS), idesc_o = make_idesc(TQ, DV) | IDESC_B_MN_MAJOR;
            int at = 0, phase = 0;
            auto wait = [&](uint32_t bar, uint32_t parity) { return (bool)__all_sync(0xffffffffu, pg_mbar_wait(bar, parity, abort_flag, status, limit_ns)); };
            auto wait_full = [&]() { return wait(bar_full + 8 * at, phase); };
            auto advance = [&]() {
                if (++at == SLOTS) {
                    at = 0;
                    phase ^= 1;
                }
            };
            // (descriptors of other addresses: only the address field, 16 bytes to one, differs)
            const uint64_t desc_q = make_smem_desc(sq), desc_ring = make_smem_desc(ring), desc_v = make_smem_desc_mn(ring, BLOCK);
            auto scores = [&](int t, int k_slot) {
                const uint64_t kt = desc_ring + (uint64_t)(k_slot * (C::SLOT >> 4)), qt = desc_q + (uint64_t)(t * (C::Q_BYTES >> 4));
#pragma unroll
                for (int i = 0; i < DK / 16; i++) {
                    constexpr int block = BLOCK >> 4;
                    const uint64_t off = (uint64_t)((i / 4) * block + (i % 4) * 2);
                    umma_f16(tmem + t * 128, qt + off, kt + off, idesc_s, i != 0, on);
                }
                umma_commit(bar_s + 8 * t, on);
            };
            bool ok = wait(bar_q, 0) && wait_full();
            tc_fence_after();
            if (ok) {
                for (int t = 0; t < 2; t++)
                    if (tiles[t] > 0) scores(t, at);
                umma_commit(bar_empty + 8 * at, on);
                advance();
            }
            for (int j = 0; ok && j < most; j++) {
                if (!(ok = wait_full())) break;         // the values of these keys
                tc_fence_after();
                const int v_slot = at;
                advance();
                bool next = false;                      // the next keys have arrived
                for (int t = 0; ok && t < 2; t++) {
                    if (j >= tiles[t]) continue;
                    if (!(ok = wait(bar_p + 8 * t, j & 1))) break;
                    tc_fence_after();
                    const uint64_t vt = desc_v + (uint64_t)(v_slot * (C::SLOT >> 4));
#pragma unroll
                    for (int i = 0; i < TKEYS / 16; i++)
                        umma_f16_ta(tmem + 256 + t * 128, tmem + t * 128 + i * 8, vt + i * (2048 >> 4), idesc_o, (j | i) != 0, on);
                    if (j + 1 < tiles[t]) {
                        if (!next) {
                            if (!(ok = wait_full())) break;
                            tc_fence_after();
                            next = true;
                        }
                        scores(t, at);
                    } else {
                        umma_commit(bar_o + 8 * t, on);
                    }
                }
                if (!ok) break;
                umma_commit(bar_empty + 8 * v_slot, on);
                if (next) {
                    umma_commit(bar_empty + 8 * at, on);
                    advance();
                }
            }
        }
    } else {
        // ---------------------------------------------------------------- softmax
        const int t = warp >> 2, q = warp & 3;
        const int rr = rr0 + t * TQ + q * 32 + lane, rc = min(rr, total - 1);
        const int lim = pos0 + rc / s.rep;              // last key of this row
        const uint32_t ts = tmem + ((uint32_t)(q * 32) << 16) + t * 128, to = ts + 256;
        const float sl = s.scale * LOG2E, sx = BIAS ? 1.0f : sl;   // (with a bias the scores are scaled before the maximum)
        const float bias = BIAS && s.slopes ? __ldg(s.slopes + g * s.rep + rc % s.rep) * LOG2E : 0.0f;
        float m = 0.0f, l0 = 0.0f, l1 = 0.0f;
        bool ok = true;
        for (int j = 0; j < tiles[t]; j++) {
            ok = pg_mbar_wait(bar_s + 8 * t, j & 1, abort_flag, status, limit_ns);
            ok = __all_sync(0xffffffffu, ok);
            if (!ok) break;
            tc_fence_after();
            uint32_t v[4][32];
#pragma unroll
            for (int c = 0; c < 4; c++) tmem_ld32_async(ts + c * 32, v[c]);
            tmem_wait_ld();
            const int key0 = key0_of(j);
            const int n = !BIAS || key0 / chunk == lim / chunk ? lim - key0 : -1;   // columns behind n are not seen
            if (BIAS) {
                const float b0 = bias * (float)(key0 - lim);
#pragma unroll
                for (int c = 0; c < 4; c++)
#pragma unroll
                    for (int i = 0; i < 32; i++)
                        v[c][i] = __float_as_uint(fmaf(__uint_as_float(v[c][i]), sl, fmaf(bias, (float)(c * 32 + i), b0)));
            }
            if (__any_sync(0xffffffffu, n < TKEYS - 1)) {
#pragma unroll
                for (int c = 0; c < 4; c++)
#pragma unroll
                    for (int i = 0; i < 32; i++)
                        if (c * 32 + i > n) v[c][i] = 0xff800000u;   // -inf
            }
            float mx[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
            for (int c = 0; c < 4; c++)
#pragma unroll
                for (int i = 0; i < 32; i++) mx[i & 3] = fmaxf(mx[i & 3], __uint_as_float(v[c][i]));
            const float top = fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3])) * sx;
            if (j == 0) {
                m = fmaxf(top, s.sink ? 0.0f : -1e30f); // (finite also where the row sees nothing of the first tile)
            } else {
                const bool behind = top > m + 8.0f;
                if (__any_sync(0xffffffffu, behind)) {
                    // (these scores were committed behind the previous keys' sums: O is at rest)
                    const float f = behind ? pg_ex2(m - top) : 1.0f;
                    if (behind) m = top;
                    l0 *= f;
                    l1 *= f;
#pragma unroll 1
                    for (int c = 0; c < DV; c += 32) {
                        uint32_t o[32];
                        tmem_ld32(to + c, o);
#pragma unroll
                        for (int i = 0; i < 32; i++) o[i] = __float_as_uint(__uint_as_float(o[i]) * f);
                        tmem_st32(to + c, o);
                    }
                    tmem_wait_st();
                }
            }
#pragma unroll
            for (int h = 0; h < 2; h++) {
                uint32_t p[32];
#pragma unroll
                for (int i = 0; i < 32; i++) {
                    const int c = h * 2 + (i >> 4), e = (i & 15) * 2;
                    const float a = pg_ex2(fmaf(__uint_as_float(v[c][e]), sx, -m)), b = pg_ex2(fmaf(__uint_as_float(v[c][e + 1]), sx, -m));
                    l0 += a;
                    l1 += b;
                    p[i] = pg_pack_bf16(a, b);
                }
                tmem_st32(ts + h * 32, p);
            }
            tmem_wait_st();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) pg_mbar_arrive(bar_p + 8 * t);
        }
        if (ok && tiles[t] > 0) {
            ok = pg_mbar_wait(bar_o + 8 * t, 0, abort_flag, status, limit_ns);
            ok = __all_sync(0xffffffffu, ok);
            tc_fence_after();
            float l = l0 + l1;
            if (s.sink) l += pg_ex2(-m);
            const float inv = __fdiv_rn(1.0f, l);
            const int head_at = (g * s.rep + rc % s.rep) * s.V;
            bf16 *dst = out + (int64_t)(row0 + rc / s.rep) * ldo + head_at;
            const float *gate = SPLIT ? sp.gate + (int64_t)(row0 + rc / s.rep) * sp.ldg + head_at : nullptr;
            const bool whole = s.V % 8 == 0;            // (and so is ldo: rows of eight columns start on 16-byte boundaries)
#pragma unroll 1
            for (int c = 0; c < DV; c += 32) {
                uint32_t o[32];
                tmem_ld32(to + c, o);
                if (!ok || rr >= total) continue;
#pragma unroll
                for (int i = 0; i < 32; i++) {
                    float y = __uint_as_float(o[i]) * inv;
                    if (SPLIT && c + i < s.V) y *= pg_sigmoid(__ldcg(gate + c + i));
                    o[i] = __float_as_uint(y);
                }
                if (!whole) {
#pragma unroll
                    for (int i = 0; i < 32; i++)
                        if (c + i < s.V) pg_put(dst + c + i, __uint_as_float(o[i]));
                    continue;
                }
#pragma unroll
                for (int i = 0; i < 32; i += 8) {
                    if (c + i >= s.V) break;
                    uint4 w;
                    w.x = pg_pack_bf16(__uint_as_float(o[i]), __uint_as_float(o[i + 1]));
                    w.y = pg_pack_bf16(__uint_as_float(o[i + 2]), __uint_as_float(o[i + 3]));
                    w.z = pg_pack_bf16(__uint_as_float(o[i + 4]), __uint_as_float(o[i + 5]));
                    w.w = pg_pack_bf16(__uint_as_float(o[i + 6]), __uint_as_float(o[i + 7]));
                    *reinterpret_cast<uint4 *>(dst + c + i) = w;
                }
            }
        }
    }
    __syncwarp();
    tc_fence_before();
    __syncthreads();
    if (warp == 9) {
        tc_fence_after();
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(512) : "memory");
    }
}

// [z][y][x], x up to `cols`, rows `ldy` and z parts `ldz` elements apart
int32_t map3(CUtensorMap *map, const bf16 *p, int64_t cols, int64_t rows, int64_t ldy, int64_t parts, int64_t ldz, int box_rows, int box_parts)
{
    const cuuint64_t dims[3] = {(cuuint64_t)cols, (cuuint64_t)rows, (cuuint64_t)parts}, strides[2] = {(cuuint64_t)ldy * 2, (cuuint64_t)ldz * 2};
    const cuuint32_t box[3] = {64, (cuuint32_t)box_rows, (cuuint32_t)box_parts};
    return pg_encode_bf16(map, p, 3, dims, strides, box);
}

template <int DK, int DV, bool BIAS, bool SPLIT>
int32_t launch(pg_ctx *ctx, const CUtensorMap (&maps)[4], const AttnShape &s, const pg_batch *bt, const SplitArgs &sp, int64_t len, int64_t seqs, bf16 *out,
               int64_t ldo)
{
    using C = AtCfg<DK, DV>;
    auto kern = attn_prompt_tc_kernel<DK, DV, BIAS, SPLIT>;
    static std::atomic<uint64_t> set{0};
    PG_CUDA(pg_max_smem_once(kern, C::SMEM, ctx->device, set));
    const int64_t tiles = (len * s.rep + 2 * TQ - 1) / (2 * TQ);
    return launch_pdl(ctx, kern, dim3((unsigned)tiles, (unsigned)s.G, (unsigned)seqs), dim3(AT_THREADS), (size_t)C::SMEM, maps[0], maps[1], maps[2], maps[3], s, *bt,
                      sp, out, ldo, ctx->d_status, ctx->wait_limit_ns);
}

template <int DK, int DV>
int32_t run(pg_ctx *ctx, const AttnShape &s, const pg_batch *bt, int64_t slots, const bf16 *q, const bf16 *kc, const bf16 *vc, bf16 *out, int64_t ldo)
{
    CUtensorMap maps[4];
    const int64_t regions = slots * s.G;
    int32_t rc = map3(&maps[0], q, s.dp, s.H, s.dp, bt->rows, (int64_t)s.H * s.dp, s.rep, TQ / s.rep);
    if (rc == PG_OK) rc = map3(&maps[1], kc, s.dp, s.cap, s.dp, regions, (int64_t)s.cap * s.dp, TKEYS, 1);
    if (rc == PG_OK) rc = map3(&maps[2], vc, s.vp, s.cap, s.vp, regions, (int64_t)s.cap * s.vp, TKEYS, 1);
    if (rc != PG_OK) return rc;
    maps[3] = maps[2];
    const SplitArgs none = {};
    if (s.slopes || s.chunk) return launch<DK, DV, true, false>(ctx, maps, s, bt, none, bt->max_len, bt->seqs, out, ldo);
    return launch<DK, DV, false, false>(ctx, maps, s, bt, none, bt->max_len, bt->seqs, out, ldo);
}

template <int DK, int DV>
int32_t run_split(pg_ctx *ctx, const AttnShape &s, const pg_batch *bt, const AttnSplitKeys &k, bf16 *out, int64_t ldo)
{
    CUtensorMap maps[4];
    // (a sequence's rows lie next to each other: the tile behind its last one reads other rows, whose results are dropped)
    int32_t rc = map3(&maps[0], k.q, k.qd, s.H, k.qd, bt->rows, (int64_t)s.H * k.qd, 1, TQ);
    if (rc == PG_OK) rc = map3(&maps[1], k.k, k.kd, k.positions, k.ldk, s.H, k.kd, TKEYS, 1);
    if (rc == PG_OK) rc = map3(&maps[2], k.v, k.vd, k.positions, k.ldk, s.H, k.vd, TKEYS, 1);
    if (rc == PG_OK) rc = map3(&maps[3], k.shared, k.sd, k.positions, k.lds, 1, k.positions * k.lds, TKEYS, 1);
    if (rc != PG_OK) return rc;
    const SplitArgs sp = {k.seq, (k.kd + 63) / 64, k.gate, k.ldg};
    return launch<DK, DV, false, true>(ctx, maps, s, bt, sp, k.len, 1, out, ldo);
}

}  // namespace

bool pgk_attention_prompt_tc_supports(const AttnShape &s, const pg_batch *bt, int64_t slots, int64_t ldo, const void *out)
{
    return s.D <= 128 && s.V <= 128 && s.rep <= 128 && (s.rep & (s.rep - 1)) == 0 && s.scale > 0.0f && slots > 0 && ldo % 8 == 0 &&
           ((uintptr_t)out & 15) == 0 && (int64_t)bt->max_len * s.rep >= TQ;
}

int32_t pgk_attention_prompt_tc(pg_ctx *ctx, const AttnShape &s, const pg_batch *bt, int64_t slots, const bf16 *q, const bf16 *kc, const bf16 *vc, bf16 *out,
                                int64_t ldo)
{
    if (s.D > 64 && s.V > 64) return run<128, 128>(ctx, s, bt, slots, q, kc, vc, out, ldo);
    if (s.D > 64) return run<128, 64>(ctx, s, bt, slots, q, kc, vc, out, ldo);
    if (s.V > 64) return run<64, 128>(ctx, s, bt, slots, q, kc, vc, out, ldo);
    return run<64, 64>(ctx, s, bt, slots, q, kc, vc, out, ldo);
}

bool pgk_attention_split_supports(int kd, int sd, int V) { return kd <= 128 && sd <= 64 && V <= 128; }

int32_t pgk_attention_split_tc(pg_ctx *ctx, const AttnShape &s, const pg_batch *bt, const AttnSplitKeys &k, bf16 *out, int64_t ldo)
{
    PG_REQUIRE(pgk_attention_split_supports(k.kd, k.sd, s.V) && s.scale > 0.0f && s.rep == 1 && !s.chunk && !s.slopes && ldo % 8 == 0 &&
                   ((uintptr_t)out & 15) == 0,
               "attention: unfolded keys that the tensor-core form does not take");
    // one block of 64 for the shared part behind one or two of the head's own
    if (k.kd > 64) return s.V > 64 ? run_split<192, 128>(ctx, s, bt, k, out, ldo) : run_split<192, 64>(ctx, s, bt, k, out, ldo);
    return s.V > 64 ? run_split<128, 128>(ctx, s, bt, k, out, ldo) : run_split<128, 64>(ctx, s, bt, k, out, ldo);
}
