// Latent attention: a position is cached as one latent c (kv_rank numbers, normalised) and one rotated key part that all heads
// share.  A head's key is [W_uk c | rotated part], its value W_uv c.
//
// Short portions never unfold the cache.  With q' = W_uk^T q the score is q' . c + q_rot . k_rot and the head's output is
// W_uv (sum p c): attention of all heads over one key of kv_rank + rot_dim, whose first kv_rank columns are the value.
//
//   bf16, short      latent_query_kernel   q' per head on mma.sync, the queries' rotation, and the new positions' cache rows
//                    latent_attn_kernel    a CTA has a slice of the context and 32 (token, head) rows, which share the keys;
//                                          both products on the 5th-generation tensor cores
//                    latent_value_kernel   adds up the slices, W_uv per head on mma.sync, output gate
//   bf16, longer     latent_prep_kernel (rotation, cache rows); then the caller unfolds keys and values of the whole context
//                    by a product, and the tcgen05 kernel of csrc/pg_attention_tc.cu reads them
//   f32              latent_query_f32_kernel, the f32 attention of csrc/pg_attention.cu, latent_value_f32_kernel
//
// A step may hold short and long sequences: the kernels of the first group pass over the rows of long ones.
#include <math.h>

#include <algorithm>

#include "pg_attention.cuh"
#include "pg_tcgen05.cuh"

namespace {

constexpr float LOG2E = 1.4426950408889634f;

struct LatentShape {
    int H, D, R, V, C;           // heads, unrotated and rotated query widths, value width, latent width
    int cp, rp, ck;              // C up to 64, R up to 16, and both: a row of the cache
    int dk;                      // D up to 32: a row of uk
    int cap, long_from;          // sequences of long_from and more tokens in a step are passed over
    int own;                     // the projection has a latent of its own, which is put into the cache
    int at_kv, at_gate;          // columns of the projection: [q H (D + R) | latent C, key part R | gate H V]
    float eps, scale;
    const float *rot;            // [cap][R / 2][2]: cos, sin
    const float *c_norm;         // [C]
    const bf16 *uk, *uv;         // [H][cp][dk], [H][V][cp]
};

__device__ __forceinline__ int seq_len(const pg_batch &bt, int seq) { return __ldcg(bt.d_seq_row0 + seq + 1) - __ldcg(bt.d_seq_row0 + seq); }

// A lane's cosines and sines for position pos: pairs lane + 32 i (rot_dim <= 128).
struct Turn {
    float2 r[2];
    __device__ __forceinline__ void ask(const LatentShape &s, int pos, int lane)
    {
        const float2 *cs = reinterpret_cast<const float2 *>(s.rot) + (int64_t)min(max(pos, 0), s.cap - 1) * (s.R / 2);
#pragma unroll
        for (int i = 0; i < 2; i++) r[i] = 2 * (lane + 32 * i) < s.R ? __ldg(cs + lane + 32 * i) : make_float2(1.0f, 0.0f);
    }
};
// One warp: the pairs of src rotated; columns R .. rp are zero.
template <typename TA>
__device__ __forceinline__ void rotate(const LatentShape &s, const float *src, const Turn &turn, TA *dst, int rp, int lane)
{
    float a[2], b[2];
#pragma unroll
    for (int i = 0; i < 2; i++) {
        const int at = 2 * (lane + 32 * i);
        a[i] = at < s.R ? __ldcg(src + at) : 0.0f;
        b[i] = at < s.R ? __ldcg(src + at + 1) : 0.0f;
    }
#pragma unroll
    for (int i = 0; i < 2; i++) {
        const int at = 2 * (lane + 32 * i);
        if (at < rp) {
            pg_put(dst + at, a[i] * turn.r[i].x - b[i] * turn.r[i].y);
            pg_put(dst + at + 1, b[i] * turn.r[i].x + a[i] * turn.r[i].y);
        }
    }
}

// One warp: the cache row of a token, [c | 0 | rotated key part | 0] (kv_rank <= 512).
struct NormWeights {
    float w[16];
    __device__ __forceinline__ void ask(const LatentShape &s, int lane)
    {
#pragma unroll
        for (int i = 0; i < 16; i++) w[i] = i * 32 + lane < s.C ? __ldg(s.c_norm + i * 32 + lane) : 0.0f;
    }
};
template <typename TA>
__device__ __forceinline__ void append(const LatentShape &s, const float *kv, const Turn &turn, const NormWeights &nw, TA *dst, int lane)
{
    float x[16], ss = 0.0f;
#pragma unroll
    for (int i = 0; i < 16; i++) x[i] = i * 32 + lane < s.C ? __ldcg(kv + i * 32 + lane) : 0.0f;
    rotate(s, kv + s.C, turn, dst + s.cp, s.rp, lane);
#pragma unroll
    for (int i = 0; i < 16; i++) ss += x[i] * x[i];
    const float inv = __fdiv_rn(1.0f, sqrtf(__fdiv_rn(pg_warp_sum(ss), (float)s.C) + s.eps));
#pragma unroll
    for (int i = 0; i < 16; i++) {
        const int c = i * 32 + lane;
        if (c < s.cp) pg_put(dst + c, x[i] * inv * nw.w[i]);
    }
}

// D[16 x 8] of one warp: rows of `a` (shared memory, ld elements apart) times eight rows of w (global), K a multiple of 32.
// A lane's 16 contiguous bytes of both feed two MMAs: K is permuted alike on both sides.  `ask` brings the first PRE pieces
// of the weights, which do not depend on the kernel before.
template <int PRE>
struct Weights8 {
    uint4 x[PRE];
    const uint4 *at;
    int pieces;
    __device__ __forceinline__ void ask(const bf16 *__restrict__ w, int64_t ldw, int K, int lane)
    {
        at = reinterpret_cast<const uint4 *>(w + (lane >> 2) * ldw + (lane & 3) * 8);
        pieces = K / 32;
#pragma unroll
        for (int i = 0; i < PRE; i++) x[i] = i < pieces ? __ldg(at + 4 * i) : make_uint4(0u, 0u, 0u, 0u);
    }
    // HI: whether rows 8 .. 15 are there
    template <bool HI>
    __device__ __forceinline__ void times(float (&d)[4], uint32_t a, int ld, int lane)
    {
        const uint32_t a0 = a + (uint32_t)((lane >> 2) * ld + (lane & 3) * 8) * 2, a1 = a0 + (uint32_t)(8 * ld) * 2;
        float e[4] = {};                                  // two sums: shorter chains
        auto step = [&](const uint4 &v, int i) {
            const uint4 lo = pg_lds128(a0 + i * 64), hi = HI ? pg_lds128(a1 + i * 64) : make_uint4(0u, 0u, 0u, 0u);
            pg_mma_bf16(d, lo.x, hi.x, lo.y, hi.y, v.x, v.y);
            pg_mma_bf16(e, lo.z, hi.z, lo.w, hi.w, v.z, v.w);
        };
        // (all in one stretch: behind the last piece the weights are zero)
#pragma unroll
        for (int i = 0; i < PRE; i++) step(x[i], i < pieces ? i : 0);
        for (int i = PRE; i < pieces; i++) step(__ldg(at + 4 * i), i);
#pragma unroll
        for (int i = 0; i < 4; i++) d[i] += e[i];
    }
};

// ---- short portions, bf16 ------------------------------------------------------------------------------------------
// grid (H + own, column parts, tiles of 16 rows).  qx [rows][H][ck]: q', rotated part
constexpr int LQ_T = 256;
__global__ void __launch_bounds__(LQ_T)
    latent_query_kernel(const LatentShape s, const pg_batch bt, const float *__restrict__ proj, int64_t ldp, bf16 *__restrict__ qx, bf16 *cache, int32_t *status)
{
    constexpr int NW = LQ_T / 32, AHEAD = 4;
    extern __shared__ __align__(128) unsigned char smem[];   // [16][dk + 8]
    const int h = blockIdx.x, m0 = blockIdx.z * 16, n = min(16, bt.rows - m0), warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int c_step = gridDim.y * NW * 8;
    int c = (blockIdx.y * NW + warp) * 8;
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    // weights and the batch's arrays do not depend on the kernel before
    Weights8<4> w;
    if (h < s.H && c < s.cp) w.ask(s.uk + ((int64_t)h * s.cp + c) * s.dk, s.dk, s.dk, lane);
    const int mine = blockIdx.y * NW + warp;                 // the first row that this warp rotates (or appends)
    const int pos_first = mine < n ? __ldcg(bt.d_pos + m0 + mine) : 0;
    Turn turn;
    turn.ask(s, pos_first, lane);
    bf16 *sa = reinterpret_cast<bf16 *>(smem);
    const int ld = s.dk + 8;
    if (h == s.H) {
        const int seq_first = mine < n ? __ldcg(bt.d_row_seq + m0 + mine) : 0;
        const int64_t slot_first = __ldcg(bt.d_seq_slot + seq_first);
        const bool skip_first = seq_len(bt, seq_first) >= s.long_from;
        NormWeights nw;
        nw.ask(s, lane);
        asm volatile("griddepcontrol.wait;" ::: "memory");
        for (int i = mine; i < n; i += gridDim.y * NW) {
            const int m = m0 + i, pos = i == mine ? pos_first : __ldcg(bt.d_pos + m), seq = i == mine ? seq_first : __ldcg(bt.d_row_seq + m);
            if (i == mine ? skip_first : seq_len(bt, seq) >= s.long_from) continue;
            if ((unsigned)pos >= (unsigned)s.cap) {   // outside the cache: record it, touch nothing
                if (lane == 0) atomicExch(status, (int32_t)PG_ERR_INVALID);
                continue;
            }
            if (i != mine) turn.ask(s, pos, lane);
            append(s, proj + (int64_t)m * ldp + s.at_kv, turn, nw, cache + ((i == mine ? slot_first : (int64_t)__ldcg(bt.d_seq_slot + seq)) * s.cap + pos) * s.ck, lane);
        }
        return;
    }
    asm volatile("griddepcontrol.wait;" ::: "memory");
    // all first loads in flight together: two rows of the unrotated part, one of the rotated
    const float *src0 = proj + (int64_t)(m0 + warp) * ldp + h * (s.D + s.R), *src1 = src0 + 8 * ldp;
    float v0[AHEAD], v1[AHEAD];
#pragma unroll
    for (int k = 0; k < AHEAD; k++) {
        v0[k] = warp < n && k * 32 + lane < s.D ? __ldcg(src0 + k * 32 + lane) : 0.0f;
        v1[k] = warp + 8 < n && k * 32 + lane < s.D ? __ldcg(src1 + k * 32 + lane) : 0.0f;
    }
    for (int i = mine; i < n; i += gridDim.y * NW) {
        const int m = m0 + i, pos = i == mine ? pos_first : __ldcg(bt.d_pos + m);
        if ((unsigned)pos >= (unsigned)s.cap) {
            if (lane == 0) atomicExch(status, (int32_t)PG_ERR_INVALID);
            continue;
        }
        if (i != mine) turn.ask(s, pos, lane);
        rotate(s, proj + (int64_t)m * ldp + h * (s.D + s.R) + s.D, turn, qx + ((int64_t)m * s.H + h) * s.ck + s.cp, s.rp, lane);
    }
#pragma unroll
    for (int k = 0; k < AHEAD; k++) {
        if (k * 32 < s.dk) {
            sa[warp * ld + k * 32 + lane] = __float2bfloat16_rn(v0[k]);
            sa[(warp + 8) * ld + k * 32 + lane] = __float2bfloat16_rn(v1[k]);
        }
    }
    for (int k = AHEAD * 32 + lane; k < s.dk; k += 32) {
        sa[warp * ld + k] = __float2bfloat16_rn(warp < n && k < s.D ? __ldcg(src0 + k) : 0.0f);
        sa[(warp + 8) * ld + k] = __float2bfloat16_rn(warp + 8 < n && k < s.D ? __ldcg(src1 + k) : 0.0f);
    }
    __syncthreads();
    const int r = lane >> 2, t = lane & 3;
    while (c < s.cp) {
        float d[4] = {};
        w.times<true>(d, pg_smem(sa), ld, lane);
#pragma unroll
        for (int half = 0; half < 2; half++)
            if (r + 8 * half < n)
                *reinterpret_cast<uint32_t *>(qx + ((int64_t)(m0 + r + 8 * half) * s.H + h) * s.ck + c + 2 * t) = pg_pack_bf16(d[2 * half], d[2 * half + 1]);
        c += c_step;
        if (c < s.cp) w.ask(s.uk + ((int64_t)h * s.cp + c) * s.dk, s.dk, s.dk, lane);
    }
}

// The slices of a tile of rows: as many as the launch has, of a multiple of 128 keys each.
struct Slices {
    int kmax, chunk, used;
};
__device__ __forceinline__ Slices slices_of(const LatentShape &s, int pos0, int T, int tile, int rows, int S)
{
    Slices v;
    v.kmax = pos0 + (min((tile + 1) * rows, T * s.H) - 1) / s.H + 1;
    v.chunk = ((v.kmax + S - 1) / S + 127) & ~127;
    v.used = (v.kmax + v.chunk - 1) / v.chunk;
    return v;
}
// The tiles of a sequence are numbered from here on: per_seq numbers for each, or (0) as many as its rows need.
__device__ __forceinline__ int64_t first_tile(const LatentShape &s, int row0, int seq, int rows, int per_seq)
{
    return per_seq ? (int64_t)seq * per_seq : (int64_t)row0 * s.H / rows + seq;
}

// Whether a condition holds in the first four warps, which all arrive here.
__device__ __forceinline__ bool all_four(bool ok)
{
    uint32_t r;
    asm volatile("{\n\t.reg .pred p, q;\n\tsetp.ne.u32 p, %1, 0;\n\tbar.red.and.pred q, 1, 128, p;\n\tselp.u32 %0, 1, 0, q;\n\t}" : "=r"(r) : "r"((uint32_t)ok) : "memory");
    return r != 0;
}

constexpr int LA_KEYS = 128, LA_ROWS = 32;
constexpr int LA_BLOCK = LA_KEYS * 128;                   // bytes of 128 keys x 64 columns
constexpr int LA_QBLOCK = LA_ROWS * 128;
constexpr int LA_THREADS = 192;

// grid (slices, tiles of 32 rows, seqs).  Everything stands on its head, so that the many keys and the many columns are the 128
// rows of the tensor cores' tiles and the 32 (token, head) rows are their columns:
//   S^T [128 keys x 32] = K Q^T                    K: a tile of keys, [block of 64 columns][128 keys][64], swizzled by the copies
//   O^T [kv_rank x 32] += V^T P^T                  V: the first kv_rank columns of the same tile, read along its other side
//   warp 4     TMA: the blocks of a key tile one by one -- those that this step does not write before griddepcontrol.wait --
//              and the queries; a block is asked for again as soon as the products that read it have run
//   warp 5     issues the products: S^T block by block as they arrive, O^T by groups of 128 columns
//   warps 0-3  a thread owns a key (S^T) and a column of every group (O^T).  The rows' maxima over the keys are found by
//              exchanging halves of the rows between lanes, 31 shuffles for 32 rows; they are only replaced, and O^T rescaled,
//              when a row falls behind by more than 2^8.
// Shared memory: key blocks | query blocks [64 columns][32 rows] | P [2][32 rows][64 keys].  TMEM: S^T 32 columns, O^T 32 for each
// group.  part [tile][slice][32][cp + 4]: sums, then maximum (log 2 units) and denominator of each row.
__global__ void __launch_bounds__(LA_THREADS, 1)
    latent_attn_kernel(const __grid_constant__ CUtensorMap map_k, const __grid_constant__ CUtensorMap map_q, const LatentShape s, const pg_batch bt,
                       float *__restrict__ part, int per_seq, int32_t *status, unsigned long long limit_ns)
{
    constexpr int MAXB = 10, TMEM_COLS = 256;
    extern __shared__ uint8_t smem_raw[];
    __shared__ __align__(8) uint64_t bars[2 * MAXB + 4];
    __shared__ uint32_t tmem_slot;
    __shared__ volatile int abort_flag;
    __shared__ __align__(16) float red[LA_ROWS][4];          // a row's maximum, or sum, of each warp
    __shared__ __align__(16) float now[4][LA_ROWS];          // the rows' maxima in use, per warp
    __shared__ int lims[LA_ROWS];
    const int nb = (s.ck + 63) / 64, ng = (s.cp + 127) / 128;   // blocks of a key, groups of 128 value columns
    const uint32_t keys_at = (pg_smem(smem_raw) + 1023u) & ~1023u, q_at = keys_at + nb * LA_BLOCK, p_at = q_at + nb * LA_QBLOCK;
    const uint32_t bar_full = pg_smem(bars), bar_empty = bar_full + 8 * MAXB, bar_q = bar_empty + 8 * MAXB, bar_s = bar_q + 8, bar_p = bar_s + 8, bar_o = bar_p + 8;
    const int split = blockIdx.x, S = gridDim.x, tile = blockIdx.y, seq = blockIdx.z, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    // the batch's arrays do not depend on the kernel before
    const int row0 = __ldcg(bt.d_seq_row0 + seq), T = seq_len(bt, seq), total = T * s.H, rr0 = tile * LA_ROWS;
    const int slot = __ldcg(bt.d_seq_slot + seq);
    if (T >= s.long_from || rr0 >= total) return;
    const int pos0 = __ldcg(bt.d_pos + row0);
    const Slices sl = slices_of(s, pos0, T, tile, LA_ROWS, S);
    const int t0 = split * sl.chunk, t1 = min(sl.kmax, t0 + sl.chunk);
    if (t0 >= t1 || sl.kmax > s.cap) return;              // (positions outside the cache are recorded by latent_query_kernel)
    const int ntiles = (t1 - t0 + LA_KEYS - 1) / LA_KEYS;
    if (threadIdx.x == 0) {
        for (int i = 0; i < nb; i++) {
            pg_mbar_init(bar_full + 8 * i, 1);
            pg_mbar_init(bar_empty + 8 * i, 1);
        }
        pg_mbar_init(bar_q, 1);
        pg_mbar_init(bar_s, 1);
        pg_mbar_init(bar_p, 4);                           // one arrival per softmax warp
        pg_mbar_init(bar_o, 1);
        abort_flag = 0;
        pg_mbar_fence();
    }
    if (threadIdx.x < LA_ROWS) lims[threadIdx.x] = pos0 + min(rr0 + (int)threadIdx.x, total - 1) / s.H;
    if (warp == 5) {
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(pg_smem(&tmem_slot)), "r"(TMEM_COLS) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    // (not before the CTA has its TMEM: nothing behind this kernel can then hold what it needs)
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    const uint32_t tmem_s = tmem_slot, tmem_o = tmem_s + LA_ROWS;

    if (warp == 4) {
        // ---------------------------------------------------------------- producer
        if (lane == 0) {
            bool ok = true, waited = false;
            for (int j = 0; ok && j < ntiles; j++) {
                const int key0 = t0 + j * LA_KEYS;
                if (!waited && (j > 0 || key0 + LA_KEYS > pos0)) {
                    // what follows may read what the kernel before has written: the queries, and the cache from pos0 on
                    asm volatile("griddepcontrol.wait;" ::: "memory");
                    waited = true;
                    pg_mbar_expect(bar_q, nb * LA_QBLOCK);
                    for (int b = 0; b < nb; b++) tma_load_2d(q_at + b * LA_QBLOCK, &map_q, bar_q, b * 64, row0 * s.H + rr0);
                }
                for (int b = 0; b < nb; b++) {
                    if (!(ok = pg_mbar_wait(bar_empty + 8 * b, (j & 1) ^ 1, &abort_flag, status, limit_ns))) break;
                    pg_mbar_expect(bar_full + 8 * b, LA_BLOCK);
                    tma_load_3d(keys_at + b * LA_BLOCK, &map_k, bar_full + 8 * b, b * 64, key0, slot);
                }
                // the next tile on its way to L2 meanwhile
                if (j + 1 < ntiles)
                    for (int b = 0; b < nb; b++) tma_prefetch_3d(&map_k, b * 64, key0 + LA_KEYS, slot);
            }
            if (!waited) {
                asm volatile("griddepcontrol.wait;" ::: "memory");
                pg_mbar_expect(bar_q, nb * LA_QBLOCK);
                for (int b = 0; b < nb; b++) tma_load_2d(q_at + b * LA_QBLOCK, &map_q, bar_q, b * 64, row0 * s.H + rr0);
            }
            if (!ok) {
                // give copies that are still in flight a bounded time to land before the CTA exits
                const unsigned long long w0 = pg_globaltimer_ns();
                while (pg_globaltimer_ns() - w0 < 2000000ull) {
                }
            }
        }
    } else if (warp == 5) {
        // ---------------------------------------------------------------- MMA issuer (the whole warp; one lane's products count)
        {
            const uint32_t on = pg_elect();
            auto wait = [&](uint32_t bar, uint32_t parity) { return (bool)__all_sync(0xffffffffu, pg_mbar_wait(bar, parity, &abort_flag, status, limit_ns)); };
            constexpr uint32_t idesc_s = make_idesc(128, LA_ROWS), idesc_o = make_idesc(128, LA_ROWS) | IDESC_A_MN_MAJOR;
            const uint64_t desc_k = make_smem_desc(keys_at), desc_q = make_smem_desc(q_at), desc_p = make_smem_desc(p_at), desc_v = make_smem_desc_mn(keys_at, LA_BLOCK);
            bool ok = wait(bar_q, 0);
            tc_fence_after();
            for (int j = 0; ok && j < ntiles; j++) {
                for (int b = 0; b < nb; b++) {
                    if (!(ok = wait(bar_full + 8 * b, j & 1))) break;
                    tc_fence_after();
                    const uint64_t dk = desc_k + (uint64_t)(b * (LA_BLOCK >> 4)), dq = desc_q + (uint64_t)(b * (LA_QBLOCK >> 4));
#pragma unroll
                    for (int i = 0; i < 4; i++) umma_f16(tmem_s, dk + i * 2, dq + i * 2, idesc_s, (b | i) != 0, on);
                    if (b * 64 >= s.cp) umma_commit(bar_empty + 8 * b, on);   // no value columns: done with
                }
                if (!ok) break;
                umma_commit(bar_s, on);
                if (!(ok = wait(bar_p, j & 1))) break;
                tc_fence_after();
                for (int g = 0; g < ng; g++) {
                    // (the last group of an odd number of blocks reads one block too many, into rows of O^T that nobody reads)
                    const uint64_t dv = desc_v + (uint64_t)(2 * g * (LA_BLOCK >> 4));
#pragma unroll
                    for (int i = 0; i < LA_KEYS / 16; i++)
                        umma_f16(tmem_o + g * LA_ROWS, dv + i * (2048 >> 4), desc_p + (i / 4) * (LA_QBLOCK >> 4) + (i % 4) * 2, idesc_o, (j | i) != 0, on);
                    for (int b = 2 * g; b < 2 * g + 2 && b * 64 < s.cp; b++) umma_commit(bar_empty + 8 * b, on);
                }
                umma_commit(bar_o, on);
            }
        }
    } else {
        // ---------------------------------------------------------------- softmax
        const uint32_t lanes = (uint32_t)(warp * 32) << 16;
        const float sl2 = s.scale * LOG2E;
        const int low = lims[0];                              // every row sees the keys up to here
        float m = -1e30f, l[LA_ROWS];                         // m: of row `lane` (finite: a row may see nothing of a slice)
#pragma unroll
        for (int c = 0; c < LA_ROWS; c++) l[c] = 0.0f;
        bool ok = true;
        for (int j = 0; j < ntiles; j++) {
            ok = ok && pg_mbar_wait(bar_s, j & 1, &abort_flag, status, limit_ns);
            ok = __all_sync(0xffffffffu, ok);
            tc_fence_after();
            const int key = t0 + j * LA_KEYS + warp * 32 + lane;
            uint32_t v[32];
            tmem_ld32(tmem_s + lanes, v);
            float x[LA_ROWS];
#pragma unroll
            for (int c = 0; c < LA_ROWS; c++) x[c] = __uint_as_float(v[c]) * sl2;
            if (__any_sync(0xffffffffu, key > low || key >= t1)) {
#pragma unroll
                for (int c = 0; c < LA_ROWS; c++)
                    if (key >= t1 || key > lims[c]) x[c] = -INFINITY;
            }
            // lane c ends with row c's maximum over the warp's 32 keys
            float y[LA_ROWS];
#pragma unroll
            for (int c = 0; c < LA_ROWS; c++) y[c] = x[c];
#pragma unroll
            for (int w = 16; w > 0; w >>= 1) {
                const bool upper = lane & w;
#pragma unroll
                for (int c = 0; c < w; c++) {
                    const float give = upper ? y[c] : y[c + w], keep = upper ? y[c + w] : y[c];
                    y[c] = fmaxf(keep, __shfl_xor_sync(0xffffffffu, give, w));
                }
            }
            red[lane][warp] = y[0];
            if (!(ok = all_four(ok))) break;                  // (the warps give up together)
            const float4 r4 = *reinterpret_cast<const float4 *>(red[lane]);
            const float top = fmaxf(fmaxf(r4.x, r4.y), fmaxf(r4.z, r4.w));
            const bool behind = j == 0 ? top > m : top > m + 8.0f;
            const float f = behind ? pg_ex2(m - top) : 1.0f;
            if (behind) m = top;
            now[warp][lane] = m;
            __syncwarp();
            if (j > 0) {
                // (the products of the tile before read P and write O^T)
                ok = pg_mbar_wait(bar_o, (j - 1) & 1, &abort_flag, status, limit_ns);
                ok = __all_sync(0xffffffffu, ok);
                tc_fence_after();
                if (ok && __any_sync(0xffffffffu, behind)) {  // (the same in all four warps)
                    for (int g = 0; g < ng; g++) {
                        uint32_t o[32];
                        tmem_ld32(tmem_o + lanes + g * LA_ROWS, o);
#pragma unroll
                        for (int c = 0; c < LA_ROWS; c++) o[c] = __float_as_uint(__uint_as_float(o[c]) * __shfl_sync(0xffffffffu, f, c));
                        tmem_st32(tmem_o + lanes + g * LA_ROWS, o);
                    }
                    tmem_wait_st();
#pragma unroll
                    for (int c = 0; c < LA_ROWS; c++) l[c] *= __shfl_sync(0xffffffffu, f, c);
                }
            }
            {
                // row c's weights: 128 bytes per row and 64 keys, 16-byte pieces exchanged by row as the copies do
                const uint32_t at = p_at + (warp >> 1) * LA_QBLOCK, col = (uint32_t)(warp & 1) * 4 + (lane >> 3), in = (uint32_t)(lane & 7) * 2;
#pragma unroll
                for (int c = 0; c < LA_ROWS; c += 4) {
                    const float4 mm = *reinterpret_cast<const float4 *>(&now[warp][c]);
                    const float mc[4] = {mm.x, mm.y, mm.z, mm.w};
#pragma unroll
                    for (int i = 0; i < 4; i++) {
                        const float p = pg_ex2(x[c + i] - mc[i]);
                        l[c + i] += p;
                        const bf16 pb = __float2bfloat16_rn(p);
                        asm volatile("st.shared.u16 [%0], %1;" ::"r"(at + (c + i) * 128 + ((col ^ ((c + i) & 7)) << 4) + in), "h"(*reinterpret_cast<const unsigned short *>(&pb))
                                     : "memory");
                    }
                }
            }
            asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
            tc_fence_before();
            __syncwarp();
            if (lane == 0) pg_mbar_arrive(bar_p);
            // (`red` is written again behind the next wait for bar_s, which is behind all four arrivals)
        }
        if (all_four(ok)) {
            // lane c ends with row c's sum over the warp's keys
#pragma unroll
            for (int w = 16; w > 0; w >>= 1) {
                const bool upper = lane & w;
#pragma unroll
                for (int c = 0; c < w; c++) {
                    const float give = upper ? l[c] : l[c + w], keep = upper ? l[c + w] : l[c];
                    l[c] = keep + __shfl_xor_sync(0xffffffffu, give, w);
                }
            }
            asm volatile("bar.sync 1, 128;" ::: "memory");
            red[lane][warp] = l[0];
            asm volatile("bar.sync 1, 128;" ::: "memory");
            const int ms = s.cp + 4;
            float *dst = part + ((first_tile(s, row0, seq, LA_ROWS, per_seq) + tile) * S + split) * LA_ROWS * ms;
            if (warp == 0) {
                const float4 r4 = *reinterpret_cast<const float4 *>(red[lane]);
                *reinterpret_cast<float2 *>(dst + (size_t)lane * ms + s.cp) = make_float2(m, (r4.x + r4.y) + (r4.z + r4.w));
            }
            ok = pg_mbar_wait(bar_o, (ntiles - 1) & 1, &abort_flag, status, limit_ns);
            ok = __all_sync(0xffffffffu, ok);
            tc_fence_after();
            const int rows = min(LA_ROWS, total - rr0);
            for (int g = 0; ok && g < ng; g++) {
                uint32_t o[32];
                tmem_ld32(tmem_o + lanes + g * LA_ROWS, o);
                const int col = g * 128 + warp * 32 + lane;
                if (col < s.cp) {
#pragma unroll
                    for (int c = 0; c < LA_ROWS; c++)
                        if (c < rows) dst[(size_t)c * ms + col] = __uint_as_float(o[c]);
                }
            }
        }
    }
    __syncwarp();
    tc_fence_before();
    __syncthreads();
    if (warp == 5) {
        tc_fence_after();
        asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_s), "r"(TMEM_COLS) : "memory");
    }
}

// grid (H, parts of 128 columns, groups of `group` <= 16 rows): adds the slices of its rows, then W_uv of its head, then the gate.
// `ways` threads share the slices of four columns of a row.
constexpr int LV_T = 512;
constexpr int LV_SLICES = 64;
constexpr int LV_AHEAD = 9;
__global__ void __launch_bounds__(LV_T, 1)
    latent_value_kernel(const LatentShape s, const pg_batch bt, const float *__restrict__ part, int per_seq, int S, int group, int ways,
                        const float *__restrict__ proj, int64_t ldp, bf16 *__restrict__ out, int64_t ldo)
{
    extern __shared__ __align__(128) unsigned char smem[];   // [16][cp + 8] | sums [ways][group][cp]
    __shared__ float weight[16][LV_SLICES];
    __shared__ int64_t base[16];
    __shared__ int used[16];
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    const int h = blockIdx.x, m0 = blockIdx.z * group, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int c = blockIdx.y * 128 + warp * 8;
    // weights and the batch's arrays do not depend on the kernel before
    Weights8<16> w;
    // (rows of W_uv behind the head's last one belong to the next head or are padding; their products are dropped)
    w.pieces = 0;
    if (c < s.V) w.ask(s.uv + ((int64_t)h * s.V + c) * s.cp, s.cp, s.cp, lane);
    bf16 *sa = reinterpret_cast<bf16 *>(smem);
    const int ld = s.cp + 8, ms = s.cp + 4;
    float *sums = reinterpret_cast<float *>(smem + (size_t)16 * ld * 2);
    if (threadIdx.x < 16) {
        // where the row's slices are
        const int m = m0 + threadIdx.x;
        int n = 0;
        int64_t at = 0;
        if ((int)threadIdx.x < group && m < bt.rows) {
            const int seq = __ldcg(bt.d_row_seq + m), row0 = __ldcg(bt.d_seq_row0 + seq), T = seq_len(bt, seq);
            const int pos0 = __ldcg(bt.d_pos + row0), rr = (m - row0) * s.H + h, tile = rr / LA_ROWS;
            const Slices sl = slices_of(s, pos0, T, tile, LA_ROWS, S);
            if (T < s.long_from && sl.kmax <= s.cap) {
                n = sl.used;
                at = ((first_tile(s, row0, seq, LA_ROWS, per_seq) + tile) * S * LA_ROWS + rr % LA_ROWS) * (int64_t)ms;
            }
        }
        used[threadIdx.x] = n;
        base[threadIdx.x] = at;
    }
    __syncthreads();
    asm volatile("griddepcontrol.wait;" ::: "memory");
    const int quads = s.cp / 4, items = group * quads * ways;
    const int64_t step = (int64_t)LA_ROWS * ms;
    const int r = lane >> 2, t = lane & 3;
    // the first loads of everything together: sums of slices, their maxima and denominators, gates
    float4 v[LV_AHEAD];
    auto ask = [&](int i, int k0) {
        const int way = i / (group * quads), x = i / quads - way * group, k4 = (i % quads) * 4, n = used[x];
        const float *src = part + base[x] + k4;
#pragma unroll
        for (int k = 0; k < LV_AHEAD; k++) v[k] = n ? __ldcg(reinterpret_cast<const float4 *>(src + (int64_t)min((k0 + k) * ways + way, n - 1) * step)) : make_float4(0.f, 0.f, 0.f, 0.f);
    };
    if ((int)threadIdx.x < items) ask(threadIdx.x, 0);
    float gate[2][2];
#pragma unroll
    for (int half = 0; half < 2; half++)
#pragma unroll
        for (int j = 0; j < 2; j++) {
            const int col = c + 2 * t + j;
            gate[half][j] = used[r + 8 * half] && col < s.V ? __ldcg(proj + (int64_t)(m0 + r + 8 * half) * ldp + s.at_gate + h * s.V + col) : 0.0f;
        }
    if (warp < group && used[warp]) {
        // a warp per row: the weights of its slices
        const int n = used[warp];
        float2 ml[LV_SLICES / 32];
        float top = -INFINITY, l = 0.0f;
#pragma unroll
        for (int i = 0; i < LV_SLICES / 32; i++) {
            const int k = i * 32 + lane;
            ml[i] = k < n ? __ldcg(reinterpret_cast<const float2 *>(part + base[warp] + k * step + s.cp)) : make_float2(-INFINITY, 0.0f);
            top = fmaxf(top, ml[i].x);
        }
#pragma unroll
        for (int y = 16; y > 0; y >>= 1) top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, y));
#pragma unroll
        for (int i = 0; i < LV_SLICES / 32; i++) {
            ml[i].x = exp2f(ml[i].x - top);
            l = fmaf(ml[i].x, ml[i].y, l);
        }
        const float inv = __fdiv_rn(1.0f, pg_warp_sum(l));
#pragma unroll
        for (int i = 0; i < LV_SLICES / 32; i++) weight[warp][i * 32 + lane] = ml[i].x * inv;
    }
    __syncthreads();
    for (int i = threadIdx.x; i < items; i += LV_T) {
        const int way = i / (group * quads), x = i / quads - way * group, k4 = (i % quads) * 4, n = used[x];
        float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
        if (i != (int)threadIdx.x) ask(i, 0);
        for (int k0 = 0; k0 * ways < n; k0 += LV_AHEAD) {
            if (k0 > 0) ask(i, k0);
#pragma unroll
            for (int k = 0; k < LV_AHEAD; k++) {
                const int slice = (k0 + k) * ways + way;
                const float f = slice < n ? weight[x][slice] : 0.0f;   // (behind the last slice: the last one again, with weight 0)
                a.x = fmaf(f, v[k].x, a.x), a.y = fmaf(f, v[k].y, a.y), a.z = fmaf(f, v[k].z, a.z), a.w = fmaf(f, v[k].w, a.w);
            }
        }
        if (ways == 1)
            *reinterpret_cast<uint2 *>(sa + x * ld + k4) = make_uint2(pg_pack_bf16(a.x, a.y), pg_pack_bf16(a.z, a.w));
        else
            *reinterpret_cast<float4 *>(sums + (size_t)(way * group + x) * s.cp + k4) = a;
    }
    __syncthreads();
    if (ways > 1) {
        for (int i = threadIdx.x; i < group * quads; i += LV_T) {
            const int x = i / quads, k4 = (i - x * quads) * 4;
            float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
            for (int way = 0; way < ways; way++) {
                const float4 u = *reinterpret_cast<const float4 *>(sums + (size_t)(way * group + x) * s.cp + k4);
                a.x += u.x, a.y += u.y, a.z += u.z, a.w += u.w;
            }
            *reinterpret_cast<uint2 *>(sa + x * ld + k4) = make_uint2(pg_pack_bf16(a.x, a.y), pg_pack_bf16(a.z, a.w));
        }
        __syncthreads();
    }
    // (rows behind the group are whatever the shared memory held: nobody reads their products)
    if (c >= s.V) return;
    float d[4] = {};
    if (group > 8)
        w.times<true>(d, pg_smem(sa), ld, lane);
    else
        w.times<false>(d, pg_smem(sa), ld, lane);
#pragma unroll
    for (int half = 0; half < 2; half++) {
        const int x = r + 8 * half, m = m0 + x;
        if (used[x] == 0) continue;
#pragma unroll
        for (int j = 0; j < 2; j++) {
            const int col = c + 2 * t + j;
            if (col < s.V) pg_put(out + (int64_t)m * ldo + h * s.V + col, d[2 * half + j] * pg_sigmoid(gate[half][j]));
        }
    }
}

// ---- longer portions: grid (tokens of the sequence) ------------------------------------------------------------------
// q [rows][H][qd]: the unrotated part up to a multiple of 64, then the rotated part, the same
__global__ void __launch_bounds__(256)
    latent_prep_kernel(const LatentShape s, const pg_batch bt, int row0, int64_t slot, const float *__restrict__ proj, int64_t ldp, bf16 *__restrict__ q, int qd,
                       bf16 *cache, int32_t *status)
{
    pg_pdl_begin();
    const int m = row0 + blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, dn = (s.D + 63) & ~63;
    const int pos = __ldcg(bt.d_pos + m);
    if ((unsigned)pos >= (unsigned)s.cap) {   // outside the cache: record it, touch nothing
        if (threadIdx.x == 0) atomicExch(status, (int32_t)PG_ERR_INVALID);
        return;
    }
    const float *row = proj + (int64_t)m * ldp;
    Turn turn;
    turn.ask(s, pos, lane);
    if (s.own && warp == 7) {
        NormWeights nw;
        nw.ask(s, lane);
        append(s, row + s.at_kv, turn, nw, cache + (slot * s.cap + pos) * s.ck, lane);
    }
    if (s.D % 4 == 0 && s.D <= 128 && s.R % 2 == 0 && s.R <= 64 && (s.D + s.R) % 4 == 0 && ldp % 4 == 0) {
        // four heads at a time, all their loads in flight
        for (int h0 = warp; h0 < s.H; h0 += 32) {
            float4 v[4];
            float2 p[4];
#pragma unroll
            for (int i = 0; i < 4; i++) {
                const float *src = row + (h0 + 8 * i) * (s.D + s.R);
                const bool in = h0 + 8 * i < s.H;
                v[i] = in && 4 * lane < s.D ? __ldcg(reinterpret_cast<const float4 *>(src) + lane) : make_float4(0.f, 0.f, 0.f, 0.f);
                p[i] = in && 2 * lane < s.R ? __ldcg(reinterpret_cast<const float2 *>(src + s.D) + lane) : make_float2(0.f, 0.f);
            }
#pragma unroll
            for (int i = 0; i < 4; i++) {
                if (h0 + 8 * i >= s.H) break;
                bf16 *dst = q + ((int64_t)m * s.H + h0 + 8 * i) * qd;
                if (4 * lane < dn) *reinterpret_cast<uint2 *>(dst + 4 * lane) = make_uint2(pg_pack_bf16(v[i].x, v[i].y), pg_pack_bf16(v[i].z, v[i].w));
                if (2 * lane < qd - dn)
                    *reinterpret_cast<uint32_t *>(dst + dn + 2 * lane) = pg_pack_bf16(p[i].x * turn.r[0].x - p[i].y * turn.r[0].y, p[i].y * turn.r[0].x + p[i].x * turn.r[0].y);
            }
        }
        return;
    }
    for (int h = warp; h < s.H; h += 8) {
        {
            const float *src = row + h * (s.D + s.R);
            bf16 *dst = q + ((int64_t)m * s.H + h) * qd;
            for (int c = 2 * lane; c < dn; c += 64)
                *reinterpret_cast<uint32_t *>(dst + c) = pg_pack_bf16(c < s.D ? __ldcg(src + c) : 0.0f, c + 1 < s.D ? __ldcg(src + c + 1) : 0.0f);
            rotate(s, src + s.D, turn, dst + dn, qd - dn, lane);
        }
    }
}

// ---- f32: grid (H + own, rows) -----------------------------------------------------------------------------------------
// y[n] = sum of w[n][k] a[k]: eight terms of K at a time (w is zero behind the true width, and so is a)
__device__ __forceinline__ float dot_row(const bf16 *__restrict__ w, const float *a, int K)
{
    float d[4] = {};
    for (int k = 0; k < K; k += 8) {
        const uint4 x = __ldg(reinterpret_cast<const uint4 *>(w + k));
        d[0] = fmaf(pg_bf16_lo(x.x), a[k], d[0]), d[1] = fmaf(pg_bf16_hi(x.x), a[k + 1], d[1]);
        d[2] = fmaf(pg_bf16_lo(x.y), a[k + 2], d[2]), d[3] = fmaf(pg_bf16_hi(x.y), a[k + 3], d[3]);
        d[0] = fmaf(pg_bf16_lo(x.z), a[k + 4], d[0]), d[1] = fmaf(pg_bf16_hi(x.z), a[k + 5], d[1]);
        d[2] = fmaf(pg_bf16_lo(x.w), a[k + 6], d[2]), d[3] = fmaf(pg_bf16_hi(x.w), a[k + 7], d[3]);
    }
    return (d[0] + d[1]) + (d[2] + d[3]);
}

__global__ void __launch_bounds__(128)
    latent_query_f32_kernel(const LatentShape s, const pg_batch bt, const float *__restrict__ proj, int64_t ldp, float *__restrict__ qx, float *cache,
                            int32_t *status)
{
    extern __shared__ float sm[];   // [dk]
    pg_pdl_begin();
    const int h = blockIdx.x, m = blockIdx.y, lane = threadIdx.x & 31;
    const int pos = __ldcg(bt.d_pos + m);
    if ((unsigned)pos >= (unsigned)s.cap) {   // outside the cache: record it, touch nothing
        if (threadIdx.x == 0) atomicExch(status, (int32_t)PG_ERR_INVALID);
        return;
    }
    if (h == s.H) {
        const int64_t slot = __ldcg(bt.d_seq_slot + __ldcg(bt.d_row_seq + m));
        if (threadIdx.x < 32) {
            Turn turn;
            NormWeights nw;
            turn.ask(s, pos, lane);
            nw.ask(s, lane);
            append(s, proj + (int64_t)m * ldp + s.at_kv, turn, nw, cache + (slot * s.cap + pos) * s.ck, lane);
        }
        return;
    }
    const float *src = proj + (int64_t)m * ldp + h * (s.D + s.R);
    float *dst = qx + ((int64_t)m * s.H + h) * s.ck;
    for (int i = threadIdx.x; i < s.dk; i += 128) sm[i] = i < s.D ? __ldcg(src + i) : 0.0f;
    if (threadIdx.x < 32) {
        Turn turn;
        turn.ask(s, pos, lane);
        rotate(s, src + s.D, turn, dst + s.cp, s.rp, lane);
    }
    __syncthreads();
    for (int n = threadIdx.x; n < s.cp; n += 128) dst[n] = dot_row(s.uk + ((int64_t)h * s.cp + n) * s.dk, sm, s.dk);
}

// o [rows][H][C], grid (H, rows)
__global__ void __launch_bounds__(128)
    latent_value_f32_kernel(const LatentShape s, const float *__restrict__ o, const float *__restrict__ proj, int64_t ldp, float *__restrict__ out, int64_t ldo)
{
    extern __shared__ float sm[];   // [cp]
    pg_pdl_begin();
    const int h = blockIdx.x, m = blockIdx.y;
    for (int i = threadIdx.x; i < s.cp; i += 128) sm[i] = i < s.C ? __ldcg(o + ((int64_t)m * s.H + h) * s.C + i) : 0.0f;
    __syncthreads();
    for (int n = threadIdx.x; n < s.V; n += 128) {
        const float g = pg_sigmoid(__ldcg(proj + (int64_t)m * ldp + s.at_gate + h * s.V + n));
        out[(int64_t)m * ldo + h * s.V + n] = g * dot_row(s.uv + ((int64_t)h * s.V + n) * s.cp, sm, s.cp);
    }
}

LatentShape shape_of(const pg_latent *p)
{
    LatentShape s;
    s.H = p->heads, s.D = p->dim, s.R = p->rot_dim, s.V = p->vdim, s.C = p->kv_rank;
    s.cp = (int)pg_up(s.C, 64), s.rp = (int)pg_up(s.R, 16), s.ck = s.cp + s.rp, s.dk = (int)pg_up(s.D, 32);
    s.cap = p->cap, s.long_from = 1 << 30, s.own = p->own;
    s.at_kv = s.H * (s.D + s.R), s.at_gate = s.at_kv + (s.own ? s.C + s.R : 0);
    s.eps = p->eps, s.scale = p->scale;
    s.rot = p->d_rot, s.c_norm = p->d_norm;
    s.uk = (const bf16 *)p->d_uk, s.uv = (const bf16 *)p->d_uv;
    return s;
}

int attn_smem(const LatentShape &s) { return 1024 + (s.ck + 63) / 64 * (LA_BLOCK + LA_QBLOCK) + 2 * LA_QBLOCK; }

// slices of the context: about one CTA per SM, none shorter than 128 positions of a full cache
int slices(const pg_ctx *ctx, int64_t units, int64_t cap)
{
    int64_t S = std::max<int64_t>(1, (int64_t)ctx->sm_count / std::max<int64_t>(1, units));
    S = std::min<int64_t>(S, std::max<int64_t>(1, cap / LA_KEYS));
    return (int)std::min<int64_t>(S, LV_SLICES);
}

int32_t check(const pg_latent *p, const pg_batch *batch, int64_t ldp, int64_t ldo)
{
    PG_REQUIRE(p && batch && p->d_rot && p->d_uk && p->d_uv && p->d_q && (p->d_norm || !p->own), "latent attention: null pointer");
    PG_REQUIRE(p->heads > 0 && p->dim > 0 && p->dim <= 512 && p->rot_dim >= 0 && p->rot_dim <= 128 && p->rot_dim % 2 == 0 && p->vdim > 0 && p->kv_rank > 0 && p->kv_rank <= 512 &&
                   p->cap > 0 && p->heads <= 65534,
               "latent attention: bad shape (dim %d and latent %d at most 512, an even rot_dim %d at most 128)", p->dim, p->kv_rank, p->rot_dim);
    const LatentShape s = shape_of(p);
    PG_REQUIRE(s.ck <= 640, "latent attention: a key of %d and %d columns is too wide", s.C, s.R);
    PG_REQUIRE(ldp >= s.at_gate + (int64_t)s.H * s.V && ldo >= (int64_t)s.H * s.V, "latent attention: rows too short");
    PG_REQUIRE(batch->rows >= 0 && batch->seqs <= 65535, "latent attention: too many sequences");
    return PG_OK;
}

}  // namespace

extern "C" {

PG_API int64_t pg_latent_part_floats(pg_ctx *ctx, const pg_latent *p, int32_t dtype, int64_t max_rows, int64_t max_seqs)
{
    if (!ctx || !p || max_rows <= 0) return 0;
    const LatentShape s = shape_of(p);
    if (dtype == PG_F32) return max_rows * s.H * s.C;
    // tiles x slices: as many as there are tiles, or about one CTA per SM
    const int64_t tiles = (max_rows * s.H + LA_ROWS - 1) / LA_ROWS + max_seqs;
    return std::max<int64_t>(tiles, 2 * ctx->sm_count) * LA_ROWS * (s.cp + 4);
}

PG_API int32_t pg_latent_run(pg_ctx *ctx, const pg_latent *p, const pg_batch *batch, int64_t long_from, int64_t short_rows, int64_t short_len,
                             const float *d_proj, int64_t ldp, void *d_cache, void *d_out, int32_t dtype, int64_t ldo)
{
    PG_ENTER(ctx);
    PG_REQUIRE(d_proj && d_cache && d_out && p && p->d_part, "latent attention: null pointer");
    int32_t rc = check(p, batch, ldp, ldo);
    if (rc != PG_OK) return rc;
    if (batch->rows == 0 || short_rows <= 0) return PG_OK;
    LatentShape s = shape_of(p);
    if (dtype == PG_F32) {
        PG_REQUIRE(long_from > batch->max_len && batch->rows <= 65535, "latent attention: the f32 form takes portions of any length together, up to 65535 rows");
        float *q = (float *)p->d_q, *cache = (float *)d_cache, *o = (float *)p->d_part;
        rc = launch_pdl(ctx, latent_query_f32_kernel, dim3((unsigned)(s.H + s.own), (unsigned)batch->rows), dim3(128), (size_t)s.dk * 4, s, *batch, d_proj, ldp, q,
                        cache, ctx->d_status);
        if (rc != PG_OK) return rc;
        AttnShape a = {};
        a.H = a.rep = s.H, a.G = 1, a.D = s.ck, a.V = s.C, a.dp = a.vp = s.ck, a.cap = a.limit = s.cap, a.scale = s.scale;
        rc = pgk_attention_f32(ctx, a, batch, q, cache, cache, o, (int64_t)s.H * s.C);
        if (rc != PG_OK) return rc;
        return launch_pdl(ctx, latent_value_f32_kernel, dim3((unsigned)s.H, (unsigned)batch->rows), dim3(128), (size_t)s.cp * 4, s, (const float *)o, d_proj, ldp,
                          (float *)d_out, ldo);
    }
    PG_REQUIRE(long_from > 0 && short_len > 0 && short_len < long_from && short_rows <= batch->rows, "latent attention: bad division of the step");
    s.long_from = (int)std::min<int64_t>(long_from, 1 << 30);
    bf16 *q = (bf16 *)p->d_q, *cache = (bf16 *)d_cache;
    const unsigned row_tiles = (unsigned)((batch->rows + 15) / 16);
    PG_REQUIRE(row_tiles <= 65535, "latent attention: too many rows");
    // columns of W_uk^T over enough CTAs for one per SM
    int parts = 1;
    while (parts < 8 && (int64_t)(s.H + 1) * row_tiles * parts < ctx->sm_count && s.cp / (parts * 2) >= 64) parts *= 2;
    rc = launch_pdl(ctx, latent_query_kernel, dim3((unsigned)(s.H + s.own), (unsigned)parts, row_tiles), dim3(LQ_T), (size_t)(16 * (s.dk + 8) * 2), s, *batch,
                    d_proj, ldp, q, cache, ctx->d_status);
    if (rc != PG_OK) return rc;
    const int64_t tiles = (short_len * s.H + LA_ROWS - 1) / LA_ROWS;
    PG_REQUIRE(tiles <= 65535, "latent attention: too many rows in one sequence");
    // the numbering of tiles that needs fewer of them, and as many slices as then have room
    const int64_t dense = (int64_t)batch->rows * s.H / LA_ROWS + batch->seqs, even = tiles * batch->seqs;
    const int per_seq = even <= dense ? (int)tiles : 0;
    const int64_t room = p->part_floats / ((int64_t)LA_ROWS * (s.cp + 4)) / std::min(even, dense);
    PG_REQUIRE(room >= 1, "latent attention: the step has more rows than d_part has room for");
    const int S = (int)std::min<int64_t>(room, slices(ctx, std::max<int64_t>(tiles, (short_rows * s.H + LA_ROWS - 1) / LA_ROWS), s.cap));
    {
        CUtensorMap mk, mq;
        const cuuint64_t dk[3] = {(cuuint64_t)s.ck, (cuuint64_t)s.cap, (cuuint64_t)p->slots}, sk[2] = {(cuuint64_t)s.ck * 2, (cuuint64_t)s.cap * s.ck * 2};
        const cuuint64_t dq[2] = {(cuuint64_t)s.ck, (cuuint64_t)batch->rows * s.H}, sq[1] = {(cuuint64_t)s.ck * 2};
        const cuuint32_t bk[3] = {64, LA_KEYS, 1}, bq[2] = {64, LA_ROWS};
        rc = pg_encode_bf16(&mk, cache, 3, dk, sk, bk);
        if (rc == PG_OK) rc = pg_encode_bf16(&mq, q, 2, dq, sq, bq);
        if (rc != PG_OK) return rc;
        static std::atomic<uint64_t> set{0};
        PG_CUDA(pg_max_smem_once(latent_attn_kernel, 224 * 1024, ctx->device, set));
        rc = launch_pdl(ctx, latent_attn_kernel, dim3((unsigned)S, (unsigned)tiles, (unsigned)batch->seqs), dim3(LA_THREADS), (size_t)attn_smem(s), mk, mq, s, *batch,
                        p->d_part, per_seq, ctx->d_status, ctx->wait_limit_ns);
        if (rc != PG_OK) return rc;
    }
    // groups of rows small enough for about one CTA per SM
    const unsigned parts128 = (unsigned)((s.V + 127) / 128);
    int group = 16;
    while (group > 1 && (int64_t)s.H * parts128 * ((batch->rows + group - 1) / group) < ctx->sm_count * 3 / 4) group /= 2;
    const int ways = std::max(1, std::min(8, LV_T / (group * s.cp / 4)));
    const int64_t groups = (batch->rows + group - 1) / group;
    PG_REQUIRE(groups <= 65535 && parts128 <= 65535, "latent attention: too many rows");
    const size_t smem = (size_t)16 * (s.cp + 8) * 2 + (ways > 1 ? (size_t)ways * group * s.cp * 4 : 0);
    static std::atomic<uint64_t> set{0};
    PG_CUDA(pg_max_smem_once(latent_value_kernel, 64 * 1024, ctx->device, set));
    return launch_pdl(ctx, latent_value_kernel, dim3((unsigned)s.H, parts128, (unsigned)groups), dim3(LV_T), smem, s, *batch, (const float *)p->d_part, per_seq, S,
                      group, ways, d_proj, ldp, (bf16 *)d_out, ldo);
}

PG_API int32_t pg_latent_prompt_supports(const pg_latent *p)
{
    return p && p->scale > 0.0f && p->rot_dim > 0 && pgk_attention_split_supports((int)pg_up(p->dim, 16), (int)pg_up(p->rot_dim, 16), p->vdim);
}

PG_API int32_t pg_latent_prompt_prep(pg_ctx *ctx, const pg_latent *p, const pg_batch *batch, int64_t row0, int64_t len, int64_t slot, const float *d_proj,
                                     int64_t ldp, void *d_cache)
{
    PG_ENTER(ctx);
    PG_REQUIRE(d_proj && d_cache, "latent attention: null pointer");
    const int32_t rc = check(p, batch, ldp, (int64_t)p->heads * p->vdim);
    if (rc != PG_OK) return rc;
    PG_REQUIRE(row0 >= 0 && len > 0 && row0 + len <= batch->rows && slot >= 0 && slot < p->slots, "latent attention: bad sequence");
    const LatentShape s = shape_of(p);
    return launch_pdl(ctx, latent_prep_kernel, dim3((unsigned)len), dim3(256), 0, s, *batch, (int)row0, slot, d_proj, ldp, (bf16 *)p->d_q,
                      (int)(pg_up(s.D, 64) + pg_up(s.R, 64)), (bf16 *)d_cache, ctx->d_status);
}

PG_API int32_t pg_latent_prompt(pg_ctx *ctx, const pg_latent *p, const pg_batch *batch, int64_t seq, int64_t len, int64_t positions, int64_t slot,
                                const float *d_proj, int64_t ldp, const void *d_cache, const void *d_kv, int64_t ldkv, void *d_out, int64_t ldo)
{
    PG_ENTER(ctx);
    PG_REQUIRE(d_proj && d_cache && d_kv && d_out, "latent attention: null pointer");
    const int32_t rc = check(p, batch, ldp, ldo);
    if (rc != PG_OK) return rc;
    const LatentShape s = shape_of(p);
    PG_REQUIRE(pg_latent_prompt_supports(p) && seq >= 0 && seq < batch->seqs && slot >= 0 && slot < p->slots && len > 0 && positions >= len && positions <= s.cap,
               "latent attention: bad sequence");
    AttnSplitKeys k;
    k.kd = (int)pg_up(s.D, 16), k.vd = (int)pg_up(s.V, 16), k.ldk = ldkv;
    PG_REQUIRE(ldkv >= (int64_t)s.H * (k.kd + k.vd) && ldkv % 8 == 0, "latent attention: rows too short");
    k.q = (const bf16 *)p->d_q, k.qd = (int)(pg_up(s.D, 64) + pg_up(s.R, 64));
    k.k = (const bf16 *)d_kv, k.v = k.k + (int64_t)s.H * k.kd;
    k.shared = (const bf16 *)d_cache + slot * s.cap * s.ck + s.cp, k.sd = s.rp, k.lds = s.ck;
    k.gate = d_proj + s.at_gate, k.ldg = ldp;
    k.seq = (int)seq, k.len = (int)len, k.positions = (int)positions;
    AttnShape a = {};
    a.H = a.G = s.H, a.rep = 1, a.D = s.D + s.R, a.V = s.V, a.cap = a.limit = (int)positions, a.scale = s.scale;
    return pgk_attention_split_tc(ctx, a, batch, k, (bf16 *)d_out, ldo);
}

}  // extern "C"
