// Latent attention: a position is cached as one latent c (kv_rank numbers, normalised) and one rotated key part that all heads
// share.  A head's key is [W_uk c | rotated part], its value W_uv c.
//
// Short portions never unfold the cache.  With q' = W_uk^T q the score is q' . c + q_rot . k_rot and the head's output is
// W_uv (sum p c): attention of all heads over one key of kv_rank + rot_dim, whose first kv_rank columns are the value.
//
//   bf16, short      latent_query_kernel   q' per head on mma.sync, the queries' rotation, and the new positions' cache rows
//                    latent_attn_kernel    a CTA has a slice of the context and 16 or 32 (token, head) rows, which share the
//                                          keys; the warps divide keys and columns between them
//                    latent_value_kernel   adds up the slices, W_uv per head on mma.sync, output gate
//   bf16, longer     latent_prep_kernel (rotation, cache rows); then the caller unfolds keys and values of the whole context
//                    by a product, and the tcgen05 kernel of csrc/pg_attention_tc.cu reads them
//   f32              latent_query_f32_kernel, the f32 attention of csrc/pg_attention.cu, latent_value_f32_kernel
//
// A step may hold short and long sequences: the kernels of the first group pass over the rows of long ones.
#include <math.h>

#include <algorithm>

#include "pg_async.cuh"
#include "pg_attention.cuh"

namespace {

constexpr float LOG2E = 1.4426950408889634f;

__device__ __forceinline__ float pg_ex2(float x)
{
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

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

// One warp: the pairs of src rotated for position pos; columns R .. rp are zero.
template <typename TA>
__device__ __forceinline__ void rotate(const LatentShape &s, const float *src, int pos, TA *dst, int rp, int lane)
{
    const float2 *cs = reinterpret_cast<const float2 *>(s.rot) + (int64_t)pos * (s.R / 2);
    for (int i = lane; i < rp / 2; i += 32) {
        float u = 0.0f, v = 0.0f;
        if (2 * i < s.R) {
            const float a = __ldcg(src + 2 * i), b = __ldcg(src + 2 * i + 1);
            const float2 r = __ldg(cs + i);
            u = a * r.x - b * r.y;
            v = b * r.x + a * r.y;
        }
        pg_put(dst + 2 * i, u);
        pg_put(dst + 2 * i + 1, v);
    }
}

// One warp: the cache row of a token, [c | 0 | rotated key part | 0] (kv_rank <= 512).
template <typename TA>
__device__ __forceinline__ void append(const LatentShape &s, const float *kv, int pos, TA *dst, int lane)
{
    float x[16], ss = 0.0f;
#pragma unroll
    for (int i = 0; i < 16; i++) x[i] = i * 32 + lane < s.C ? __ldcg(kv + i * 32 + lane) : 0.0f;
    rotate(s, kv + s.C, pos, dst + s.cp, s.rp, lane);
#pragma unroll
    for (int i = 0; i < 16; i++) ss += x[i] * x[i];
    const float inv = __fdiv_rn(1.0f, sqrtf(__fdiv_rn(pg_warp_sum(ss), (float)s.C) + s.eps));
#pragma unroll
    for (int i = 0; i < 16; i++) {
        const int c = i * 32 + lane;
        if (c < s.cp) pg_put(dst + c, c < s.C ? x[i] * inv * __ldg(s.c_norm + c) : 0.0f);
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
    __device__ __forceinline__ void times(float (&d)[4], uint32_t a, int ld, int lane)
    {
        const uint32_t a0 = a + (uint32_t)((lane >> 2) * ld + (lane & 3) * 8) * 2, a1 = a0 + (uint32_t)(8 * ld) * 2;
        float e[4] = {};                                  // two sums: shorter chains
        auto step = [&](const uint4 &v, int i) {
            const uint4 lo = pg_lds128(a0 + i * 64), hi = pg_lds128(a1 + i * 64);
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
    constexpr int NW = LQ_T / 32;
    extern __shared__ __align__(128) unsigned char smem[];   // [16][dk + 8]
    const int h = blockIdx.x, m0 = blockIdx.z * 16, n = min(16, bt.rows - m0), warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int c_step = gridDim.y * NW * 8;
    int c = (blockIdx.y * NW + warp) * 8;
    Weights8<4> w;
    if (h < s.H && c < s.cp) w.ask(s.uk + ((int64_t)h * s.cp + c) * s.dk, s.dk, s.dk, lane);
    pg_pdl_begin();
    bf16 *sa = reinterpret_cast<bf16 *>(smem);
    const int ld = s.dk + 8;
    if (h == s.H) {
        for (int i = blockIdx.y * NW + warp; i < n; i += gridDim.y * NW) {
            const int m = m0 + i, pos = __ldcg(bt.d_pos + m), seq = __ldcg(bt.d_row_seq + m);
            if (seq_len(bt, seq) >= s.long_from) continue;
            if ((unsigned)pos >= (unsigned)s.cap) {   // outside the cache: record it, touch nothing
                if (lane == 0) atomicExch(status, (int32_t)PG_ERR_INVALID);
                continue;
            }
            append(s, proj + (int64_t)m * ldp + s.at_kv, pos, cache + ((int64_t)__ldcg(bt.d_seq_slot + seq) * s.cap + pos) * s.ck, lane);
        }
        return;
    }
    for (int i = warp; i < 16; i += NW) {
        const float *src = proj + (int64_t)(m0 + i) * ldp + h * (s.D + s.R);
#pragma unroll 4
        for (int k = lane; k < s.dk; k += 32) sa[i * ld + k] = __float2bfloat16_rn(i < n && k < s.D ? __ldcg(src + k) : 0.0f);
    }
    for (int i = blockIdx.y * NW + warp; i < n; i += gridDim.y * NW) {
        const int m = m0 + i, pos = __ldcg(bt.d_pos + m);
        if ((unsigned)pos >= (unsigned)s.cap) {
            if (lane == 0) atomicExch(status, (int32_t)PG_ERR_INVALID);
            continue;
        }
        rotate(s, proj + (int64_t)m * ldp + h * (s.D + s.R) + s.D, pos, qx + ((int64_t)m * s.H + h) * s.ck + s.cp, s.rp, lane);
    }
    __syncthreads();
    const int r = lane >> 2, t = lane & 3;
    while (c < s.cp) {
        float d[4] = {};
        w.times(d, pg_smem(sa), ld, lane);
#pragma unroll
        for (int half = 0; half < 2; half++)
            if (r + 8 * half < n)
                *reinterpret_cast<uint32_t *>(qx + ((int64_t)(m0 + r + 8 * half) * s.H + h) * s.ck + c + 2 * t) = pg_pack_bf16(d[2 * half], d[2 * half + 1]);
        c += c_step;
        if (c < s.cp) w.ask(s.uk + ((int64_t)h * s.cp + c) * s.dk, s.dk, s.dk, lane);
    }
}

// The slices of a tile of rows: as many as the launch has, of a multiple of 64 keys each.
struct Slices {
    int kmax, chunk, used;
};
__device__ __forceinline__ Slices slices_of(const LatentShape &s, int pos0, int T, int tile, int rows, int S)
{
    Slices v;
    v.kmax = pos0 + (min((tile + 1) * rows, T * s.H) - 1) / s.H + 1;
    v.chunk = ((v.kmax + S - 1) / S + 63) & ~63;
    v.used = (v.kmax + v.chunk - 1) / v.chunk;
    return v;
}
// The tiles of a sequence are numbered from here on: per_seq numbers for each, or (0) as many as its rows need.
__device__ __forceinline__ int64_t first_tile(const LatentShape &s, int row0, int seq, int rows, int per_seq)
{
    return per_seq ? (int64_t)seq * per_seq : (int64_t)row0 * s.H / rows + seq;
}

constexpr int LA_KEYS = 64;
constexpr int LA_PS = LA_KEYS + 8;      // row stride of the weights in shared memory

// grid (slices, row tiles, seqs), 8 RT warps.  A warp has 16 keys of a tile, 16 rows and half of the key's columns for the
// scores -- two warps exchange their halves' sums, and each goes on with eight keys -- and 64 / RT columns of all rows for the
// sums.  KS: 16-column steps of half a key; the warp's part of the queries stays in registers (KS = 0: any number, queries from
// shared memory).  The unrolled loops have no branches: behind the true width they repeat a step with zero queries, or make
// columns that nobody reads.
// Shared memory: ring of `stages` tiles of keys [64][ck + 8] | queries [16 RT][ck + 8] | weights [16 RT][LA_PS] | halves' sums
// [8 RT warps][32 lanes][4].  part [tile][slice][16 RT][cp + 4]: sums, then maximum (log 2 units) and denominator of each row.
template <int RT, int KS>
__global__ void __launch_bounds__(RT * 256, 1)
    latent_attn_kernel(const LatentShape s, const pg_batch bt, const bf16 *__restrict__ qx, const bf16 *__restrict__ cache, float *__restrict__ part, int per_seq,
                       int stages, int32_t *status, unsigned long long limit_ns)
{
    constexpr int NW = 8 * RT, ROWS = 16 * RT, VT = 512 / NW / 8;   // 8-column tiles of a warp (kv_rank up to 512)
    extern __shared__ __align__(128) unsigned char smem[];
    __shared__ __align__(8) uint64_t bars[4];
    __shared__ __align__(16) float red[RT][16][8];
    __shared__ volatile int abort_flag;
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    const int split = blockIdx.x, S = gridDim.x, tile = blockIdx.y, seq = blockIdx.z;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, r = lane >> 2, t = lane & 3;
    const int kh = warp & 1, kq = (warp >> 1) & 3, rt = warp >> 3;   // half of the columns, group of keys, row tile
    if (threadIdx.x == 0) {
        for (int i = 0; i < 4; i++) pg_mbar_init(pg_smem(bars) + 8 * i, 1);
        abort_flag = 0;
        pg_mbar_fence();
    }
    __syncthreads();
    asm volatile("griddepcontrol.wait;" ::: "memory");
    const int row0 = __ldcg(bt.d_seq_row0 + seq), T = seq_len(bt, seq), total = T * s.H, rr0 = tile * ROWS;
    const int64_t slot = __ldcg(bt.d_seq_slot + seq);
    if (T >= s.long_from || rr0 >= total) return;
    const int pos0 = __ldcg(bt.d_pos + row0);
    const Slices sl = slices_of(s, pos0, T, tile, ROWS, S);
    const int t0 = split * sl.chunk, t1 = min(sl.kmax, t0 + sl.chunk);
    if (t0 >= t1 || sl.kmax > s.cap) return;              // (positions outside the cache are recorded by latent_query_kernel)
    const int stride = s.ck * 2 + 16, stage = LA_KEYS * stride;
    const uint32_t ring = pg_smem(smem), qs = ring + stages * stage, ps = qs + ROWS * stride, xs = ps + ROWS * LA_PS * 2;
    const uint32_t bar = pg_smem(bars);
    const bf16 *keys = cache + slot * (int64_t)s.cap * s.ck;
    const int ntiles = (t1 - t0 + LA_KEYS - 1) / LA_KEYS;
    // every warp asks for some of a tile's rows (rows behind the slice repeat its last one and are masked)
    auto fetch = [&](int i) {
        const uint32_t at = ring + (uint32_t)(i % stages) * stage, on = bar + (uint32_t)(i % stages) * 8;
        if (threadIdx.x == 0) pg_mbar_expect(on, (uint32_t)LA_KEYS * s.ck * 2u);
        if (lane < LA_KEYS / NW) {
            const int x = warp * (LA_KEYS / NW) + lane;
            pg_bulk_load(at + (uint32_t)x * stride, keys + (int64_t)min(t0 + i * LA_KEYS + x, t1 - 1) * s.ck, (uint32_t)s.ck * 2u, on);
        }
    };
    for (int i = 0; i < stages && i < ntiles; i++) fetch(i);
    for (int x = warp; x < ROWS; x += NW) {
        const bf16 *src = qx + ((int64_t)row0 * s.H + min(rr0 + x, total - 1)) * s.ck;
        for (int e = lane * 8; e < s.ck; e += 256) pg_cp16(qs + (uint32_t)(x * stride + e * 2), src + e);
    }
    pg_cp_commit();
    pg_cp_wait<0>();
    __syncthreads();

    const int steps = s.ck / 16, half = (steps + 1) / 2, s0 = kh * half, sn = min(half, steps - s0);   // this warp's steps of the columns
    const uint32_t q_at = qs + (uint32_t)((rt * 16 + (lane & 15)) * stride + (lane >> 4) * 16 + s0 * 32);
    const uint32_t k_at = (uint32_t)((kq * 16 + (lane & 7) + ((lane >> 4) << 3)) * stride + ((lane >> 3) & 1) * 16 + s0 * 32);
    uint32_t qf[KS ? KS : 1][4];
#pragma unroll
    for (int i = 0; i < KS; i++) {
        qf[i][0] = qf[i][1] = qf[i][2] = qf[i][3] = 0u;
        if (i < sn) pg_ldsm4(qf[i], q_at + i * 32);
    }
    const int cw = ((s.cp + NW - 1) / NW + 15) & ~15, c0 = warp * cw, nv = max(0, min(cw, s.cp - c0)) / 8;   // this warp's columns of the sums
    const int lim0 = pos0 + min(rr0 + rt * 16 + r, total - 1) / s.H, lim1 = pos0 + min(rr0 + rt * 16 + r + 8, total - 1) / s.H;
    const float scale = s.scale * LOG2E;
    float o[RT][VT][4], m[RT][2], l0 = 0.0f, l1 = 0.0f;
#pragma unroll
    for (int x = 0; x < RT; x++) {
        m[x][0] = m[x][1] = -1e30f;                       // (finite: a row may see nothing of a slice)
#pragma unroll
        for (int i = 0; i < VT; i++)
#pragma unroll
            for (int j = 0; j < 4; j++) o[x][i][j] = 0.0f;
    }
    const uint32_t v_at = (uint32_t)(((lane & 7) + ((lane >> 3) & 1) * 8) * stride + ((lane >> 4) * 8 + c0) * 2);
    const uint32_t mine = xs + (uint32_t)(warp * 32 + lane) * 16, theirs = xs + (uint32_t)((warp ^ 1) * 32 + lane) * 16;
    bool ok = true;
    for (int it = 0; it < ntiles; it++) {
        ok = pg_mbar_wait(bar + (uint32_t)(it % stages) * 8, (uint32_t)(it / stages) & 1u, &abort_flag, status, limit_ns);
        const uint32_t kt = ring + (uint32_t)(it % stages) * stage;
        float sc[2][4] = {};
        if (KS) {
#pragma unroll
            for (int i = 0; i < KS; i++) {
                uint32_t b[4];
                pg_ldsm4(b, kt + k_at + (i < sn ? i : 0) * 32);
                pg_mma_bf16(sc[0], qf[i][0], qf[i][1], qf[i][2], qf[i][3], b[0], b[1]);
                pg_mma_bf16(sc[1], qf[i][0], qf[i][1], qf[i][2], qf[i][3], b[2], b[3]);
            }
        } else {
            for (int i = 0; i < sn; i++) {
                uint32_t a[4], b[4];
                pg_ldsm4(a, q_at + i * 32);
                pg_ldsm4(b, kt + k_at + i * 32);
                pg_mma_bf16(sc[0], a[0], a[1], a[2], a[3], b[0], b[1]);
                pg_mma_bf16(sc[1], a[0], a[1], a[2], a[3], b[2], b[3]);
            }
        }
        // eight keys each: the other half's sums of them from the neighbour
        {
            const float (&give)[4] = kh ? sc[0] : sc[1];
            asm volatile("st.shared.v4.f32 [%0], {%1, %2, %3, %4};" ::"r"(mine), "f"(give[0]), "f"(give[1]), "f"(give[2]), "f"(give[3]) : "memory");
        }
        // also: every warp is done with the tile before, so its slot can be filled again
        if (!__syncthreads_and(ok)) {
            ok = false;
            break;
        }
        if (it > 0 && it - 1 + stages < ntiles) fetch(it - 1 + stages);
        float sv[4];
        {
            const uint4 g = pg_lds128(theirs);
            const float got[4] = {__uint_as_float(g.x), __uint_as_float(g.y), __uint_as_float(g.z), __uint_as_float(g.w)};
            const int j0 = t0 + it * LA_KEYS + kq * 16 + kh * 8 + 2 * t;
#pragma unroll
            for (int j = 0; j < 4; j++) {
                const int key = j0 + (j & 1);
                const bool in = key < t1 && key <= (j < 2 ? lim0 : lim1);
                sv[j] = in ? ((kh ? sc[1][j] : sc[0][j]) + got[j]) * scale : -INFINITY;
            }
        }
        float b0 = fmaxf(sv[0], sv[1]), b1 = fmaxf(sv[2], sv[3]);
#pragma unroll
        for (int x = 1; x < 4; x <<= 1) {
            b0 = fmaxf(b0, __shfl_xor_sync(0xffffffffu, b0, x));
            b1 = fmaxf(b1, __shfl_xor_sync(0xffffffffu, b1, x));
        }
        if (t == 0) {
            red[rt][r][kq * 2 + kh] = b0;
            red[rt][r + 8][kq * 2 + kh] = b1;
        }
        __syncthreads();                                  // the maxima are there
        float f[RT][2];
        bool moved = false;
#pragma unroll
        for (int x = 0; x < RT; x++)
#pragma unroll
            for (int e = 0; e < 2; e++) {
                const float4 u = *reinterpret_cast<const float4 *>(red[x][r + 8 * e]), v = *reinterpret_cast<const float4 *>(red[x][r + 8 * e] + 4);
                const float top = fmaxf(m[x][e], fmaxf(fmaxf(fmaxf(u.x, u.y), fmaxf(u.z, u.w)), fmaxf(fmaxf(v.x, v.y), fmaxf(v.z, v.w))));
                f[x][e] = pg_ex2(m[x][e] - top);
                moved |= top > m[x][e];
                m[x][e] = top;
            }
        float m0 = m[0][0], m1 = m[0][1], f0 = f[0][0], f1 = f[0][1];
        if (RT == 2 && rt == 1) m0 = m[RT - 1][0], m1 = m[RT - 1][1], f0 = f[RT - 1][0], f1 = f[RT - 1][1];
        const float p0 = pg_ex2(sv[0] - m0), p1 = pg_ex2(sv[1] - m0), p2 = pg_ex2(sv[2] - m1), p3 = pg_ex2(sv[3] - m1);
        l0 = fmaf(l0, f0, p0 + p1);
        l1 = fmaf(l1, f1, p2 + p3);
        {
            const uint32_t at = ps + (uint32_t)((rt * 16 + r) * LA_PS + kq * 16 + kh * 8 + 2 * t) * 2;
            asm volatile("st.shared.u32 [%0], %1;" ::"r"(at), "r"(pg_pack_bf16(p0, p1)) : "memory");
            asm volatile("st.shared.u32 [%0], %1;" ::"r"(at + 8 * LA_PS * 2), "r"(pg_pack_bf16(p2, p3)) : "memory");
        }
        __syncthreads();                                  // the weights are there
        if (nv == 0) continue;
        if (__any_sync(0xffffffffu, moved)) {
#pragma unroll
            for (int x = 0; x < RT; x++)
#pragma unroll
                for (int i = 0; i < VT; i++) {
                    o[x][i][0] *= f[x][0];
                    o[x][i][1] *= f[x][0];
                    o[x][i][2] *= f[x][1];
                    o[x][i][3] *= f[x][1];
                }
        }
#pragma unroll
        for (int kk = 0; kk < LA_KEYS / 16; kk++) {
            uint32_t a[RT][4];
#pragma unroll
            for (int x = 0; x < RT; x++) pg_ldsm4(a[x], ps + (uint32_t)((x * 16 + (lane & 15)) * LA_PS + kk * 16 + (lane >> 4) * 8) * 2);
#pragma unroll
            for (int i = 0; i < VT; i += 2) {
                uint32_t b[4];
                pg_ldsm4_t(b, kt + v_at + (uint32_t)(kk * 16 * stride + (i < nv ? i : 0) * 16));
#pragma unroll
                for (int x = 0; x < RT; x++) {
                    pg_mma_bf16(o[x][i], a[x][0], a[x][1], a[x][2], a[x][3], b[0], b[1]);
                    pg_mma_bf16(o[x][i + 1], a[x][0], a[x][1], a[x][2], a[x][3], b[2], b[3]);
                }
            }
        }
    }
    if (!ok) {
        // copies that are still in flight get a bounded time to land before the shared memory goes
        const unsigned long long w0 = pg_globaltimer_ns();
        while (pg_globaltimer_ns() - w0 < 2000000ull) {
        }
        return;
    }
#pragma unroll
    for (int x = 1; x < 4; x <<= 1) {
        l0 += __shfl_xor_sync(0xffffffffu, l0, x);
        l1 += __shfl_xor_sync(0xffffffffu, l1, x);
    }
    __syncthreads();
    if (t == 0) {
        red[rt][r][kq * 2 + kh] = l0;
        red[rt][r + 8][kq * 2 + kh] = l1;
    }
    __syncthreads();
    const int ms = s.cp + 4;
    float *dst = part + ((first_tile(s, row0, seq, ROWS, per_seq) + tile) * S + split) * ROWS * ms;
#pragma unroll
    for (int x = 0; x < RT; x++)
#pragma unroll
        for (int e = 0; e < 2; e++) {
            float *row = dst + (size_t)(x * 16 + r + 8 * e) * ms;
#pragma unroll
            for (int i = 0; i < VT; i++)
                if (i < nv) *reinterpret_cast<float2 *>(row + c0 + i * 8 + 2 * t) = make_float2(o[x][i][2 * e], o[x][i][2 * e + 1]);
            if (warp == 0 && t == 0) {
                const float *g = red[x][r + 8 * e];
                *reinterpret_cast<float2 *>(row + s.cp) = make_float2(m[x][e], ((g[0] + g[1]) + (g[2] + g[3])) + ((g[4] + g[5]) + (g[6] + g[7])));
            }
        }
}

// grid (H, parts of 64 columns, groups of `group` <= 16 rows): adds the slices of its rows, then W_uv of its head, then the gate
constexpr int LV_T = 256;
constexpr int LV_SLICES = 64;
__global__ void __launch_bounds__(LV_T)
    latent_value_kernel(const LatentShape s, const pg_batch bt, const float *__restrict__ part, int per_seq, int S, int rows, int group,
                        const float *__restrict__ proj, int64_t ldp, bf16 *__restrict__ out, int64_t ldo)
{
    extern __shared__ __align__(128) unsigned char smem[];   // [16][cp + 8]
    __shared__ float weight[16][LV_SLICES];
    __shared__ int64_t base[16];
    __shared__ int used[16];
    const int h = blockIdx.x, m0 = blockIdx.z * group, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int c = blockIdx.y * 64 + warp * 8;
    Weights8<16> w;
    // (rows of W_uv behind the head's last one belong to the next head or are padding; their products are dropped)
    if (c < s.V) w.ask(s.uv + ((int64_t)h * s.V + c) * s.cp, s.cp, s.cp, lane);
    pg_pdl_begin();
    bf16 *sa = reinterpret_cast<bf16 *>(smem);
    const int ld = s.cp + 8, ms = s.cp + 4;
    for (int x = warp; x < 16; x += LV_T / 32) {
        // a warp per row: where its slices are, and their weights
        const int m = m0 + x;
        int n = 0;
        if (x < group && m < bt.rows) {
            const int seq = __ldcg(bt.d_row_seq + m), row0 = __ldcg(bt.d_seq_row0 + seq), T = seq_len(bt, seq);
            const int pos0 = __ldcg(bt.d_pos + row0), rr = (m - row0) * s.H + h, tile = rr / rows;
            const Slices sl = slices_of(s, pos0, T, tile, rows, S);
            if (T < s.long_from && sl.kmax <= s.cap) {
                n = sl.used;
                const int64_t at = ((first_tile(s, row0, seq, rows, per_seq) + tile) * S * rows + rr % rows) * (int64_t)ms;
                float2 ml[LV_SLICES / 32];
                float top = -INFINITY, l = 0.0f;
#pragma unroll
                for (int i = 0; i < LV_SLICES / 32; i++) {
                    const int k = i * 32 + lane;
                    ml[i] = k < n ? __ldcg(reinterpret_cast<const float2 *>(part + at + (int64_t)k * rows * ms + s.cp)) : make_float2(-INFINITY, 0.0f);
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
                for (int i = 0; i < LV_SLICES / 32; i++) weight[x][i * 32 + lane] = ml[i].x * inv;
                if (lane == 0) base[x] = at;
            }
        }
        if (lane == 0) used[x] = n;
    }
    __syncthreads();
    const int quads = s.cp / 4;
    for (int i = threadIdx.x; i < 16 * quads; i += LV_T) {
        const int x = i / quads, k4 = (i - x * quads) * 4, n = used[x];
        float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
        const float *src = part + (n ? base[x] : 0) + k4;
        for (int k0 = 0; k0 < n; k0 += 12) {              // twelve loads in flight; behind the last slice its weight is 0
            float4 v[12];
#pragma unroll
            for (int k = 0; k < 12; k++) v[k] = __ldcg(reinterpret_cast<const float4 *>(src + (int64_t)min(k0 + k, n - 1) * rows * ms));
#pragma unroll
            for (int k = 0; k < 12; k++) {
                const float f = k0 + k < n ? weight[x][k0 + k] : 0.0f;
                a.x = fmaf(f, v[k].x, a.x), a.y = fmaf(f, v[k].y, a.y), a.z = fmaf(f, v[k].z, a.z), a.w = fmaf(f, v[k].w, a.w);
            }
        }
        *reinterpret_cast<uint2 *>(sa + x * ld + k4) = make_uint2(pg_pack_bf16(a.x, a.y), pg_pack_bf16(a.z, a.w));
    }
    const int r = lane >> 2, t = lane & 3;
    float gate[2][2];
#pragma unroll
    for (int half = 0; half < 2; half++)
#pragma unroll
        for (int j = 0; j < 2; j++) {
            const int col = c + 2 * t + j;
            gate[half][j] = used[r + 8 * half] && col < s.V ? __ldcg(proj + (int64_t)(m0 + r + 8 * half) * ldp + s.at_gate + h * s.V + col) : 0.0f;
        }
    __syncthreads();
    if (c >= s.V) return;
    float d[4] = {};
    w.times(d, pg_smem(sa), ld, lane);
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
    for (int h = warp; h < s.H + s.own; h += 8) {
        if (h == s.H) {
            append(s, row + s.at_kv, pos, cache + (slot * s.cap + pos) * s.ck, lane);
        } else {
            const float *src = row + h * (s.D + s.R);
            bf16 *dst = q + ((int64_t)m * s.H + h) * qd;
            for (int c = 2 * lane; c < dn; c += 64)
                *reinterpret_cast<uint32_t *>(dst + c) = pg_pack_bf16(c < s.D ? __ldcg(src + c) : 0.0f, c + 1 < s.D ? __ldcg(src + c + 1) : 0.0f);
            rotate(s, src + s.D, pos, dst + dn, qd - dn, lane);
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
        if (threadIdx.x < 32) append(s, proj + (int64_t)m * ldp + s.at_kv, pos, cache + (slot * s.cap + pos) * s.ck, lane);
        return;
    }
    const float *src = proj + (int64_t)m * ldp + h * (s.D + s.R);
    float *dst = qx + ((int64_t)m * s.H + h) * s.ck;
    for (int i = threadIdx.x; i < s.dk; i += 128) sm[i] = i < s.D ? __ldcg(src + i) : 0.0f;
    if (threadIdx.x < 32) rotate(s, src + s.D, pos, dst + s.cp, s.rp, lane);
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

constexpr int LA_SMEM = 220 * 1024;
int attn_rows(const LatentShape &s) { return s.H > 16 ? 32 : 16; }
int attn_smem(const LatentShape &s, int stages) { return (stages * LA_KEYS + attn_rows(s)) * (s.ck * 2 + 16) + attn_rows(s) * (LA_PS * 2 + 256); }

// slices of the context: about one CTA per SM, none shorter than 64 positions of a full cache
int slices(const pg_ctx *ctx, int64_t units, int64_t cap)
{
    int64_t S = std::max<int64_t>(1, (int64_t)ctx->sm_count / std::max<int64_t>(1, units));
    S = std::min<int64_t>(S, std::max<int64_t>(1, cap / LA_KEYS));
    return (int)std::min<int64_t>(S, LV_SLICES);
}

template <int RT>
int32_t launch_attn(pg_ctx *ctx, const LatentShape &s, const pg_batch *batch, dim3 grid, const bf16 *q, const bf16 *cache, float *part, int per_seq, int stages)
{
    auto go = [&](auto kern, std::atomic<uint64_t> &set) -> int32_t {
        PG_CUDA(pg_max_smem_once(kern, LA_SMEM, ctx->device, set));
        return launch_pdl(ctx, kern, grid, dim3(RT * 256), (size_t)attn_smem(s, stages), s, *batch, q, cache, part, per_seq, stages, ctx->d_status,
                          ctx->wait_limit_ns);
    };
    static std::atomic<uint64_t> set[5] = {};
    if (s.ck <= 96) return go(latent_attn_kernel<RT, 3>, set[0]);
    if (s.ck <= 160) return go(latent_attn_kernel<RT, 5>, set[1]);
    if (s.ck <= 320) return go(latent_attn_kernel<RT, 10>, set[2]);
    if (s.ck <= 576) return go(latent_attn_kernel<RT, 18>, set[3]);
    return go(latent_attn_kernel<RT, 0>, set[4]);
}

int32_t check(const pg_latent *p, const pg_batch *batch, int64_t ldp, int64_t ldo)
{
    PG_REQUIRE(p && batch && p->d_rot && p->d_uk && p->d_uv && p->d_q && (p->d_norm || !p->own), "latent attention: null pointer");
    PG_REQUIRE(p->heads > 0 && p->dim > 0 && p->dim <= 512 && p->rot_dim >= 0 && p->rot_dim % 2 == 0 && p->vdim > 0 && p->kv_rank > 0 && p->kv_rank <= 512 &&
                   p->cap > 0 && p->heads <= 65534,
               "latent attention: bad shape (dim %d and latent %d at most 512, an even rot_dim %d)", p->dim, p->kv_rank, p->rot_dim);
    const LatentShape s = shape_of(p);
    PG_REQUIRE(attn_smem(s, 2) <= LA_SMEM, "latent attention: a key of %d and %d columns is too wide", s.C, s.R);
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
    const int64_t tiles = (max_rows * s.H + attn_rows(s) - 1) / attn_rows(s) + max_seqs;
    return std::max<int64_t>(tiles, 2 * ctx->sm_count) * attn_rows(s) * (s.cp + 4);
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
    const int rows = attn_rows(s);
    const int64_t tiles = (short_len * s.H + rows - 1) / rows;
    PG_REQUIRE(tiles <= 65535, "latent attention: too many rows in one sequence");
    // the numbering of tiles that needs fewer of them, and as many slices as then have room
    const int64_t dense = (int64_t)batch->rows * s.H / rows + batch->seqs, even = tiles * batch->seqs;
    const int per_seq = even <= dense ? (int)tiles : 0;
    const int64_t room = p->part_floats / ((int64_t)rows * (s.cp + 4)) / std::min(even, dense);
    PG_REQUIRE(room >= 1, "latent attention: the step has more rows than d_part has room for");
    const int S = (int)std::min<int64_t>(room, slices(ctx, std::max<int64_t>(tiles, (short_rows * s.H + rows - 1) / rows), s.cap));
    int stages = 4;
    while (stages > 2 && attn_smem(s, stages) > LA_SMEM) stages--;
    const dim3 grid((unsigned)S, (unsigned)tiles, (unsigned)batch->seqs);
    rc = rows == 32 ? launch_attn<2>(ctx, s, batch, grid, q, cache, p->d_part, per_seq, stages) : launch_attn<1>(ctx, s, batch, grid, q, cache, p->d_part, per_seq, stages);
    if (rc != PG_OK) return rc;
    // groups of rows small enough for about one CTA per SM
    const unsigned parts64 = (unsigned)((s.V + 63) / 64);
    int group = 16;
    while (group > 1 && (int64_t)s.H * parts64 * ((batch->rows + group - 1) / group) < ctx->sm_count * 3 / 4) group /= 2;
    const int64_t groups = (batch->rows + group - 1) / group;
    PG_REQUIRE(groups <= 65535 && parts64 <= 65535, "latent attention: too many rows");
    return launch_pdl(ctx, latent_value_kernel, dim3((unsigned)s.H, parts64, (unsigned)groups), dim3(LV_T), (size_t)(16 * (s.cp + 8) * 2), s, *batch,
                      (const float *)p->d_part, per_seq, S, rows, group, d_proj, ldp, (bf16 *)d_out, ldo);
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
