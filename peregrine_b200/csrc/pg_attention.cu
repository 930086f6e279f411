// Causal attention for prompts and decoding over a cache per slot and key/value head.  Each of these may be there or not:
// per-head query / key norms, a query temperature, a softmax sink, a bias that grows with the distance (slope per head), and
// a mask of chunks (a position sees its own chunk only; the cache is then a ring of whole chunks).
//
//   bf16, one token per sequence    attn_step_kernel: streams the cache once.  A CTA has one slice of the context of one
//                                   (sequence, key/value head); it normalises the group's queries itself, the CTA with
//                                   the newest position also normalises and appends the key and the value.  Scores and
//                                   sums run on mma.sync with the group's heads as the 16 rows; each warp streams keys
//                                   through its own ring.  The last CTA of a (sequence, head) to finish merges the slices.
//   bf16, longer portions           attn_prep_kernel (norms, temperature, append), then the tcgen05 kernel of
//                                   csrc/pg_attention_tc.cu, or attn_prompt_kernel (mma.sync) for short portions and for
//                                   head widths that the former does not take.  Rows of a tile are (token, head of the
//                                   group) pairs, which share the keys and values.
//   f32                             attn_prep_kernel, then attn_f32_kernel (one CTA per token and head, FFMA)
//
// The sink is a score of 0 without a value: the running maximum starts at 0 and exp(-max) joins the denominator.
#include <math.h>

#include <algorithm>

#include "pg_async.cuh"
#include "pg_attention.cuh"

namespace {

constexpr float LOG2E = 1.4426950408889634f;

__device__ __forceinline__ float temperature(const AttnShape &s, int pos)
{
    if (s.every <= 0.0f) return 1.0f;
    return 1.0f + s.coef * logf(floorf(__fdiv_rn((float)(pos + 1), s.every)) + 1.0f);
}

// One warp: dst = rms_norm(src[0 .. D)) * w * mul, or src * mul where w is null; columns D .. dp are zero (D <= 256).
template <typename TA>
__device__ __forceinline__ void head_norm(const float *src, const float *__restrict__ w, int D, int dp, float eps, float mul, TA *dst, int lane)
{
    float x[8], ss = 0.0f;
#pragma unroll
    for (int i = 0; i < 8; i++) {
        x[i] = i * 32 + lane < D ? __ldcg(src + i * 32 + lane) : 0.0f;
        ss += x[i] * x[i];
    }
    ss = pg_warp_sum(ss);
    const float inv = w ? __fdiv_rn(1.0f, sqrtf(__fdiv_rn(ss, (float)D) + eps)) : 1.0f;
#pragma unroll
    for (int i = 0; i < 8; i++) {
        const int c = i * 32 + lane;
        if (c < dp) pg_put(dst + c, c < D ? x[i] * inv * (w ? __ldg(w + c) : 1.0f) * mul : 0.0f);
    }
}

// four columns per lane, four heads per warp with their loads in flight together (widths up to 128, all multiples of four)
__device__ __forceinline__ void put4(float *p, const float4 &v) { *reinterpret_cast<float4 *>(p) = v; }
__device__ __forceinline__ void put4(bf16 *p, const float4 &v) { *reinterpret_cast<uint2 *>(p) = make_uint2(pg_pack_bf16(v.x, v.y), pg_pack_bf16(v.z, v.w)); }
template <typename TA>
__device__ __forceinline__ void prep_heads4(const AttnShape &s, const float *row, int64_t q_at, int64_t kv_at, float mul, TA *q, TA *kc, TA *vc, int warp, int lane)
{
    const int n = s.H + 2 * s.G, c = 4 * lane;
    auto norm4 = [&](const float *w, bool in) { return w && in && c < s.D ? __ldg(reinterpret_cast<const float4 *>(w) + lane) : make_float4(1.f, 1.f, 1.f, 1.f); };
    const float4 wq = norm4(s.qn, true), wk = norm4(s.kn, true);
    for (int i0 = warp; i0 < n; i0 += 32) {
        float4 x[4];
#pragma unroll
        for (int u = 0; u < 4; u++) {
            const int i = i0 + 8 * u;
            const float *src = i < s.H + s.G ? row + i * s.D : row + (int64_t)(s.H + s.G) * s.D + (int64_t)(i - s.H - s.G) * s.V;
            x[u] = i < n && c < (i < s.H + s.G ? s.D : s.V) ? __ldcg(reinterpret_cast<const float4 *>(src) + lane) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
#pragma unroll
        for (int u = 0; u < 4; u++) {
            const int i = i0 + 8 * u;
            if (i >= n) break;
            if (i >= s.H + s.G) {
                if (c < s.vp) put4(vc + (kv_at + (int64_t)(i - s.H - s.G) * s.cap) * s.vp + c, x[u]);
                continue;
            }
            const bool query = i < s.H;
            float f = query ? mul : 1.0f;
            float4 w = make_float4(1.f, 1.f, 1.f, 1.f);
            if (query ? s.qn : s.kn) {
                f *= __fdiv_rn(1.0f, sqrtf(__fdiv_rn(pg_warp_sum((x[u].x * x[u].x + x[u].y * x[u].y) + (x[u].z * x[u].z + x[u].w * x[u].w)), (float)s.D) + s.eps));
                w = query ? wq : wk;
            }
            const float4 y = make_float4(x[u].x * f * w.x, x[u].y * f * w.y, x[u].z * f * w.z, x[u].w * f * w.w);
            if (c < s.dp) put4(query ? q + (q_at + i) * s.dp + c : kc + (kv_at + (int64_t)(i - s.H) * s.cap) * s.dp + c, y);
        }
    }
}

// a CTA per token; wide: prep_heads4 fits
template <typename TA>
__global__ void __launch_bounds__(256)
    attn_prep_kernel(const AttnShape s, const pg_batch bt, const float *__restrict__ proj, int64_t ldp, TA *__restrict__ q, TA *kc, TA *vc, int wide, int32_t *status)
{
    pg_pdl_begin();
    const int m = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int pos = __ldcg(bt.d_pos + m);
    const int64_t slot = __ldcg(bt.d_seq_slot + __ldcg(bt.d_row_seq + m));
    if ((unsigned)pos >= (unsigned)s.limit) {   // outside the cache: record it, touch nothing
        if (threadIdx.x == 0) atomicExch(status, (int32_t)PG_ERR_INVALID);
        return;
    }
    const float *row = proj + (int64_t)m * ldp;
    const float mul = temperature(s, pos);
    const int at = attn_row(s, pos);
    if (wide) {
        prep_heads4(s, row, (int64_t)m * s.H, slot * s.G * s.cap + at, mul, q, kc, vc, warp, lane);
        return;
    }
    for (int i = warp; i < s.H + 2 * s.G; i += 8) {
        if (i < s.H) {
            head_norm(row + i * s.D, s.qn, s.D, s.dp, s.eps, mul, q + ((int64_t)m * s.H + i) * s.dp, lane);
        } else if (i < s.H + s.G) {
            const int g = i - s.H;
            head_norm(row + i * s.D, s.kn, s.D, s.dp, s.eps, 1.0f, kc + ((slot * s.G + g) * s.cap + at) * s.dp, lane);
        } else {
            const int g = i - s.H - s.G;
            const float *src = row + (int64_t)(s.H + s.G) * s.D + (int64_t)g * s.V;
            TA *dst = vc + ((slot * s.G + g) * s.cap + at) * s.vp;
            for (int c = lane; c < s.vp; c += 32) pg_put(dst + c, c < s.V ? __ldcg(src + c) : 0.0f);
        }
    }
}

// ---- f32: grid (H, rows) -----------------------------------------------------------------------------------------
constexpr int AF_T = 128;
__global__ void __launch_bounds__(AF_T)
    attn_f32_kernel(const AttnShape s, const pg_batch bt, const float *__restrict__ q, const float *__restrict__ kc, const float *__restrict__ vc,
                    float *__restrict__ out, int64_t ldo)
{
    extern __shared__ float sm[];   // q[dp] | p[AF_T]
    __shared__ float red[8];
    pg_pdl_begin();
    const int h = blockIdx.x, m = blockIdx.y, g = h / s.rep, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int pos = __ldcg(bt.d_pos + m);
    const int64_t slot = __ldcg(bt.d_seq_slot + __ldcg(bt.d_row_seq + m));
    if ((unsigned)pos >= (unsigned)s.limit) return;
    float *sq = sm, *sp = sm + s.dp;
    for (int i = tid; i < s.dp; i += AF_T) sq[i] = __ldcg(q + ((int64_t)m * s.H + h) * s.dp + i);
    const int low = attn_low(s, pos);
    const int64_t first = (slot * s.G + g) * (int64_t)s.cap + attn_row(s, low) - low;   // row of position 0, as it were
    const float *kb = kc + first * s.dp, *vb = vc + first * s.vp;
    const float slope = s.slopes ? __ldg(s.slopes + h) : 0.0f;
    constexpr int NV = 8;                      // value columns per thread (vdim <= 1024)
    float acc[NV], mx = s.sink ? 0.0f : -INFINITY, l = s.sink ? 1.0f : 0.0f;
#pragma unroll
    for (int i = 0; i < NV; i++) acc[i] = 0.0f;
    __syncthreads();
    for (int j0 = low; j0 <= pos; j0 += AF_T) {
        const int j = j0 + tid;
        float sc = -INFINITY;
        if (j <= pos) {
            // dp is a multiple of 16, zero behind D
            float d[8] = {};
            for (int i = 0; i < s.dp; i += 8) {
                const float4 a = __ldcg(reinterpret_cast<const float4 *>(kb + (int64_t)j * s.dp + i));
                const float4 b = __ldcg(reinterpret_cast<const float4 *>(kb + (int64_t)j * s.dp + i + 4));
                d[0] = fmaf(sq[i], a.x, d[0]), d[1] = fmaf(sq[i + 1], a.y, d[1]), d[2] = fmaf(sq[i + 2], a.z, d[2]), d[3] = fmaf(sq[i + 3], a.w, d[3]);
                d[4] = fmaf(sq[i + 4], b.x, d[4]), d[5] = fmaf(sq[i + 5], b.y, d[5]), d[6] = fmaf(sq[i + 6], b.z, d[6]), d[7] = fmaf(sq[i + 7], b.w, d[7]);
            }
            sc = (((d[0] + d[1]) + (d[2] + d[3])) + ((d[4] + d[5]) + (d[6] + d[7]))) * s.scale - slope * (float)(pos - j);
        }
        float bm = sc;
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) bm = fmaxf(bm, __shfl_xor_sync(0xffffffffu, bm, o));
        if (lane == 0) red[warp] = bm;
        __syncthreads();
        bm = fmaxf(fmaxf(red[0], red[1]), fmaxf(red[2], red[3]));
        const float mn = fmaxf(mx, bm), corr = expf(mx - mn), p = expf(sc - mn);
        sp[tid] = p;
        const float ps = pg_warp_sum(p);
        if (lane == 0) red[4 + warp] = ps;
        __syncthreads();
        l = l * corr + ((red[4] + red[5]) + (red[6] + red[7]));
        mx = mn;
        const int n = min(AF_T, pos + 1 - j0);
#pragma unroll
        for (int i = 0; i < NV; i++) {
            const int c = tid + i * AF_T;
            if (c >= s.V) break;
            float a = acc[i] * corr;
            for (int k = 0; k < n; k++) a = fmaf(sp[k], __ldcg(vb + (int64_t)(j0 + k) * s.vp + c), a);
            acc[i] = a;
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < NV; i++) {
        const int c = tid + i * AF_T;
        if (c < s.V) out[(int64_t)m * ldo + (int64_t)h * s.V + c] = __fdiv_rn(acc[i], l);
    }
}

// ---- bf16 tiles --------------------------------------------------------------------------------------------------
// 16-byte address of (row, 8-element group) in a tile whose rows are `stride` bytes apart (16 mod 32 words: no conflicts)
__device__ __forceinline__ uint32_t tile_at(uint32_t base, int stride, int row, int elem) { return base + (uint32_t)(row * stride + elem * 2); }

// S[16 x 16 keys] of one row tile: two 8-key accumulators
template <int DC>
__device__ __forceinline__ void scores16(const uint32_t (&qf)[DC][4], int nk, uint32_t kt, int kstride, int key0, int lane, float (&s0)[4], float (&s1)[4])
{
    const int row = key0 + (lane & 7) + ((lane >> 4) << 3), el = ((lane >> 3) & 1) * 8;
#pragma unroll
    for (int i = 0; i < DC; i++) {
        if (i < nk) {
            uint32_t b[4];
            pg_ldsm4(b, tile_at(kt, kstride, row, i * 16 + el));
            pg_mma_bf16(s0, qf[i][0], qf[i][1], qf[i][2], qf[i][3], b[0], b[1]);
            pg_mma_bf16(s1, qf[i][0], qf[i][1], qf[i][2], qf[i][3], b[2], b[3]);
        }
    }
}
// O[16 x V] += P[16 x 16 keys] V
template <int VC>
__device__ __forceinline__ void values16(float (&o)[VC][4], int nv, const uint32_t (&p)[4], uint32_t vt, int vstride, int key0, int lane)
{
    const int row = key0 + (lane & 7) + ((lane >> 3) & 1) * 8, el = (lane >> 4) * 8;
#pragma unroll
    for (int i = 0; i < VC; i += 2) {
        if (i < nv) {
            uint32_t b[4];
            pg_ldsm4_t(b, tile_at(vt, vstride, row, i * 8 + el));
            pg_mma_bf16(o[i], p[0], p[1], p[2], p[3], b[0], b[1]);
            pg_mma_bf16(o[i + 1], p[0], p[1], p[2], p[3], b[2], b[3]);
        }
    }
}

// ---- prompts: grid (row tiles, G, seqs) --------------------------------------------------------------------------
constexpr int AP_KEYS = 64;

template <int DC, int VC, int WARPS>
__global__ void __launch_bounds__(WARPS * 32)
    attn_prompt_kernel(const AttnShape s, const pg_batch bt, const bf16 *__restrict__ q, const bf16 *__restrict__ kc, const bf16 *__restrict__ vc,
                       bf16 *__restrict__ out, int64_t ldo)
{
    extern __shared__ __align__(128) unsigned char smem[];
    pg_pdl_begin();
    const int g = blockIdx.y, seq = blockIdx.z, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, r = lane >> 2, t = lane & 3;
    const int row0 = __ldcg(bt.d_seq_row0 + seq), T = __ldcg(bt.d_seq_row0 + seq + 1) - row0;
    const int total = T * s.rep;
    const int tile = gridDim.x - 1 - blockIdx.x;          // long tiles first
    const int rr0 = tile * WARPS * 16;
    if (rr0 >= total) return;
    const int pos0 = __ldcg(bt.d_pos + row0);
    const int64_t slot = __ldcg(bt.d_seq_slot + seq);
    const bf16 *kb = kc + (slot * s.G + g) * (int64_t)s.cap * s.dp, *vb = vc + (slot * s.G + g) * (int64_t)s.cap * s.vp;
    const int last = min(rr0 + WARPS * 16, total) - 1;
    const int kmax = pos0 + last / s.rep + 1;             // the tile sees keys kmin .. kmax - 1
    if (kmax > s.limit) return;                           // recorded by attn_prep_kernel
    const int kmin = attn_low(s, pos0 + rr0 / s.rep);
    const int low_last = attn_low(s, kmax - 1);           // the first key of its last row
    const int nk = s.dp / 16, nv = s.vp / 8;
    const int kstride = s.dp * 2 + 16, vstride = s.vp * 2 + 16;
    const uint32_t ks = pg_smem(smem), vs = ks + 2 * AP_KEYS * kstride;

    const int my0 = rr0 + warp * 16 + r, my1 = my0 + 8;
    const int c0 = min(my0, total - 1), c1 = min(my1, total - 1);
    const int lim0 = pos0 + c0 / s.rep, lim1 = pos0 + c1 / s.rep;    // last key of the lane's two rows
    const int low0 = attn_low(s, lim0), low1 = attn_low(s, lim1);    // and the first
    const float bias0 = s.slopes ? __ldg(s.slopes + g * s.rep + c0 % s.rep) * LOG2E : 0.0f, bias1 = s.slopes ? __ldg(s.slopes + g * s.rep + c1 % s.rep) * LOG2E : 0.0f;
    uint32_t qf[DC][4];
    {
        const bf16 *q0 = q + ((int64_t)(row0 + c0 / s.rep) * s.H + g * s.rep + c0 % s.rep) * s.dp + 2 * t;
        const bf16 *q1 = q + ((int64_t)(row0 + c1 / s.rep) * s.H + g * s.rep + c1 % s.rep) * s.dp + 2 * t;
#pragma unroll
        for (int i = 0; i < DC; i++) {
            if (i < nk) {
                qf[i][0] = __ldcg(reinterpret_cast<const uint32_t *>(q0 + i * 16));
                qf[i][1] = __ldcg(reinterpret_cast<const uint32_t *>(q1 + i * 16));
                qf[i][2] = __ldcg(reinterpret_cast<const uint32_t *>(q0 + i * 16 + 8));
                qf[i][3] = __ldcg(reinterpret_cast<const uint32_t *>(q1 + i * 16 + 8));
            }
        }
    }
    auto fetch = [&](int buf, int j0) {
        const int kw = s.dp / 8, vw = s.vp / 8, e0 = attn_row(s, j0), left = kmax - 1 - j0;
        auto row_of = [&](int k) {                        // (at most one turn of the ring: it holds more than a tile's keys)
            int e = e0 + min(k, left);
            while (e >= s.cap) e -= s.cap;
            return (int64_t)e;
        };
        for (int i = threadIdx.x; i < AP_KEYS * kw; i += WARPS * 32) {
            const int k = i / kw, e = (i - k * kw) * 8;
            pg_cp16(tile_at(ks + buf * AP_KEYS * kstride, kstride, k, e), kb + row_of(k) * s.dp + e);
        }
        for (int i = threadIdx.x; i < AP_KEYS * vw; i += WARPS * 32) {
            const int k = i / vw, e = (i - k * vw) * 8;
            pg_cp16(tile_at(vs + buf * AP_KEYS * vstride, vstride, k, e), vb + row_of(k) * s.vp + e);
        }
        pg_cp_commit();
    };
    float o[VC][4];
#pragma unroll
    for (int i = 0; i < VC; i++)
#pragma unroll
        for (int j = 0; j < 4; j++) o[i][j] = 0.0f;
    const float sl = s.scale * LOG2E;                     // scores in units of log 2
    // (a row may see no key of a chunk in front of its own: the maxima start finite, so that exp2(-inf - m) is 0)
    float m0 = s.sink ? 0.0f : -1e30f, m1 = m0, l0 = 0.0f, l1 = 0.0f;
    fetch(0, kmin);
    int buf = 0;
    for (int j0 = kmin; j0 < kmax; j0 += AP_KEYS, buf ^= 1) {
        if (j0 + AP_KEYS < kmax) {
            fetch(buf ^ 1, j0 + AP_KEYS);
            pg_cp_wait<1>();
        } else {
            pg_cp_wait<0>();
        }
        __syncthreads();
        const uint32_t kt = ks + buf * AP_KEYS * kstride, vt = vs + buf * AP_KEYS * vstride;
        float sc[AP_KEYS / 8][4];
#pragma unroll
        for (int n = 0; n < AP_KEYS / 8; n++)
#pragma unroll
            for (int j = 0; j < 4; j++) sc[n][j] = 0.0f;
#pragma unroll
        for (int n = 0; n < AP_KEYS / 16; n++) scores16<DC>(qf, nk, kt, kstride, n * 16, lane, sc[2 * n], sc[2 * n + 1]);
        float b0 = -INFINITY, b1 = -INFINITY;
        const bool edge = j0 + AP_KEYS - 1 > pos0 + rr0 / s.rep || j0 < low_last;   // some row of the tile does not see all of these keys
#pragma unroll
        for (int n = 0; n < AP_KEYS / 8; n++)
#pragma unroll
            for (int j = 0; j < 2; j++) {
                const int key = j0 + n * 8 + 2 * t + j;
                sc[n][j] = (!edge || (key <= lim0 && key >= low0)) ? fmaf(bias0, (float)(key - lim0), sc[n][j] * sl) : -INFINITY;
                sc[n][2 + j] = (!edge || (key <= lim1 && key >= low1)) ? fmaf(bias1, (float)(key - lim1), sc[n][2 + j] * sl) : -INFINITY;
                b0 = fmaxf(b0, sc[n][j]);
                b1 = fmaxf(b1, sc[n][2 + j]);
            }
#pragma unroll
        for (int x = 1; x < 4; x <<= 1) {
            b0 = fmaxf(b0, __shfl_xor_sync(0xffffffffu, b0, x));
            b1 = fmaxf(b1, __shfl_xor_sync(0xffffffffu, b1, x));
        }
        const float n0 = fmaxf(m0, b0), n1 = fmaxf(m1, b1);
        const float f0 = exp2f(m0 - n0), f1 = exp2f(m1 - n1);
        m0 = n0;
        m1 = n1;
        l0 *= f0;
        l1 *= f1;
#pragma unroll
        for (int i = 0; i < VC; i++) {
            o[i][0] *= f0;
            o[i][1] *= f0;
            o[i][2] *= f1;
            o[i][3] *= f1;
        }
#pragma unroll
        for (int n = 0; n < AP_KEYS / 16; n++) {
            float p[8];
#pragma unroll
            for (int j = 0; j < 2; j++) {
                p[j] = exp2f(sc[2 * n][j] - m0);
                p[2 + j] = exp2f(sc[2 * n][2 + j] - m1);
                p[4 + j] = exp2f(sc[2 * n + 1][j] - m0);
                p[6 + j] = exp2f(sc[2 * n + 1][2 + j] - m1);
                l0 += p[j] + p[4 + j];
                l1 += p[2 + j] + p[6 + j];
            }
            const uint32_t pf[4] = {pg_pack_bf16(p[0], p[1]), pg_pack_bf16(p[2], p[3]), pg_pack_bf16(p[4], p[5]), pg_pack_bf16(p[6], p[7])};
            values16<VC>(o, nv, pf, vt, vstride, n * 16, lane);
        }
        __syncthreads();
    }
#pragma unroll
    for (int x = 1; x < 4; x <<= 1) {
        l0 += __shfl_xor_sync(0xffffffffu, l0, x);
        l1 += __shfl_xor_sync(0xffffffffu, l1, x);
    }
    if (s.sink) {
        l0 += exp2f(-m0);
        l1 += exp2f(-m1);
    }
    const float i0 = __fdiv_rn(1.0f, l0), i1 = __fdiv_rn(1.0f, l1);
#pragma unroll
    for (int h = 0; h < 2; h++) {
        const int rr = h ? my1 : my0;
        if (rr >= total) continue;
        bf16 *dst = out + (int64_t)(row0 + rr / s.rep) * ldo + (int64_t)(g * s.rep + rr % s.rep) * s.V;
        const float inv = h ? i1 : i0;
#pragma unroll
        for (int i = 0; i < VC; i++) {
            const int c = i * 8 + 2 * t;
            if (c < s.V) pg_put(dst + c, o[i][2 * h] * inv);
            if (c + 1 < s.V) pg_put(dst + c + 1, o[i][2 * h + 1] * inv);
        }
    }
}

// ---- one token per sequence: grid (slices, G, rows), 4 warps ------------------------------------------------------
constexpr int AS_WARPS = 4, AS_STAGES = 3, AS_SLICES = 64;

// part [rows][G][slices][16][vp + 4]: sums, then maximum (log 2 units) and denominator of each head
template <int DC, int VC, bool FUSED>
__global__ void __launch_bounds__(AS_WARPS * 32)
    attn_step_kernel(const AttnShape s, const pg_batch bt, const float *__restrict__ proj, int64_t ldp, const bf16 *__restrict__ q, bf16 *kc, bf16 *vc,
                     float *part, int32_t *tickets, bf16 *__restrict__ out, int64_t ldo, int32_t *status, unsigned long long limit_ns)
{
    extern __shared__ __align__(128) unsigned char smem[];
    __shared__ __align__(8) uint64_t bars[AS_WARPS * AS_STAGES];
    __shared__ float weight[16][AS_SLICES];
    __shared__ float denom[16];
    __shared__ int last_in;
    __shared__ volatile int abort_flag;
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    const int split = blockIdx.x, S = gridDim.x, ht = FUSED ? 0 : blockIdx.y / s.G, g = FUSED ? blockIdx.y : blockIdx.y % s.G, b = blockIdx.z;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, r = lane >> 2, t = lane & 3;
    const int kstride = s.dp * 2 + 16, vstride = s.vp * 2 + 16, stage = 16 * (kstride + vstride);
    const uint32_t ring = pg_smem(smem) + (uint32_t)warp * AS_STAGES * stage, bar = pg_smem(bars) + (uint32_t)warp * AS_STAGES * 8;
    bf16 *qs = reinterpret_cast<bf16 *>(smem + AS_WARPS * AS_STAGES * stage);   // [16][dp + 8]
    bf16 *k_new = qs + 16 * (s.dp + 8), *v_new = k_new + s.dp;                  // the newest position's key and value
    float *mg = reinterpret_cast<float *>(smem);                                // the merge reuses the rings
    if (threadIdx.x == 0) {
        for (int i = 0; i < AS_WARPS * AS_STAGES; i++) pg_mbar_init(pg_smem(bars) + 8 * i, 1);
        abort_flag = 0;
        pg_mbar_fence();
    }
    const int heads = min(16, s.rep - ht * 16), h0 = g * s.rep + ht * 16;
    for (int i = threadIdx.x; i < (16 - heads) * (s.dp + 8) / 2; i += AS_WARPS * 32) reinterpret_cast<uint32_t *>(qs + heads * (s.dp + 8))[i] = 0u;
    __syncthreads();
    asm volatile("griddepcontrol.wait;" ::: "memory");
    const int pos = __ldcg(bt.d_pos + b);
    const int64_t slot = __ldcg(bt.d_seq_slot + b);
    const int low = attn_low(s, pos), len = pos + 1 - low;   // keys are counted from the first that is seen
    if ((unsigned)pos >= (unsigned)s.limit) {   // outside the cache: record it, touch nothing (all CTAs of the row leave)
        if (threadIdx.x == 0) atomicExch(status, (int32_t)PG_ERR_INVALID);
        return;
    }
    const int chunk = ((len + S - 1) / S + 63) & ~63;
    const int t0 = split * chunk, t1 = min(len, t0 + chunk);
    const int used = (len + chunk - 1) / chunk;           // slices with keys; the others leave at once
    if (t0 >= t1) return;
    const bool newest = FUSED && t1 == len;
    const int64_t first = (slot * s.G + g) * (int64_t)s.cap + attn_row(s, low);
    bf16 *kb = kc + first * s.dp, *vb = vc + first * s.vp;
    const int nk = s.dp / 16, nv = s.vp / 8;

    // the warp's 16-key tiles: t0 + 16 (warp + 4 i); lanes 0 .. 15 ask for a key each, lanes 16 .. 31 for a value each
    // (rows behind the slice repeat its last one and are masked)
    const int ntiles = (t1 - t0 + 15) / 16, mine = ntiles > warp ? (ntiles - warp + AS_WARPS - 1) / AS_WARPS : 0;
    auto fetch = [&](int i) {
        const uint32_t at = ring + (uint32_t)(i % AS_STAGES) * stage, on = bar + (uint32_t)(i % AS_STAGES) * 8;
        const int64_t key = min(t0 + 16 * (warp + AS_WARPS * i) + (lane & 15), t1 - 1);
        if (lane == 0) pg_mbar_expect(on, 16u * (uint32_t)(s.dp + s.vp) * 2u);
        __syncwarp();
        if (lane < 16)
            pg_bulk_load(at + (uint32_t)lane * kstride, kb + key * s.dp, (uint32_t)s.dp * 2u, on);
        else
            pg_bulk_load(at + 16u * kstride + (uint32_t)(lane - 16) * vstride, vb + key * s.vp, (uint32_t)s.vp * 2u, on);
    };
    auto prime = [&]() {
        for (int i = 0; i < AS_STAGES && i < mine; i++) fetch(i);
    };
    prime();
    const float *row = proj + (int64_t)b * ldp;
    if (newest && warp == 2) head_norm(row + (int64_t)(s.H + g) * s.D, s.kn, s.D, s.dp, s.eps, 1.0f, k_new, lane);
    if (newest && warp == 3) {
        const float *src = row + (int64_t)(s.H + s.G) * s.D + (int64_t)g * s.V;
        for (int c = lane; c < s.vp; c += 32) pg_put(v_new + c, c < s.V ? __ldcg(src + c) : 0.0f);
    }
    for (int h = warp; h < heads; h += AS_WARPS) {
        bf16 *dst = qs + h * (s.dp + 8);
        if (FUSED) {
            head_norm(row + (int64_t)(h0 + h) * s.D, s.qn, s.D, s.dp, s.eps, temperature(s, pos), dst, lane);
        } else {
            for (int i = lane; i < s.dp; i += 32) dst[i] = __float2bfloat16_rn(pg_get(q + ((int64_t)b * s.H + h0 + h) * s.dp + i));
        }
    }
    __syncthreads();
    if (newest) {
        // appended for later steps; this step takes the row from shared memory (below)
        for (int i = threadIdx.x; i < (s.dp + s.vp) / 2; i += AS_WARPS * 32) {
            const uint32_t x = reinterpret_cast<const uint32_t *>(k_new)[i];
            if (i < s.dp / 2)
                reinterpret_cast<uint32_t *>(kb + (int64_t)(len - 1) * s.dp)[i] = x;
            else
                reinterpret_cast<uint32_t *>(vb + (int64_t)(len - 1) * s.vp)[i - s.dp / 2] = x;
        }
    }
    uint32_t qf[DC][4];
    {
        const uint32_t qb = pg_smem(qs);
#pragma unroll
        for (int i = 0; i < DC; i++)
            if (i < nk) pg_ldsm4(qf[i], tile_at(qb, s.dp * 2 + 16, lane & 15, i * 16 + (lane >> 4) * 8));
    }
    float o[VC][4];
#pragma unroll
    for (int i = 0; i < VC; i++)
#pragma unroll
        for (int j = 0; j < 4; j++) o[i][j] = 0.0f;
    const float sl = s.scale * LOG2E;
    const float bias0 = s.slopes && r < heads ? __ldg(s.slopes + h0 + r) * LOG2E : 0.0f, bias1 = s.slopes && r + 8 < heads ? __ldg(s.slopes + h0 + r + 8) * LOG2E : 0.0f;
    float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.0f, l1 = 0.0f;
    bool ok = true;
    for (int i = 0; i < mine; i++) {
        ok = pg_mbar_wait(bar + (uint32_t)(i % AS_STAGES) * 8, (uint32_t)(i / AS_STAGES) & 1u, &abort_flag, status, limit_ns);
        ok = __all_sync(0xffffffffu, ok);
        if (!ok) break;
        const int j0 = t0 + 16 * (warp + AS_WARPS * i);
        const uint32_t kt = ring + (uint32_t)(i % AS_STAGES) * stage, vt = kt + 16 * kstride;
        if (newest && j0 + 16 >= len) {
            // the copies brought what the cache held at the newest position: put the new row in its place
            unsigned char *at = smem + (size_t)warp * AS_STAGES * stage + (size_t)(i % AS_STAGES) * stage;
            for (int x = lane; x < s.dp / 2; x += 32) reinterpret_cast<uint32_t *>(at + (len - 1 - j0) * kstride)[x] = reinterpret_cast<const uint32_t *>(k_new)[x];
            for (int x = lane; x < s.vp / 2; x += 32)
                reinterpret_cast<uint32_t *>(at + 16 * kstride + (len - 1 - j0) * vstride)[x] = reinterpret_cast<const uint32_t *>(v_new)[x];
            __syncwarp();
        }
        float sc[2][4] = {};
        scores16<DC>(qf, nk, kt, kstride, 0, lane, sc[0], sc[1]);
        float b0 = -INFINITY, b1 = -INFINITY;
#pragma unroll
        for (int n = 0; n < 2; n++)
#pragma unroll
            for (int j = 0; j < 2; j++) {
                const int key = j0 + n * 8 + 2 * t + j;
                const float back = (float)(key - (len - 1));
                sc[n][j] = key < t1 ? fmaf(bias0, back, sc[n][j] * sl) : -INFINITY;
                sc[n][2 + j] = key < t1 ? fmaf(bias1, back, sc[n][2 + j] * sl) : -INFINITY;
                b0 = fmaxf(b0, sc[n][j]);
                b1 = fmaxf(b1, sc[n][2 + j]);
            }
#pragma unroll
        for (int x = 1; x < 4; x <<= 1) {
            b0 = fmaxf(b0, __shfl_xor_sync(0xffffffffu, b0, x));
            b1 = fmaxf(b1, __shfl_xor_sync(0xffffffffu, b1, x));
        }
        const float n0 = fmaxf(m0, b0), n1 = fmaxf(m1, b1);   // finite: a tile has at least one key
        const float f0 = exp2f(m0 - n0), f1 = exp2f(m1 - n1);
        m0 = n0;
        m1 = n1;
        float p[8];
#pragma unroll
        for (int j = 0; j < 2; j++) {
            p[j] = exp2f(sc[0][j] - m0);
            p[2 + j] = exp2f(sc[0][2 + j] - m1);
            p[4 + j] = exp2f(sc[1][j] - m0);
            p[6 + j] = exp2f(sc[1][2 + j] - m1);
        }
        l0 = l0 * f0 + ((p[0] + p[1]) + (p[4] + p[5]));
        l1 = l1 * f1 + ((p[2] + p[3]) + (p[6] + p[7]));
        if (__any_sync(0xffffffffu, f0 != 1.0f || f1 != 1.0f)) {
#pragma unroll
            for (int x = 0; x < VC; x++) {
                o[x][0] *= f0;
                o[x][1] *= f0;
                o[x][2] *= f1;
                o[x][3] *= f1;
            }
        }
        const uint32_t pf[4] = {pg_pack_bf16(p[0], p[1]), pg_pack_bf16(p[2], p[3]), pg_pack_bf16(p[4], p[5]), pg_pack_bf16(p[6], p[7])};
        values16<VC>(o, nv, pf, vt, vstride, 0, lane);
        __syncwarp();                                     // every lane is done with the stage before it is filled again
        if (i + AS_STAGES < mine) fetch(i + AS_STAGES);
    }
    if (!ok) {
        // copies that are still in flight get a bounded time to land before their shared memory is used again
        const unsigned long long w0 = pg_globaltimer_ns();
        while (pg_globaltimer_ns() - w0 < 2000000ull) {
        }
    }
#pragma unroll
    for (int x = 1; x < 4; x <<= 1) {
        l0 += __shfl_xor_sync(0xffffffffu, l0, x);
        l1 += __shfl_xor_sync(0xffffffffu, l1, x);
    }
    __syncthreads();                                      // the rings are free
    // warps meet in shared memory: [warp][16][vp + 4]
    const int ms = s.vp + 4;
    float *w0 = mg + ((size_t)warp * 16 + r) * ms, *w1 = w0 + 8 * ms;
#pragma unroll
    for (int i = 0; i < VC; i++) {
        if (i < nv) {
            *reinterpret_cast<float2 *>(w0 + i * 8 + 2 * t) = make_float2(o[i][0], o[i][1]);
            if (heads > 8) *reinterpret_cast<float2 *>(w1 + i * 8 + 2 * t) = make_float2(o[i][2], o[i][3]);
        }
    }
    if (t == 0) {
        *reinterpret_cast<float2 *>(w0 + s.vp) = make_float2(m0, l0);
        *reinterpret_cast<float2 *>(w1 + s.vp) = make_float2(m1, l1);
    }
    __syncthreads();
    const int64_t unit = ((int64_t)b * gridDim.y + blockIdx.y);
    float *mine_part = part + (unit * S + split) * 16 * ms;
    const int vq = s.vp / 4;
    for (int x = threadIdx.x; x < heads * vq; x += AS_WARPS * 32) {
        const int h = x / vq, c = (x - h * vq) * 4;
        float m = -INFINITY;
#pragma unroll
        for (int w = 0; w < AS_WARPS; w++) m = fmaxf(m, mg[((size_t)w * 16 + h) * ms + s.vp]);
        float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
        float l = 0.0f;
#pragma unroll
        for (int w = 0; w < AS_WARPS; w++) {
            const float *at = mg + ((size_t)w * 16 + h) * ms;
            const float f = exp2f(at[s.vp] - m);          // 0 for a warp without keys
            const float4 v = *reinterpret_cast<const float4 *>(at + c);
            a.x = fmaf(f, v.x, a.x), a.y = fmaf(f, v.y, a.y), a.z = fmaf(f, v.z, a.z), a.w = fmaf(f, v.w, a.w);
            l = fmaf(f, at[s.vp + 1], l);
        }
        if (used == 1) {
            float f = 1.0f;
            if (s.sink) {
                const float mm = fmaxf(m, 0.0f);
                f = exp2f(m - mm);
                l = l * f + exp2f(-mm);
            }
            f = __fdiv_rn(f, l);
            bf16 *dst = out + (int64_t)b * ldo + (int64_t)(h0 + h) * s.V + c;
            const float y[4] = {a.x * f, a.y * f, a.z * f, a.w * f};
#pragma unroll
            for (int i = 0; i < 4; i++)
                if (c + i < s.V) pg_put(dst + i, y[i]);
        } else {
            *reinterpret_cast<float4 *>(mine_part + (size_t)h * ms + c) = a;
            if (c == 0) *reinterpret_cast<float2 *>(mine_part + (size_t)h * ms + s.vp) = make_float2(m, l);
        }
    }
    if (used == 1) return;
    __threadfence();
    __syncthreads();
    if (threadIdx.x == 0) {
        __threadfence();
        last_in = atomicAdd(tickets + unit, 1) == used - 1;
    }
    __syncthreads();
    if (!last_in) return;
    __threadfence();
    if (threadIdx.x == 0) tickets[unit] = 0;
    // a warp per head: the slices' weights; then all columns with their loads in flight together
    const float *parts = part + unit * S * 16 * ms;
    for (int h = warp; h < heads; h += AS_WARPS) {
        float2 ml[AS_SLICES / 32];
        float m = s.sink ? 0.0f : -INFINITY, l = 0.0f;
#pragma unroll
        for (int i = 0; i < AS_SLICES / 32; i++) {
            const int k = i * 32 + lane;
            ml[i] = k < used ? __ldcg(reinterpret_cast<const float2 *>(parts + ((size_t)k * 16 + h) * ms + s.vp)) : make_float2(-INFINITY, 0.0f);
            m = fmaxf(m, ml[i].x);
        }
#pragma unroll
        for (int o2 = 16; o2 > 0; o2 >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o2));
#pragma unroll
        for (int i = 0; i < AS_SLICES / 32; i++) {
            const float f = exp2f(ml[i].x - m);
            weight[h][i * 32 + lane] = f;
            l = fmaf(f, ml[i].y, l);
        }
        l = pg_warp_sum(l) + (s.sink ? exp2f(-m) : 0.0f);
        if (lane == 0) denom[h] = __fdiv_rn(1.0f, l);
    }
    __syncthreads();
    for (int x = threadIdx.x; x < heads * vq; x += AS_WARPS * 32) {
        const int h = x / vq, c = (x - h * vq) * 4;
        const float *at = parts + (size_t)h * ms + c;
        float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
        for (int k0 = 0; k0 < used; k0 += 8) {            // eight loads in flight; behind the last slice its weight is 0
            float4 v[8];
#pragma unroll
            for (int k = 0; k < 8; k++) v[k] = __ldcg(reinterpret_cast<const float4 *>(at + (size_t)min(k0 + k, used - 1) * 16 * ms));
#pragma unroll
            for (int k = 0; k < 8; k++) {
                const float f = k0 + k < used ? weight[h][k0 + k] : 0.0f;
                a.x = fmaf(f, v[k].x, a.x), a.y = fmaf(f, v[k].y, a.y), a.z = fmaf(f, v[k].z, a.z), a.w = fmaf(f, v[k].w, a.w);
            }
        }
        bf16 *dst = out + (int64_t)b * ldo + (int64_t)(h0 + h) * s.V + c;
        const float f = denom[h], y[4] = {a.x * f, a.y * f, a.z * f, a.w * f};
#pragma unroll
        for (int i = 0; i < 4; i++)
            if (c + i < s.V) pg_put(dst + i, y[i]);
    }
}

AttnShape shape_of(const pg_attention *p)
{
    AttnShape s;
    s.H = p->heads, s.G = p->kv_heads, s.rep = p->heads / p->kv_heads, s.D = p->dim, s.V = p->vdim;
    s.dp = (int)pg_up(s.D, 16), s.vp = (int)pg_up(s.V, 16);
    s.cap = p->cap, s.sink = p->sink, s.chunk = p->chunk, s.limit = p->positions > 0 ? p->positions : p->cap;
    s.slopes = p->d_slopes;
    s.eps = p->eps, s.scale = p->scale, s.coef = p->temp_coef, s.every = p->temp_every;
    s.qn = p->d_q_norm, s.kn = p->d_k_norm;
    return s;
}

// slices of the context: enough CTAs for about two per SM, none shorter than 128 positions of the longest context
int slices(const pg_ctx *ctx, int64_t units, const AttnShape &s)
{
    const int64_t cap = s.chunk && s.chunk < s.cap ? s.chunk : s.cap;
    int64_t S = std::max<int64_t>(1, 2 * (int64_t)ctx->sm_count / std::max<int64_t>(1, units));
    S = std::min<int64_t>(S, std::max<int64_t>(1, cap / 128));
    return (int)std::min<int64_t>(S, AS_SLICES);
}

template <int DC, int VC>
int32_t run_prompt(pg_ctx *ctx, const AttnShape &s, const pg_batch *bt, const bf16 *q, const bf16 *kc, const bf16 *vc, bf16 *out, int64_t ldo)
{
    constexpr int WARPS = DC > 8 || VC > 16 ? 4 : 8;
    const int smem = 2 * AP_KEYS * ((s.dp + s.vp) * 2 + 32);
    static std::atomic<uint64_t> set{0};
    PG_CUDA(pg_max_smem_once(attn_prompt_kernel<DC, VC, WARPS>, 2 * AP_KEYS * ((DC * 16 + VC * 8) * 2 + 32), ctx->device, set));
    const int64_t tiles = ((int64_t)bt->max_len * s.rep + WARPS * 16 - 1) / (WARPS * 16);
    return launch_pdl(ctx, attn_prompt_kernel<DC, VC, WARPS>, dim3((unsigned)tiles, (unsigned)s.G, (unsigned)bt->seqs), dim3(WARPS * 32), (size_t)smem, s, *bt,
                      q, kc, vc, out, ldo);
}

template <int DC, int VC, bool FUSED>
int32_t run_step(pg_ctx *ctx, const AttnShape &s, const pg_batch *bt, const float *proj, int64_t ldp, const bf16 *q, bf16 *kc, bf16 *vc, float *part,
                 int32_t *tickets, bf16 *out, int64_t ldo)
{
    const int stage = 16 * ((s.dp + s.vp) * 2 + 32);
    const int rings = AS_WARPS * AS_STAGES * stage;
    const int smem = std::max(rings + 16 * (s.dp + 8) * 2 + (s.dp + s.vp) * 2, AS_WARPS * 16 * (s.vp + 4) * 4);
    static std::atomic<uint64_t> set{0};
    PG_CUDA(pg_max_smem_once(attn_step_kernel<DC, VC, FUSED>, 220 * 1024, ctx->device, set));
    const int ht = (s.rep + 15) / 16;
    const int S = slices(ctx, (int64_t)bt->rows * s.G * ht, s);
    return launch_pdl(ctx, attn_step_kernel<DC, VC, FUSED>, dim3((unsigned)S, (unsigned)(s.G * ht), (unsigned)bt->rows), dim3(AS_WARPS * 32), (size_t)smem, s,
                      *bt, proj, ldp, q, kc, vc, part, tickets, out, ldo, ctx->d_status, ctx->wait_limit_ns);
}

}  // namespace

int32_t pgk_attention_f32(pg_ctx *ctx, const AttnShape &s, const pg_batch *bt, const float *q, const float *kc, const float *vc, float *out, int64_t ldo)
{
    PG_REQUIRE(bt->rows <= 65535, "attention: too many rows for the f32 form");
    PG_REQUIRE(s.V <= 8 * AF_T && (s.dp + AF_T) * 4 <= 48 * 1024, "attention: heads too wide for the f32 form");
    return launch_pdl(ctx, attn_f32_kernel, dim3((unsigned)s.H, (unsigned)bt->rows), dim3(AF_T), (size_t)(s.dp + AF_T) * 4, s, *bt, q, kc, vc, out, ldo);
}

extern "C" {

PG_API int64_t pg_attention_part_floats(pg_ctx *ctx, const pg_attention *p, int64_t max_seqs)
{
    if (!ctx || !p || p->kv_heads <= 0 || max_seqs <= 0) return 0;
    const AttnShape s = shape_of(p);
    const int64_t per = (int64_t)s.G * ((s.rep + 15) / 16);
    int64_t most = 0;
    for (int64_t rows = 1; rows <= max_seqs; rows++) most = std::max(most, rows * per * slices(ctx, rows * per, s));
    return most * 16 * (s.vp + 4);
}

PG_API int32_t pg_attention_run(pg_ctx *ctx, const pg_attention *p, const pg_batch *batch, const float *d_proj, int64_t ldp, void *d_kcache,
                                void *d_vcache, void *d_out, int32_t dtype, int64_t ldo)
{
    PG_ENTER(ctx);
    PG_REQUIRE(p && batch && d_proj && d_kcache && d_vcache && d_out && p->d_q && p->d_part && p->d_tickets,
               "attention: null pointer");
    PG_REQUIRE(p->heads > 0 && p->kv_heads > 0 && p->heads % p->kv_heads == 0 && p->dim > 0 && p->dim <= 256 && p->vdim > 0 && p->vdim <= 256 && p->cap > 0,
               "attention: bad shape (heads %d / %d, dim %d and vdim %d at most 256)", p->heads, p->kv_heads, p->dim, p->vdim);
    PG_REQUIRE(p->chunk >= 0 && (p->chunk == 0 ? p->positions <= p->cap : p->cap % p->chunk == 0),
               "attention: a cache of %d rows for %d positions in chunks of %d", p->cap, p->positions, p->chunk);
    PG_REQUIRE(p->chunk == 0 || p->positions <= p->cap || ((int64_t)(p->chunk + batch->max_len - 2) / p->chunk + 1) * p->chunk <= p->cap,
               "attention: a step of %d tokens has more chunks of %d than the cache of %d rows", batch->max_len, p->chunk, p->cap);
    const AttnShape s = shape_of(p);
    PG_REQUIRE(ldp >= (int64_t)(s.H + s.G) * s.D + (int64_t)s.G * s.V && ldo >= (int64_t)s.H * s.V, "attention: rows too short");
    PG_REQUIRE(s.G <= 65535 && batch->rows >= 0 && batch->seqs <= 65535, "attention: too many heads or sequences");
    if (batch->rows == 0) return PG_OK;
    const int M = batch->rows;
    const int wide = s.D % 4 == 0 && s.V % 4 == 0 && s.D <= 128 && s.V <= 128 && ldp % 4 == 0 && ((uintptr_t)d_proj & 15) == 0;
    if (dtype == PG_F32) {
        int32_t rc = launch_pdl(ctx, attn_prep_kernel<float>, dim3((unsigned)M), dim3(256), 0, s, *batch, d_proj, ldp, (float *)p->d_q, (float *)d_kcache,
                                (float *)d_vcache, wide, ctx->d_status);
        if (rc != PG_OK) return rc;
        return pgk_attention_f32(ctx, s, batch, (const float *)p->d_q, (const float *)d_kcache, (const float *)d_vcache, (float *)d_out, ldo);
    }
    bf16 *q = (bf16 *)p->d_q, *kc = (bf16 *)d_kcache, *vc = (bf16 *)d_vcache, *out = (bf16 *)d_out;
    const bool step = batch->max_len == 1, fused = step && s.rep <= 16;
    if (!fused) {
        const int32_t rc = launch_pdl(ctx, attn_prep_kernel<bf16>, dim3((unsigned)M), dim3(256), 0, s, *batch, d_proj, ldp, q, kc, vc, wide, ctx->d_status);
        if (rc != PG_OK) return rc;
    }
    if (!step && pgk_attention_prompt_tc_supports(s, batch, p->slots, ldo, out)) return pgk_attention_prompt_tc(ctx, s, batch, p->slots, q, kc, vc, out, ldo);
#define PG_AT(DC, VC)                                                                                                        \
    do {                                                                                                                     \
        if (fused) return run_step<DC, VC, true>(ctx, s, batch, d_proj, ldp, q, kc, vc, p->d_part, p->d_tickets, out, ldo);  \
        if (step) return run_step<DC, VC, false>(ctx, s, batch, d_proj, ldp, q, kc, vc, p->d_part, p->d_tickets, out, ldo);  \
        return run_prompt<DC, VC>(ctx, s, batch, q, kc, vc, out, ldo);                                                       \
    } while (0)
    if (s.dp <= 64 && s.vp <= 64) PG_AT(4, 8);
    if (s.dp <= 128 && s.vp <= 128) PG_AT(8, 16);
    PG_AT(16, 32);
#undef PG_AT
}

}  // extern "C"
