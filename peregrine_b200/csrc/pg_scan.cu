// Selective scan with a short causal convolution in front of it.
//
// Per channel c and state n (f32):  S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c x_c B_n;   y_c = sum_n S[c, n] C_n + D_c x_c,
// then y * silu(z).  Channels and states are independent of each other; a token only meets the one before it.
//
//   scan_conv_kernel    convolution and silu of the rows; x in the step's type, which the products behind it read
//   scan_step_kernel    one token per sequence: W_dt, softplus, update, read-out and gate in one launch; the state is read and
//                       written once
//   scan_run_kernel     portions: a CTA has 32 channels of a sequence, four lanes per channel, whose states stay in registers;
//                       step sizes, inputs, B and C come in tiles of tokens through shared memory, the next tile's loads in
//                       flight meanwhile.  It also stores the convolution inputs that the next portion needs.
//
// Convolution inputs are kept per slot in a ring of `taps` entries, position p in entry p mod taps: a single token writes an
// entry that nobody reads any more.  A sequence starts at position 0: what its slot holds is then taken as zero.
#include <algorithm>

#include "pg_lm.cuh"

namespace {

struct ScanShape {
    int inner, N, taps, ss, dtp;     // ss: state row stride; dtp: columns of the low-rank step size, up to 64
    const float *conv, *conv_bias, *a, *d, *dt_bias;
    const bf16 *dt;
};

__device__ __forceinline__ float softplus(float x) { return x > 20.0f ? x : log1pf(expf(x)); }

__device__ __forceinline__ float ex2(float x)
{
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

template <int V>
struct Lanes {
    float v[V];
};
template <int V>
__device__ __forceinline__ Lanes<V> load_lanes(const float *p)
{
    Lanes<V> r;
    if constexpr (V == 4) {
        const float4 q = __ldcg(reinterpret_cast<const float4 *>(p));
        r.v[0] = q.x, r.v[1] = q.y, r.v[2] = q.z, r.v[3] = q.w;
    } else {
        r.v[0] = __ldcg(p);
    }
    return r;
}

// ---- convolution: grid (channel blocks, ceil(longest / 8), seqs) ----------------------------------------------------
constexpr int SC_T = 128, SC_TOKENS = 8;
// TAPS: the number of taps, 0 = any; V: channels per thread
template <int TAPS, int V, typename TA>
__global__ void __launch_bounds__(SC_T)
    scan_conv_kernel(const ScanShape s, const pg_batch bt, const float *__restrict__ proj, int64_t ldp, float *ring, TA *__restrict__ x, int64_t ldx, int keep)
{
    pg_pdl_begin();
    const int seq = blockIdx.z, row0 = __ldcg(bt.d_seq_row0 + seq), T = __ldcg(bt.d_seq_row0 + seq + 1) - row0;
    const int t0 = blockIdx.y * SC_TOKENS, n = min(SC_TOKENS, T - t0), c = (blockIdx.x * SC_T + threadIdx.x) * V;
    if (n <= 0 || c >= s.inner) return;
    const int pos0 = __ldcg(bt.d_pos + row0), taps = TAPS > 0 ? TAPS : s.taps;
    float *rg = ring + (int64_t)__ldcg(bt.d_seq_slot + seq) * taps * s.inner + c;
    const float *row = proj + (int64_t)row0 * ldp + c;
    // the input of the portion's token t (negative: before the portion)
    auto input = [&](int t) {
        if (t >= 0) return load_lanes<V>(row + (int64_t)t * ldp);
        if (pos0 + t >= 0) return load_lanes<V>(rg + (int64_t)((pos0 + t) % taps) * s.inner);
        return Lanes<V>{};
    };
    auto put = [&](int t, const Lanes<V> &y) {
        TA *dst = x + (int64_t)(row0 + t) * ldx + c;
        float v[V];
#pragma unroll
        for (int i = 0; i < V; i++) v[i] = pg_silu(y.v[i]);
        if constexpr (V == 4 && sizeof(TA) == 4)
            *reinterpret_cast<float4 *>(dst) = make_float4(v[0], v[1], v[2], v[3]);
        else if constexpr (V == 4)
            *reinterpret_cast<uint2 *>(dst) = make_uint2(pg_pack_bf16(v[0], v[1]), pg_pack_bf16(v[2], v[3]));
        else
            pg_put(dst, v[0]);
    };
    const Lanes<V> bias = load_lanes<V>(s.conv_bias + c);
    if constexpr (TAPS > 0) {
        Lanes<V> wt[TAPS], in[TAPS - 1 + SC_TOKENS];
#pragma unroll
        for (int j = 0; j < TAPS; j++) wt[j] = load_lanes<V>(s.conv + (int64_t)j * s.inner + c);
#pragma unroll
        for (int j = 0; j < TAPS - 1 + SC_TOKENS; j++) in[j] = j - (TAPS - 1) < n ? input(t0 + j - (TAPS - 1)) : Lanes<V>{};
#pragma unroll
        for (int t = 0; t < SC_TOKENS; t++) {
            if (t < n) {
                Lanes<V> y = bias;
#pragma unroll
                for (int j = 0; j < TAPS; j++)
#pragma unroll
                    for (int i = 0; i < V; i++) y.v[i] = fmaf(wt[j].v[i], in[t + j].v[i], y.v[i]);
                put(t0 + t, y);
            }
        }
    } else {
        for (int t = 0; t < n; t++) {
            Lanes<V> y = bias;
            for (int j = 0; j < taps; j++) {
                const Lanes<V> w = load_lanes<V>(s.conv + (int64_t)j * s.inner + c), v = input(t0 + t + j - (taps - 1));
#pragma unroll
                for (int i = 0; i < V; i++) y.v[i] = fmaf(w.v[i], v.v[i], y.v[i]);
            }
            put(t0 + t, y);
        }
    }
    if (keep) {
        // one token: its entry of the ring is older than anything a convolution still reads
        const Lanes<V> in = input(0);
#pragma unroll
        for (int i = 0; i < V; i++) rg[(int64_t)(pos0 % taps) * s.inner + i] = in.v[i];
    }
}

// ---- the recurrence ------------------------------------------------------------------------------------------------
constexpr int SR_T = 128, SR_CH = 32;   // channels of a CTA: four lanes each, quads q, q + 4, .. of a channel's states

// A quad of states takes a token; returns its part of the read-out.
__device__ __forceinline__ float update(float4 &S, const float4 &a, float dt, float du, const float4 &b, const float4 &c)
{
    S.x = fmaf(ex2(dt * a.x), S.x, du * b.x);
    S.y = fmaf(ex2(dt * a.y), S.y, du * b.y);
    S.z = fmaf(ex2(dt * a.z), S.z, du * b.z);
    S.w = fmaf(ex2(dt * a.w), S.w, du * b.w);
    return fmaf(S.x, c.x, S.y * c.y) + fmaf(S.z, c.z, S.w * c.w);
}

// grid (ceil(inner / 32), ceil(rows / R)).  NC: quads of states per lane
template <int NC, int R, typename TA>
__global__ void __launch_bounds__(SR_T)
    scan_step_kernel(const ScanShape s, const pg_batch bt, const float *__restrict__ proj, int64_t ldp, const TA *__restrict__ x, int64_t ldx,
                     const float *__restrict__ low, int64_t ldl, float *state, TA *__restrict__ out, int64_t ldo)
{
    extern __shared__ __align__(16) float sm[];   // [R][dtp] low-rank step sizes | [R][2][16 NC] B and C
    constexpr int NP = 16 * NC;
    const int tid = threadIdx.x, q = tid & 3, c = blockIdx.x * SR_CH + (tid >> 2), m0 = blockIdx.y * R;
    const bool live = c < s.inner;
    const int quads = s.ss / 4;
    float *sdt = sm, *sbc = sm + R * s.dtp;
    asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
    // weights do not depend on the kernel before
    float4 a[NC];
#pragma unroll
    for (int i = 0; i < NC; i++)
        a[i] = live && q + 4 * i < quads ? __ldg(reinterpret_cast<const float4 *>(s.a + (int64_t)c * s.ss) + q + 4 * i) : make_float4(0.f, 0.f, 0.f, 0.f);
    const float dt_bias = live ? __ldg(s.dt_bias + c) : 0.0f, skip = live ? __ldg(s.d + c) : 0.0f;
    asm volatile("griddepcontrol.wait;" ::: "memory");
    float4 S[R][NC];
    int64_t at[R];
    float xv[R], z[R];
#pragma unroll
    for (int r = 0; r < R; r++) {
        const int m = m0 + r;
        const bool on = live && m < bt.rows;
        at[r] = on ? ((int64_t)__ldcg(bt.d_seq_slot + __ldcg(bt.d_row_seq + m)) * s.inner + c) * s.ss : -1;
        const bool old = on && __ldcg(bt.d_pos + m) > 0;
#pragma unroll
        for (int i = 0; i < NC; i++)
            S[r][i] = old && q + 4 * i < quads ? __ldcg(reinterpret_cast<const float4 *>(state + at[r]) + q + 4 * i) : make_float4(0.f, 0.f, 0.f, 0.f);
        xv[r] = on ? pg_get(x + (int64_t)m * ldx + c) : 0.0f;
        z[r] = on ? __ldcg(proj + (int64_t)m * ldp + s.inner + c) : 0.0f;
    }
    for (int i = tid; i < R * s.dtp; i += SR_T) {
        const int r = i / s.dtp, k = i - r * s.dtp;
        sdt[i] = m0 + r < bt.rows ? __ldcg(low + (int64_t)(m0 + r) * ldl + k) : 0.0f;
    }
    for (int i = tid; i < R * 2 * NP; i += SR_T) {
        const int r = i / (2 * NP), k = i - r * 2 * NP, which = k / NP, n = k - which * NP;
        sbc[i] = m0 + r < bt.rows && n < s.N ? __ldcg(low + (int64_t)(m0 + r) * ldl + s.dtp + which * s.N + n) : 0.0f;
    }
    __syncthreads();
    float acc[R] = {};
    if (live) {
        const uint4 *w = reinterpret_cast<const uint4 *>(s.dt + (int64_t)c * s.dtp) + q;
#pragma unroll 2
        for (int k = 0; k < s.dtp / 32; k++) {
            const uint4 b = __ldg(w + 4 * k);
#pragma unroll
            for (int r = 0; r < R; r++) {
                const float4 *v = reinterpret_cast<const float4 *>(sdt + r * s.dtp + k * 32 + q * 8);
                const float4 u0 = v[0], u1 = v[1];
                acc[r] += (fmaf(pg_bf16_lo(b.x), u0.x, pg_bf16_hi(b.x) * u0.y) + fmaf(pg_bf16_lo(b.y), u0.z, pg_bf16_hi(b.y) * u0.w)) +
                          (fmaf(pg_bf16_lo(b.z), u1.x, pg_bf16_hi(b.z) * u1.y) + fmaf(pg_bf16_lo(b.w), u1.z, pg_bf16_hi(b.w) * u1.w));
            }
        }
    }
#pragma unroll
    for (int r = 0; r < R; r++) {
        acc[r] += __shfl_xor_sync(0xffffffffu, acc[r], 1);
        acc[r] += __shfl_xor_sync(0xffffffffu, acc[r], 2);
        const float dt = softplus(acc[r] + dt_bias), du = dt * xv[r];
        float y = 0.0f;
#pragma unroll
        for (int i = 0; i < NC; i++) {
            const float4 *b = reinterpret_cast<const float4 *>(sbc + r * 2 * NP) + q + 4 * i;
            y += update(S[r][i], a[i], dt, du, b[0], b[NP / 4]);
            if (at[r] >= 0 && q + 4 * i < quads) reinterpret_cast<float4 *>(state + at[r])[q + 4 * i] = S[r][i];
        }
        y += __shfl_xor_sync(0xffffffffu, y, 1);
        y += __shfl_xor_sync(0xffffffffu, y, 2);
        if (q == 0 && at[r] >= 0) pg_put(out + (int64_t)(m0 + r) * ldo + c, fmaf(skip, xv[r], y) * pg_silu(z[r]));
    }
}

// grid (ceil(inner / 32), seqs)
constexpr int SR_TOKENS = 16;
template <int NC, typename TA>
__global__ void __launch_bounds__(SR_T)
    scan_run_kernel(const ScanShape s, const pg_batch bt, const float *__restrict__ proj, int64_t ldp, float *ring, const TA *__restrict__ x, int64_t ldx,
                    const float *__restrict__ dt, int64_t ldt, const float *__restrict__ bc, int64_t ldb, float *state, TA *__restrict__ out, int64_t ldo)
{
    constexpr int NP = 16 * NC, TT = SR_TOKENS, PER = TT * SR_CH / SR_T, PERB = TT * 2 * NP / SR_T;
    __shared__ __align__(16) float sdt[TT][SR_CH], sdu[TT][SR_CH], sy[TT][SR_CH];
    __shared__ __align__(16) float sbc[TT][2][NP];
    pg_pdl_begin();
    const int tid = threadIdx.x, q = tid & 3, cl = tid >> 2, c0 = blockIdx.x * SR_CH, c = c0 + cl;
    const int seq = blockIdx.y, row0 = __ldcg(bt.d_seq_row0 + seq), T = __ldcg(bt.d_seq_row0 + seq + 1) - row0;
    if (T <= 0) return;
    const int pos0 = __ldcg(bt.d_pos + row0), quads = s.ss / 4;
    const int64_t slot = __ldcg(bt.d_seq_slot + seq);
    const bool live = c < s.inner;
    float4 *st = reinterpret_cast<float4 *>(state + (slot * s.inner + c) * s.ss);
    float4 a[NC], S[NC];
#pragma unroll
    for (int i = 0; i < NC; i++) {
        const bool on = live && q + 4 * i < quads;
        a[i] = on ? __ldg(reinterpret_cast<const float4 *>(s.a + (int64_t)c * s.ss) + q + 4 * i) : make_float4(0.f, 0.f, 0.f, 0.f);
        S[i] = on && pos0 > 0 ? __ldcg(st + q + 4 * i) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    // elements of a tile that this thread brings and finishes: tokens tid / 32 + 4 i of channel tid % 32
    const int ec = c0 + (tid & 31), et = tid >> 5;
    const bool elive = ec < s.inner;
    const float dt_bias = elive ? __ldg(s.dt_bias + ec) : 0.0f, skip = elive ? __ldg(s.d + ec) : 0.0f;
    float rdt[PER], rx[PER], rz[PER], rbc[PERB];
    auto fetch = [&](int t0) {
#pragma unroll
        for (int i = 0; i < PER; i++) {
            const int t = t0 + et + i * (SR_T / 32);
            const bool on = elive && t < T;
            const int64_t m = row0 + t;
            rdt[i] = on ? __ldcg(dt + m * ldt + ec) : 0.0f;
            rx[i] = on ? pg_get(x + m * ldx + ec) : 0.0f;
            rz[i] = on ? __ldcg(proj + m * ldp + s.inner + ec) : 0.0f;
        }
#pragma unroll
        for (int i = 0; i < PERB; i++) {
            const int e = tid + i * SR_T, t = t0 + e / (2 * NP), k = e % (2 * NP), which = k / NP, n = k - which * NP;
            rbc[i] = t < T && n < s.N ? __ldcg(bc + (int64_t)(row0 + t) * ldb + which * s.N + n) : 0.0f;
        }
    };
    fetch(0);
    for (int t0 = 0; t0 < T; t0 += TT) {
        float kx[PER], kz[PER];
#pragma unroll
        for (int i = 0; i < PER; i++) {
            const int t = et + i * (SR_T / 32);
            // (tokens behind the end leave the state alone: exp(0) S + 0)
            const float d = elive && t0 + t < T ? softplus(rdt[i] + dt_bias) : 0.0f;
            sdt[t][tid & 31] = d;
            sdu[t][tid & 31] = d * rx[i];
            kx[i] = rx[i];
            kz[i] = rz[i];
        }
#pragma unroll
        for (int i = 0; i < PERB; i++) (&sbc[0][0][0])[tid + i * SR_T] = rbc[i];
        __syncthreads();
        if (t0 + TT < T) fetch(t0 + TT);
#pragma unroll
        for (int t = 0; t < TT; t += 4) {
            float y[4];
#pragma unroll
            for (int u = 0; u < 4; u++) {
                const float d = sdt[t + u][cl], du = sdu[t + u][cl];
                y[u] = 0.0f;
#pragma unroll
                for (int i = 0; i < NC; i++)
                    y[u] += update(S[i], a[i], d, du, reinterpret_cast<const float4 *>(sbc[t + u][0])[q + 4 * i],
                                   reinterpret_cast<const float4 *>(sbc[t + u][1])[q + 4 * i]);
            }
            // four tokens' sums over four lanes: lane q ends with token q's
            const bool odd = q & 1, up = q & 2;
            const float g0 = __shfl_xor_sync(0xffffffffu, odd ? y[0] : y[1], 1), g1 = __shfl_xor_sync(0xffffffffu, odd ? y[2] : y[3], 1);
            const float k0 = (odd ? y[1] : y[0]) + g0, k1 = (odd ? y[3] : y[2]) + g1;
            const float g2 = __shfl_xor_sync(0xffffffffu, up ? k0 : k1, 2);
            sy[t + q][cl] = (up ? k1 : k0) + g2;
        }
        __syncthreads();
#pragma unroll
        for (int i = 0; i < PER; i++) {
            const int t = et + i * (SR_T / 32);
            if (elive && t0 + t < T) pg_put(out + (int64_t)(row0 + t0 + t) * ldo + ec, fmaf(skip, kx[i], sy[t][tid & 31]) * pg_silu(kz[i]));
        }
    }
#pragma unroll
    for (int i = 0; i < NC; i++)
        if (live && q + 4 * i < quads) st[q + 4 * i] = S[i];
    // the inputs that the next portion's convolution reads (scan_conv_kernel is done with the old ones)
    if (elive)
        for (int t = max(0, T - s.taps) + et; t < T; t += SR_T / 32)
            ring[(slot * s.taps + (pos0 + t) % s.taps) * s.inner + ec] = __ldcg(proj + (int64_t)(row0 + t) * ldp + ec);
}

ScanShape shape_of(const pg_scan *p)
{
    ScanShape s;
    s.inner = p->inner, s.N = p->state, s.taps = p->taps, s.ss = (int)pg_up(p->state, 4), s.dtp = (int)pg_up(p->dt_rank, 64);
    s.conv = p->d_conv, s.conv_bias = p->d_conv_bias, s.a = p->d_a, s.d = p->d_d, s.dt_bias = p->d_dt_bias, s.dt = (const bf16 *)p->d_dt;
    return s;
}

int32_t check(const pg_scan *p, const pg_batch *batch, int64_t ldp)
{
    PG_REQUIRE(p && batch && p->d_conv && p->d_conv_bias && p->d_a && p->d_d && p->d_dt_bias && p->d_dt, "scan: null pointer");
    PG_REQUIRE(p->inner > 0 && p->state > 0 && p->state <= 256 && p->dt_rank > 0 && p->dt_rank <= 2048 && p->taps > 0 && p->taps <= 64,
               "scan: bad shape (state %d at most 256, rank %d at most 2048, %d taps at most 64)", p->state, p->dt_rank, p->taps);
    PG_REQUIRE(ldp >= 2 * (int64_t)p->inner && batch->rows >= 0 && batch->seqs <= 65535, "scan: rows too short or too many sequences");
    return PG_OK;
}

template <typename TA>
int32_t run_conv(pg_ctx *ctx, const ScanShape &s, const pg_batch *bt, const float *proj, int64_t ldp, float *ring, TA *x, int64_t ldx)
{
    const int keep = bt->max_len == 1;
    const int V = s.inner % 4 == 0 && ldp % 4 == 0 && ldx % 4 == 0 ? 4 : 1;
    const dim3 grid((unsigned)((s.inner + SC_T * V - 1) / (SC_T * V)), (unsigned)((bt->max_len + SC_TOKENS - 1) / SC_TOKENS), (unsigned)bt->seqs);
    PG_REQUIRE(grid.y <= 65535, "scan: a portion is too long");
#define PG_SC(TAPS, V) return launch_pdl(ctx, scan_conv_kernel<TAPS, V, TA>, grid, dim3(SC_T), 0, s, *bt, proj, ldp, ring, x, ldx, keep)
    if (V == 4 && s.taps == 4) PG_SC(4, 4);
    if (V == 4) PG_SC(0, 4);
    PG_SC(0, 1);
#undef PG_SC
}

template <int NC, int R, typename TA>
int32_t launch_step(pg_ctx *ctx, const ScanShape &s, const pg_batch *bt, const float *proj, int64_t ldp, const TA *x, int64_t ldx, const float *low, int64_t ldl,
                    float *state, TA *out, int64_t ldo)
{
    const dim3 grid((unsigned)((s.inner + SR_CH - 1) / SR_CH), (unsigned)((bt->rows + R - 1) / R));
    return launch_pdl(ctx, scan_step_kernel<NC, R, TA>, grid, dim3(SR_T), (size_t)R * (s.dtp + 32 * NC) * 4, s, *bt, proj, ldp, x, ldx, low, ldl, state, out, ldo);
}

template <typename TA>
int32_t run_step(pg_ctx *ctx, const ScanShape &s, const pg_batch *bt, const float *proj, int64_t ldp, const TA *x, int64_t ldx, const float *low, int64_t ldl,
                 float *state, TA *out, int64_t ldo)
{
    if (s.N <= 16) return launch_step<1, 4, TA>(ctx, s, bt, proj, ldp, x, ldx, low, ldl, state, out, ldo);
    if (s.N <= 32) return launch_step<2, 4, TA>(ctx, s, bt, proj, ldp, x, ldx, low, ldl, state, out, ldo);
    if (s.N <= 64) return launch_step<4, 2, TA>(ctx, s, bt, proj, ldp, x, ldx, low, ldl, state, out, ldo);
    if (s.N <= 128) return launch_step<8, 1, TA>(ctx, s, bt, proj, ldp, x, ldx, low, ldl, state, out, ldo);
    return launch_step<16, 1, TA>(ctx, s, bt, proj, ldp, x, ldx, low, ldl, state, out, ldo);
}

template <typename TA>
int32_t run_scan(pg_ctx *ctx, const ScanShape &s, const pg_batch *bt, const float *proj, int64_t ldp, float *ring, const TA *x, int64_t ldx, const float *dt,
                 int64_t ldt, const float *bc, int64_t ldb, float *state, TA *out, int64_t ldo)
{
    const dim3 grid((unsigned)((s.inner + SR_CH - 1) / SR_CH), (unsigned)bt->seqs);
#define PG_SR(NC) return launch_whole(ctx, scan_run_kernel<NC, TA>, grid, dim3(SR_T), 0, s, *bt, proj, ldp, ring, x, ldx, dt, ldt, bc, ldb, state, out, ldo)
    if (s.N <= 16) PG_SR(1);
    if (s.N <= 32) PG_SR(2);
    if (s.N <= 64) PG_SR(4);
    if (s.N <= 128) PG_SR(8);
    PG_SR(16);
#undef PG_SR
}

}  // namespace

extern "C" {

PG_API int32_t pg_scan_conv(pg_ctx *ctx, const pg_scan *p, const pg_batch *batch, const float *d_proj, int64_t ldp, float *d_ring, void *d_x, int32_t dtype,
                            int64_t ldx)
{
    PG_ENTER(ctx);
    PG_REQUIRE(d_proj && d_ring && d_x && ldx >= (p ? p->inner : 0), "scan: null pointer or rows too short");
    const int32_t rc = check(p, batch, ldp);
    if (rc != PG_OK || batch->rows == 0) return rc;
    const ScanShape s = shape_of(p);
    if (dtype == PG_F32) return run_conv<float>(ctx, s, batch, d_proj, ldp, d_ring, (float *)d_x, ldx);
    return run_conv<bf16>(ctx, s, batch, d_proj, ldp, d_ring, (bf16 *)d_x, ldx);
}

PG_API int32_t pg_scan_step(pg_ctx *ctx, const pg_scan *p, const pg_batch *batch, const float *d_proj, int64_t ldp, const void *d_x, int64_t ldx,
                            const float *d_low, int64_t ldl, float *d_state, void *d_out, int32_t dtype, int64_t ldo)
{
    PG_ENTER(ctx);
    PG_REQUIRE(d_proj && d_x && d_low && d_state && d_out, "scan: null pointer");
    const int32_t rc = check(p, batch, ldp);
    if (rc != PG_OK || batch->rows == 0) return rc;
    const ScanShape s = shape_of(p);
    PG_REQUIRE(batch->max_len == 1 && ldx >= s.inner && ldo >= s.inner && ldl >= s.dtp + 2 * s.N && batch->rows <= 65535, "scan: not a step, or rows too short");
    if (dtype == PG_F32) return run_step<float>(ctx, s, batch, d_proj, ldp, (const float *)d_x, ldx, d_low, ldl, d_state, (float *)d_out, ldo);
    return run_step<bf16>(ctx, s, batch, d_proj, ldp, (const bf16 *)d_x, ldx, d_low, ldl, d_state, (bf16 *)d_out, ldo);
}

PG_API int32_t pg_scan_run(pg_ctx *ctx, const pg_scan *p, const pg_batch *batch, const float *d_proj, int64_t ldp, float *d_ring, const void *d_x, int64_t ldx,
                           const float *d_dt, int64_t ldt, const float *d_bc, int64_t ldb, float *d_state, void *d_out, int32_t dtype, int64_t ldo)
{
    PG_ENTER(ctx);
    PG_REQUIRE(d_proj && d_ring && d_x && d_dt && d_bc && d_state && d_out, "scan: null pointer");
    const int32_t rc = check(p, batch, ldp);
    if (rc != PG_OK || batch->rows == 0) return rc;
    const ScanShape s = shape_of(p);
    PG_REQUIRE(ldx >= s.inner && ldt >= s.inner && ldb >= 2 * s.N && ldo >= s.inner, "scan: rows too short");
    if (dtype == PG_F32) return run_scan<float>(ctx, s, batch, d_proj, ldp, d_ring, (const float *)d_x, ldx, d_dt, ldt, d_bc, ldb, d_state, (float *)d_out, ldo);
    return run_scan<bf16>(ctx, s, batch, d_proj, ldp, d_ring, (const bf16 *)d_x, ldx, d_dt, ldt, d_bc, ldb, d_state, (bf16 *)d_out, ldo);
}

}  // extern "C"
