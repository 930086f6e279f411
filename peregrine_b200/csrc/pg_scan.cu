// Selective scan with a short causal convolution in front of it.
//
// Per channel c and state n (f32):  S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c x_c B_n;   y_c = sum_n S[c, n] C_n + D_c x_c,
// then y * silu(z).  Channels and states are independent of each other; a token only meets the one before it.
//
//   scan_conv_kernel    convolution and silu of the rows; x in the step's type, which the products behind it read
//   scan_step_kernel    one token per sequence: W_dt, softplus, update, read-out and gate in one launch; the state is read and
//                       written once
//   scan_run_kernel     portions: a CTA has 32 channels of a sequence, four lanes per channel, whose states stay in registers;
//                       step sizes, inputs, B and C come in tiles of tokens through a ring in shared memory, brought and
//                       finished by four more warps.  It also stores the convolution inputs that the next portion needs.
//
// Convolution inputs are kept per slot in a ring of `taps` entries, position p in entry p mod taps: a single token writes an
// entry that nobody reads any more.  A sequence starts at position 0: what its slot holds is then taken as zero.
#include <algorithm>

#include "pg_async.cuh"
#include "pg_lm.cuh"

namespace {

struct ScanShape {
    int inner, N, taps, ss, dtp;     // ss: state row stride; dtp: columns of the low-rank step size, up to 64
    const float *conv, *conv_bias, *a, *d, *dt_bias;
    const bf16 *dt;
};

// ln(1 + e^x) = max(x, 0) + ln(1 + e) with e = e^-|x| in (0, 1], and ln(1 + e) = 2 artanh(e / (2 + e)) by its power series:
// the argument is at most 1/3, and what is left out is below 2^-26 of the sum.
__device__ __forceinline__ float softplus(float x)
{
    const float e = pg_ex2(-1.4426950408889634f * fabsf(x)), z = __fdividef(e, 2.0f + e), w = z * z;
    float p = 1.0f / 15.0f;
    p = fmaf(p, w, 1.0f / 13.0f);
    p = fmaf(p, w, 1.0f / 11.0f);
    p = fmaf(p, w, 1.0f / 9.0f);
    p = fmaf(p, w, 1.0f / 7.0f);
    p = fmaf(p, w, 1.0f / 5.0f);
    p = fmaf(p, w, 1.0f / 3.0f);
    p = fmaf(p, w, 1.0f);
    return fmaf(2.0f * z, p, fmaxf(x, 0.0f));
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
constexpr int SR_CH = 32, SR_T = 128;   // channels of a CTA: four lanes each, quads q, q + 4, .. of a channel's states

// a pair of f32 in one register pair, and the pairwise instructions
typedef unsigned long long f32x2;
__device__ __forceinline__ f32x2 pair(float lo, float hi)
{
    f32x2 v;
    asm("mov.b64 %0, {%1, %2};" : "=l"(v) : "f"(lo), "f"(hi));
    return v;
}
__device__ __forceinline__ float2 halves(f32x2 v)
{
    float2 r;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v));
    return r;
}
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b)
{
    f32x2 d;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c)
{
    f32x2 d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
struct Quad {
    f32x2 lo, hi;
};
__device__ __forceinline__ Quad quad(const float4 &v) { return {pair(v.x, v.y), pair(v.z, v.w)}; }
__device__ __forceinline__ float4 quad4(const Quad &v)
{
    const float2 a = halves(v.lo), b = halves(v.hi);
    return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ Quad load_quad(const float *p)   // shared memory
{
    const ulonglong2 v = *reinterpret_cast<const ulonglong2 *>(p);
    return {v.x, v.y};
}
__device__ __forceinline__ f32x2 ex2_pair(f32x2 v)
{
    const float2 h = halves(v);
    return pair(pg_ex2(h.x), pg_ex2(h.y));
}

// A quad of states takes a token (dt and dt x in both halves); returns its part of the read-out.
__device__ __forceinline__ f32x2 update(Quad &S, const Quad &a, f32x2 dt, f32x2 du, const Quad &b, const Quad &c)
{
    S.lo = fma2(ex2_pair(mul2(dt, a.lo)), S.lo, mul2(du, b.lo));
    S.hi = fma2(ex2_pair(mul2(dt, a.hi)), S.hi, mul2(du, b.hi));
    return fma2(S.lo, c.lo, mul2(S.hi, c.hi));
}
__device__ __forceinline__ float sum2(f32x2 v)
{
    const float2 h = halves(v);
    return h.x + h.y;
}

// grid (ceil(inner / 32), ceil(rows / R)).  NC: quads of states per lane
constexpr int SS_W = 4;                  // 16-byte pieces of a row of W_dt that a lane has in flight together
template <int NC, int R, typename TA>
__global__ void __launch_bounds__(SR_T, NC == 1 ? 7 : 1)
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
    const uint4 *wrow = reinterpret_cast<const uint4 *>(s.dt + (int64_t)c * s.dtp) + q;
    const int pieces = live ? s.dtp / 32 : 0;
    uint4 w[SS_W];
#pragma unroll
    for (int k = 0; k < SS_W; k++) w[k] = k < pieces ? __ldg(wrow + 4 * k) : make_uint4(0u, 0u, 0u, 0u);
    Quad a[NC];
#pragma unroll
    for (int i = 0; i < NC; i++)
        a[i] = quad(live && q + 4 * i < quads ? __ldg(reinterpret_cast<const float4 *>(s.a + (int64_t)c * s.ss) + q + 4 * i) : make_float4(0.f, 0.f, 0.f, 0.f));
    const float dt_bias = live ? __ldg(s.dt_bias + c) : 0.0f, skip = live ? __ldg(s.d + c) : 0.0f;
    // neither do the batch's arrays and what earlier steps left
    int slot[R];
    Quad S[R][NC];
#pragma unroll
    for (int r = 0; r < R; r++) slot[r] = live && m0 + r < bt.rows ? __ldcg(bt.d_seq_slot + m0 + r) : -1;   // (one row per sequence)
    auto at = [&](int r) { return reinterpret_cast<float4 *>(state + ((int64_t)slot[r] * s.inner + c) * s.ss) + q; };
#pragma unroll
    for (int r = 0; r < R; r++) {
        const bool old = slot[r] >= 0 && __ldcg(bt.d_pos + m0 + r) > 0;
        // (asked for before the position is there: at position 0 it is dropped)
#pragma unroll
        for (int i = 0; i < NC; i++) {
            const float4 v = slot[r] >= 0 && q + 4 * i < quads ? __ldcg(at(r) + 4 * i) : make_float4(0.f, 0.f, 0.f, 0.f);
            S[r][i] = quad(old ? v : make_float4(0.f, 0.f, 0.f, 0.f));
        }
    }
    asm volatile("griddepcontrol.wait;" ::: "memory");
    float xv[R], z[R];
#pragma unroll
    for (int r = 0; r < R; r++) {
        xv[r] = slot[r] >= 0 ? pg_get(x + (int64_t)(m0 + r) * ldx + c) : 0.0f;
        z[r] = slot[r] >= 0 ? __ldcg(proj + (int64_t)(m0 + r) * ldp + s.inner + c) : 0.0f;
    }
    // the low-rank rows, all copies in flight together
    const uint32_t at_dt = pg_smem(sdt), at_bc = pg_smem(sbc);
    const bool quads_fit = s.N % 4 == 0 && ldl % 4 == 0;
#pragma unroll
    for (int r = 0; r < R; r++) {
        const bool on = m0 + r < bt.rows;
        const float *src = low + (on ? (int64_t)(m0 + r) * ldl : 0);
        if (quads_fit) {
            for (int k = tid * 4; k < s.dtp; k += SR_T * 4) pg_cp_in<16>(at_dt + (r * s.dtp + k) * 4, src + k, on);
            for (int k = tid * 4; k < 2 * NP; k += SR_T * 4) {
                const int which = k / NP, n = k - which * NP;
                pg_cp_in<16>(at_bc + (r * 2 * NP + k) * 4, src + (n < s.N ? s.dtp + which * s.N + n : 0), on && n < s.N);
            }
        } else {
            for (int k = tid; k < s.dtp; k += SR_T) sdt[r * s.dtp + k] = on ? __ldcg(src + k) : 0.0f;
            for (int k = tid; k < 2 * NP; k += SR_T) {
                const int which = k / NP, n = k - which * NP;
                sbc[r * 2 * NP + k] = on && n < s.N ? __ldcg(src + s.dtp + which * s.N + n) : 0.0f;
            }
        }
    }
    pg_cp_commit();
    pg_cp_wait<0>();
    __syncthreads();
    f32x2 sums[R];
#pragma unroll
    for (int r = 0; r < R; r++) sums[r] = pair(0.0f, 0.0f);
    auto dot = [&](const uint4 &b, int k) {
        const f32x2 b0 = pair(pg_bf16_lo(b.x), pg_bf16_hi(b.x)), b1 = pair(pg_bf16_lo(b.y), pg_bf16_hi(b.y)), b2 = pair(pg_bf16_lo(b.z), pg_bf16_hi(b.z)),
                    b3 = pair(pg_bf16_lo(b.w), pg_bf16_hi(b.w));
#pragma unroll
        for (int r = 0; r < R; r++) {
            const float *v = sdt + r * s.dtp + k * 32 + q * 8;
            const Quad u0 = load_quad(v), u1 = load_quad(v + 4);
            sums[r] = fma2(b0, u0.lo, fma2(b1, u0.hi, fma2(b2, u1.lo, fma2(b3, u1.hi, sums[r]))));
        }
    };
    // (all in one stretch: behind the rank's last piece the weights are zero)
#pragma unroll
    for (int k = 0; k < SS_W; k++) dot(w[k], k < pieces ? k : 0);
    for (int k0 = SS_W; k0 < pieces; k0 += SS_W) {
#pragma unroll
        for (int k = 0; k < SS_W; k++) w[k] = k0 + k < pieces ? __ldg(wrow + 4 * (k0 + k)) : make_uint4(0u, 0u, 0u, 0u);
#pragma unroll
        for (int k = 0; k < SS_W; k++) dot(w[k], k0 + k < pieces ? k0 + k : 0);
    }
    float acc[R];
#pragma unroll
    for (int r = 0; r < R; r++) acc[r] = sum2(sums[r]);
#pragma unroll
    for (int r = 0; r < R; r++) acc[r] += __shfl_xor_sync(0xffffffffu, acc[r], 1);
#pragma unroll
    for (int r = 0; r < R; r++) acc[r] += __shfl_xor_sync(0xffffffffu, acc[r], 2);
#pragma unroll
    for (int r = 0; r < R; r++) {
        const float dt = softplus(acc[r] + dt_bias), du = dt * xv[r];
        float y = 0.0f;
#pragma unroll
        for (int i = 0; i < NC; i++) {
            const float *b = sbc + r * 2 * NP + (q + 4 * i) * 4;
            y += sum2(update(S[r][i], a[i], pair(dt, dt), pair(du, du), load_quad(b), load_quad(b + NP)));
            if (slot[r] >= 0 && q + 4 * i < quads) at(r)[4 * i] = quad4(S[r][i]);
        }
        y += __shfl_xor_sync(0xffffffffu, y, 1);
        y += __shfl_xor_sync(0xffffffffu, y, 2);
        if (q == 0 && slot[r] >= 0) pg_put(out + (int64_t)(m0 + r) * ldo + c, fmaf(skip, xv[r], y) * pg_silu(z[r]));
    }
}

// Bytes of one tile as it is brought: dt and z [TT][32] f32, x [TT][32] in the step's type, B and C [TT][2][16 NC] f32.
template <int NC, typename TA>
struct ScanTile {
    static constexpr int NP = 16 * NC, TT = NC > 4 ? 4 : 16;
    static constexpr int Z = TT * SR_CH * 4, X = 2 * Z, BC = X + TT * SR_CH * (int)sizeof(TA), BYTES = BC + TT * 2 * NP * 4;
    static constexpr int DEPTH = 6;      // tiles in shared memory: one being finished, one being run, one being converted, three on their way
};

// grid (ceil(inner / 32), seqs), eight warps.  While warps 0 .. 3 run tile i through the states, warps 4 .. 7 finish the outputs
// of tile i - 1, turn the raw step sizes of tile i + 1 into what the recurrence takes, and ask for tile i + 5 where tile i - 1 lay.
// VEC: rows and channels allow copies of 16 bytes.
template <int NC, typename TA, bool VEC>
__global__ void __launch_bounds__(2 * SR_T)
    scan_run_kernel(const ScanShape s, const pg_batch bt, const float *__restrict__ proj, int64_t ldp, float *ring, const TA *__restrict__ x, int64_t ldx,
                    const float *__restrict__ dt, int64_t ldt, const float *__restrict__ bc, int64_t ldb, float *state, TA *__restrict__ out, int64_t ldo)
{
    using Tile = ScanTile<NC, TA>;
    constexpr int NP = Tile::NP, TT = Tile::TT, DEPTH = Tile::DEPTH, PER = TT * SR_CH / SR_T;
    extern __shared__ __align__(16) float sm[];            // [DEPTH] tiles
    __shared__ __align__(16) float4 sd[2][TT][SR_CH];      // dt, dt, dt x, dt x
    __shared__ float sy[2][TT][SR_CH];
    pg_pdl_begin();
    const bool aux = threadIdx.x >= SR_T;
    const int tid = threadIdx.x & (SR_T - 1), c0 = blockIdx.x * SR_CH;
    const int seq = blockIdx.y, row0 = __ldcg(bt.d_seq_row0 + seq), T = __ldcg(bt.d_seq_row0 + seq + 1) - row0;
    if (T <= 0) return;
    const int pos0 = __ldcg(bt.d_pos + row0), tiles = (T + TT - 1) / TT;
    const int64_t slot = __ldcg(bt.d_seq_slot + seq);
    const unsigned char *raw = reinterpret_cast<const unsigned char *>(sm);
    if (aux) {
        // tokens tid / 32 + 4 i of channel tid % 32
        const int cx = tid & 31, ec = c0 + cx, et = tid >> 5;
        const bool on = ec < s.inner;
        const float dt_bias = on ? __ldg(s.dt_bias + ec) : 0.0f, skip = on ? __ldg(s.d + ec) : 0.0f;
        const uint32_t sm_at = pg_smem(sm);
        auto fetch = [&](int tile) {
            const uint32_t at = sm_at + (uint32_t)(tile % DEPTH) * Tile::BYTES;
            const int t0 = tile * TT;
            constexpr int V = VEC ? 4 : 1;                 // f32 elements of a copy
#pragma unroll
            for (int e = tid * V; e < TT * SR_CH; e += SR_T * V) {
                const int t = e / SR_CH, c = e % SR_CH;
                const bool in = t0 + t < T && c0 + c < s.inner;
                const int64_t m = in ? row0 + t0 + t : row0;
                const int64_t ch = in ? c0 + c : 0;
                pg_cp_in<4 * V>(at + e * 4, dt + m * ldt + ch, in);
                pg_cp_in<4 * V>(at + Tile::Z + e * 4, proj + m * ldp + s.inner + ch, in);
            }
            constexpr int VX = VEC ? 16 / (int)sizeof(TA) : 4 / (int)sizeof(TA);
#pragma unroll
            for (int e = tid * VX; e < TT * SR_CH; e += SR_T * VX) {
                const int t = e / SR_CH, c = e % SR_CH;
                const bool in = t0 + t < T && c0 + c < s.inner;   // (a pair may reach one column behind the last channel: ldx is even)
                pg_cp_in<VX * (int)sizeof(TA)>(at + Tile::X + e * (int)sizeof(TA), x + (in ? (row0 + t0 + t) * ldx + c0 + c : 0), in);
            }
#pragma unroll
            for (int e = tid * V; e < TT * 2 * NP; e += SR_T * V) {
                const int t = e / (2 * NP), k = e % (2 * NP), which = k / NP, n = k - which * NP;
                const bool in = t0 + t < T && n < s.N;
                pg_cp_in<4 * V>(at + Tile::BC + e * 4, bc + (in ? (int64_t)(row0 + t0 + t) * ldb + which * s.N + n : 0), in);
            }
            pg_cp_commit();
        };
        auto x_of = [&](const unsigned char *at, int t) { return pg_get_plain(reinterpret_cast<const TA *>(at + Tile::X) + t * SR_CH + cx); };
        auto convert = [&](int tile) {
            const unsigned char *at = raw + (size_t)(tile % DEPTH) * Tile::BYTES;
#pragma unroll
            for (int i = 0; i < PER; i++) {
                const int t = et + i * (SR_T / 32);
                // (tokens behind the end leave the state alone: exp(0) S + 0)
                const float r = reinterpret_cast<const float *>(at)[t * SR_CH + cx];
                const float d = on && tile * TT + t < T ? softplus(r + dt_bias) : 0.0f, u = d * x_of(at, t);
                sd[tile & 1][t][cx] = make_float4(d, d, u, u);
            }
        };
        auto finish = [&](int tile) {
            const unsigned char *at = raw + (size_t)(tile % DEPTH) * Tile::BYTES;
#pragma unroll
            for (int i = 0; i < PER; i++) {
                const int t = et + i * (SR_T / 32);
                const float z = reinterpret_cast<const float *>(at + Tile::Z)[t * SR_CH + cx];
                const float y = fmaf(skip, x_of(at, t), sy[tile & 1][t][cx]) * pg_silu(z);
                if (on && tile * TT + t < T) pg_put(out + (int64_t)(row0 + tile * TT + t) * ldo + ec, y);
            }
        };
        // (the warps of this half meet on their own where one has copied what another reads)
        auto landed = [&]() {
            pg_cp_wait<DEPTH - 3>();
            asm volatile("bar.sync 1, 128;" ::: "memory");
        };
        // one group of copies per tile, empty behind the end, so that the wait counts tiles
        for (int i = 0; i < DEPTH - 1; i++) {
            if (i < tiles)
                fetch(i);
            else
                pg_cp_commit();
        }
        pg_cp_wait<DEPTH - 2>();
        asm volatile("bar.sync 1, 128;" ::: "memory");
        convert(0);
        for (int i = 0; i < tiles; i++) {
            __syncthreads();                              // tile i may be run; tile i - 1 has been
            if (i > 0) finish(i - 1);
            landed();                                     // tile i + 1; tile i - 1 is finished everywhere
            if (i + 1 < tiles) convert(i + 1);
            if (i + DEPTH - 1 < tiles)
                fetch(i + DEPTH - 1);
            else
                pg_cp_commit();
        }
        __syncthreads();
        finish(tiles - 1);
        pg_cp_wait<0>();
        // the inputs that the next portion's convolution reads (scan_conv_kernel is done with the old ones)
        if (on)
            for (int t = max(0, T - s.taps) + et; t < T; t += SR_T / 32)
                ring[(slot * s.taps + (pos0 + t) % s.taps) * s.inner + ec] = __ldcg(proj + (int64_t)(row0 + t) * ldp + ec);
        return;
    }
    const int q = tid & 3, cl = tid >> 2, c = c0 + cl, quads = s.ss / 4;
    const bool live = c < s.inner;
    float4 *st = reinterpret_cast<float4 *>(state + (slot * s.inner + c) * s.ss);
    Quad a[NC], S[NC];
#pragma unroll
    for (int i = 0; i < NC; i++) {
        const bool on = live && q + 4 * i < quads;
        a[i] = quad(on ? __ldg(reinterpret_cast<const float4 *>(s.a + (int64_t)c * s.ss) + q + 4 * i) : make_float4(0.f, 0.f, 0.f, 0.f));
        S[i] = quad(on && pos0 > 0 ? __ldcg(st + q + 4 * i) : make_float4(0.f, 0.f, 0.f, 0.f));
    }
    for (int i = 0; i < tiles; i++) {
        __syncthreads();
        const int b = i & 1;
        const float *sbc = reinterpret_cast<const float *>(raw + (size_t)(i % DEPTH) * Tile::BYTES + Tile::BC);
        float y[TT];
#pragma unroll
        for (int t = 0; t < TT; t += 4) {
            // four tokens: everything that does not depend on the state first, then the chain
            f32x2 part[4];
#pragma unroll
            for (int n = 0; n < NC; n++) {
                Quad e[4], g[4], c4[4];
#pragma unroll
                for (int u = 0; u < 4; u++) {
                    const Quad d = load_quad(reinterpret_cast<const float *>(&sd[b][t + u][cl])), bb = load_quad(sbc + (t + u) * 2 * NP + (q + 4 * n) * 4);
                    c4[u] = load_quad(sbc + (t + u) * 2 * NP + NP + (q + 4 * n) * 4);
                    e[u] = {mul2(d.lo, a[n].lo), mul2(d.lo, a[n].hi)};
                    g[u] = {mul2(d.hi, bb.lo), mul2(d.hi, bb.hi)};
                }
#pragma unroll
                for (int u = 0; u < 4; u++) e[u] = {ex2_pair(e[u].lo), ex2_pair(e[u].hi)};
#pragma unroll
                for (int u = 0; u < 4; u++) {
                    S[n].lo = fma2(e[u].lo, S[n].lo, g[u].lo);
                    S[n].hi = fma2(e[u].hi, S[n].hi, g[u].hi);
                    part[u] = n == 0 ? mul2(S[n].lo, c4[u].lo) : fma2(S[n].lo, c4[u].lo, part[u]);
                    part[u] = fma2(S[n].hi, c4[u].hi, part[u]);
                }
            }
#pragma unroll
            for (int u = 0; u < 4; u++) y[t + u] = sum2(part[u]);
        }
        // four tokens' sums over four lanes: lane q ends with token q's
        const bool odd = q & 1, up = q & 2;
#pragma unroll
        for (int t = 0; t < TT; t += 4) {
            const float g0 = __shfl_xor_sync(0xffffffffu, odd ? y[t] : y[t + 1], 1), g1 = __shfl_xor_sync(0xffffffffu, odd ? y[t + 2] : y[t + 3], 1);
            const float k0 = (odd ? y[t + 1] : y[t]) + g0, k1 = (odd ? y[t + 3] : y[t + 2]) + g1;
            const float g2 = __shfl_xor_sync(0xffffffffu, up ? k0 : k1, 2);
            sy[b][t + q][cl] = (up ? k1 : k0) + g2;
        }
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < NC; i++)
        if (live && q + 4 * i < quads) st[q + 4 * i] = quad4(S[i]);
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
    PG_REQUIRE(ldx % 2 == 0 && ((uintptr_t)x & 3) == 0, "scan: rows of x start on 4-byte boundaries");
    const bool vec = s.inner % 8 == 0 && s.N % 4 == 0 && ldt % 4 == 0 && ldp % 4 == 0 && ldb % 4 == 0 && ldx % 8 == 0 &&
                     (((uintptr_t)dt | (uintptr_t)proj | (uintptr_t)bc | (uintptr_t)x) & 15) == 0;
    auto go = [&](auto kern, std::atomic<uint64_t> &set, int smem) -> int32_t {
        PG_CUDA(pg_max_smem_once(kern, smem, ctx->device, set));
        return launch_whole(ctx, kern, grid, dim3(2 * SR_T), (size_t)smem, s, *bt, proj, ldp, ring, x, ldx, dt, ldt, bc, ldb, state, out, ldo);
    };
#define PG_SR(NC, I)                                                                                                    \
    do {                                                                                                                \
        constexpr int smem = ScanTile<NC, TA>::DEPTH * ScanTile<NC, TA>::BYTES;                                         \
        return vec ? go(scan_run_kernel<NC, TA, true>, set[2 * I], smem) : go(scan_run_kernel<NC, TA, false>, set[2 * I + 1], smem); \
    } while (0)
    static std::atomic<uint64_t> set[10] = {};
    if (s.N <= 16) PG_SR(1, 0);
    if (s.N <= 32) PG_SR(2, 1);
    if (s.N <= 64) PG_SR(4, 2);
    if (s.N <= 128) PG_SR(8, 3);
    PG_SR(16, 4);
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
