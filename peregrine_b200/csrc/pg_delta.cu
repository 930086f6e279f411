// Gated delta rule with short causal convolutions.
//
// Per token and head (S: dim x vdim, f32):  S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q.
// Both read-outs can be taken from the S the token finds:  S^T k and S^T q of the old state give
//   u = beta (v - g S^T k),   o = g S^T q + (k . q) u,
// so a token needs one pass of reductions over the state before the update.
//
//   one token per sequence   delta_step_kernel: convolution, unit norms, gates, the state update and the gated output
//                            norm of one (head, sequence) in one CTA; the state is read and written once
//   longer portions          delta_prep_kernel (convolution, unit norms, gates; a CTA per four tokens), delta_scan_kernel
//                            (the recurrence, four tokens at a time: their read-outs come from the state the first of them
//                            finds, corrected by the pairs' products k_a . k_b and q_a . k_b, so that one round of
//                            reductions serves four tokens; a warp holds eight columns of a head's state in registers),
//                            delta_out_kernel (output norm and gate; also stores the convolution inputs that the next
//                            portion needs)
//
// Convolution inputs are kept per slot in a ring of `taps` entries, position p in entry p mod taps: a single token
// writes an entry that nobody reads any more, so heads that share channels need no order among their CTAs.
// A sequence starts at position 0: what its slot holds is then taken as zero.
#include "pg_async.cuh"
#include "pg_lm.cuh"

namespace {

struct DeltaShape {
    int H, G, D, V, taps, C;        // C: convolution channels 2 G D + H V
    int vs;                         // state row stride
    float eps, unit_eps, qscale;
    const float *conv, *a_log, *dt_bias, *norm;
};

__device__ __forceinline__ float softplus(float x) { return x > 20.0f ? x : log1pf(expf(x)); }
__device__ __forceinline__ float log_decay(float a, float a_log, float dt_bias) { return -expf(a_log) * softplus(a + dt_bias); }

// one channel of the convolution at position pos; row: this token's input row, t: tokens of the same sequence and step
// in front of it; older inputs come from the ring
__device__ __forceinline__ float conv_at(const DeltaShape &s, const float *row, int64_t ldp, const float *ring, int c, int t, int pos)
{
    float acc = 0.0f;
    for (int j = 0; j < s.taps; j++) {
        const int back = s.taps - 1 - j;                  // tokens back
        float x = 0.0f;
        if (back <= t)
            x = __ldcg(row - (int64_t)back * ldp + c);
        else if (back <= pos)
            x = __ldcg(ring + (int64_t)((pos - back) % s.taps) * s.C + c);
        acc = fmaf(__ldg(s.conv + (int64_t)j * s.C + c), x, acc);
    }
    return pg_silu(acc);
}

// ---- one token per sequence: grid (H, rows) ----------------------------------------------------------------------
constexpr int DS_T = 256;
constexpr int DS_KEEP = 16;      // state rows per thread that stay in registers between the two passes

// TAPS: the number of taps, 0 = any
template <int TAPS, typename TA>
__global__ void __launch_bounds__(DS_T)
    delta_step_kernel(const DeltaShape s, const float *__restrict__ proj, int64_t ldp, const int32_t *__restrict__ positions,
                      const int32_t *__restrict__ slots, float *ring, float *state, TA *__restrict__ out, int64_t ldo)
{
    extern __shared__ __align__(16) float sm[];   // k[D] | q[D] | v[vs] | o[vs] | partials [2][groups][vs]
    __shared__ float red[32];
    __shared__ float bc[4];
    pg_pdl_begin();
    const int h = blockIdx.x, b = blockIdx.y, rep = s.H / s.G, g = h / rep, tid = threadIdx.x;
    const int pos = __ldcg(positions + b);
    const int64_t slot = __ldcg(slots + b);
    const float *row = proj + (int64_t)b * ldp;
    float *rg = ring + slot * s.taps * s.C;
    float *st = state + (slot * s.H + h) * (int64_t)s.D * s.vs;
    const int dp = (s.D + 3) & ~3;
    float *sk = sm, *sq = sk + dp, *sv = sq + dp, *so = sv + s.vs, *pk = so + s.vs;
    const int vq = s.vs / 4, cpt = min(vq, DS_T), groups = DS_T / cpt;
    float *pq = pk + (size_t)groups * s.vs;

    // what the end of the kernel needs and the state's rows are asked for first
    const float *tail = row + s.C + (int64_t)s.H * s.V;
    const float in_b = __ldcg(tail + h), in_a = __ldcg(tail + s.H + h);
    float in_gate[4];                                     // vdim <= 1024
#pragma unroll
    for (int i = 0; i < 4; i++) in_gate[i] = tid + i * DS_T < s.V ? __ldcg(row + s.C + (int64_t)h * s.V + tid + i * DS_T) : 0.0f;
    const int rgid = tid / cpt, cv = tid - rgid * cpt;    // row group, column quad (in steps of cpt quads)
    const bool live = rgid < groups;
    float4 keep[DS_KEEP];
    if (live && cv < vq && pos > 0) {
#pragma unroll
        for (int i = 0; i < DS_KEEP; i++) {
            const int r = rgid + i * groups;
            keep[i] = r < s.D ? __ldcg(reinterpret_cast<const float4 *>(st + (int64_t)r * s.vs) + cv) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
    } else {
#pragma unroll
        for (int i = 0; i < DS_KEEP; i++) keep[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    }

    const int cq = g * s.D, ck = s.G * s.D + g * s.D, cvv = 2 * s.G * s.D + h * s.V;
    const int now = pos % s.taps;
    // two channels per round, all their loads in flight together
    for (int i0 = tid; i0 < 2 * s.D + s.V; i0 += 2 * DS_T) {
        int ch[2];
        float y[2], in[2];
#pragma unroll
        for (int u = 0; u < 2; u++) {
            const int i = i0 + u * DS_T;
            ch[u] = i >= 2 * s.D + s.V ? -1 : i < s.D ? cq + i : (i < 2 * s.D ? ck + i - s.D : cvv + i - 2 * s.D);
        }
        if constexpr (TAPS > 0) {
            float x[2][TAPS], wt[2][TAPS];
#pragma unroll
            for (int u = 0; u < 2; u++)
#pragma unroll
                for (int j = 0; j < TAPS; j++) {
                    const int back = TAPS - 1 - j;
                    const int at = now - back < 0 ? now - back + TAPS : now - back;
                    x[u][j] = ch[u] < 0 || back > pos ? 0.0f : back == 0 ? __ldcg(row + ch[u]) : __ldcg(rg + (int64_t)at * s.C + ch[u]);
                    wt[u][j] = ch[u] < 0 ? 0.0f : __ldg(s.conv + (int64_t)j * s.C + ch[u]);
                }
#pragma unroll
            for (int u = 0; u < 2; u++) {
                float acc = 0.0f;
#pragma unroll
                for (int j = 0; j < TAPS; j++) acc = fmaf(wt[u][j], x[u][j], acc);
                y[u] = pg_silu(acc);
                in[u] = x[u][TAPS - 1];
            }
        } else {
#pragma unroll
            for (int u = 0; u < 2; u++) {
                y[u] = ch[u] < 0 ? 0.0f : conv_at(s, row, ldp, rg, ch[u], 0, pos);
                in[u] = ch[u] < 0 ? 0.0f : __ldcg(row + ch[u]);
            }
        }
#pragma unroll
        for (int u = 0; u < 2; u++) {
            const int i = i0 + u * DS_T;
            if (ch[u] < 0) continue;
            if (i < s.D)
                sq[i] = y[u];
            else if (i < 2 * s.D)
                sk[i - s.D] = y[u];
            else
                sv[i - 2 * s.D] = y[u];
            // the entry this position takes is older than anything a convolution still reads
            if (i >= 2 * s.D || h % rep == 0) rg[(int64_t)now * s.C + ch[u]] = in[u];
        }
    }
    for (int i = s.V + tid; i < s.vs; i += DS_T) sv[i] = 0.0f;
    __syncthreads();
    if (tid < 64) {
        float *x = tid < 32 ? sq : sk;
        const int lane = tid & 31;
        float ss = 0.0f;
        for (int i = lane; i < s.D; i += 32) ss += x[i] * x[i];
        ss = pg_warp_sum(ss);
        const float inv = __fdiv_rn(tid < 32 ? s.qscale : 1.0f, sqrtf(ss + s.unit_eps));
        for (int i = lane; i < s.D; i += 32) x[i] *= inv;
    } else if (tid == 64) {
        bc[0] = pg_sigmoid(in_b);
        bc[1] = expf(log_decay(in_a, __ldg(s.a_log + h), __ldg(s.dt_bias + h)));
    }
    __syncthreads();
    if (tid < 32) {
        float kq = 0.0f;
        for (int i = tid; i < s.D; i += 32) kq += sk[i] * sq[i];
        kq = pg_warp_sum(kq);
        if (tid == 0) bc[2] = kq;
    }
    // S^T k and S^T q of the old state
    if (live) {
        for (int c0 = cv; c0 < vq; c0 += cpt) {
            float4 ak = make_float4(0.f, 0.f, 0.f, 0.f), aq = ak;
            auto add = [&](int r, float4 x) {
                const float kk = sk[r], qq = sq[r];
                ak.x = fmaf(kk, x.x, ak.x), ak.y = fmaf(kk, x.y, ak.y), ak.z = fmaf(kk, x.z, ak.z), ak.w = fmaf(kk, x.w, ak.w);
                aq.x = fmaf(qq, x.x, aq.x), aq.y = fmaf(qq, x.y, aq.y), aq.z = fmaf(qq, x.z, aq.z), aq.w = fmaf(qq, x.w, aq.w);
            };
            if (c0 == cv) {
#pragma unroll
                for (int i = 0; i < DS_KEEP; i++)
                    if (rgid + i * groups < s.D) add(rgid + i * groups, keep[i]);
            }
            if (pos > 0)
                for (int r = rgid + (c0 == cv ? DS_KEEP * groups : 0); r < s.D; r += groups)
                    add(r, __ldcg(reinterpret_cast<const float4 *>(st + (int64_t)r * s.vs) + c0));
            reinterpret_cast<float4 *>(pk + (size_t)rgid * s.vs)[c0] = ak;
            reinterpret_cast<float4 *>(pq + (size_t)rgid * s.vs)[c0] = aq;
        }
    }
    __syncthreads();
    const float beta = bc[0], dec = bc[1], kq = bc[2];
    for (int c = tid; c < s.vs; c += DS_T) {
        float a = 0.0f, q = 0.0f;
        for (int r = 0; r < groups; r++) {
            a += pk[(size_t)r * s.vs + c];
            q += pq[(size_t)r * s.vs + c];
        }
        const float u = c < s.V ? beta * (sv[c] - dec * a) : 0.0f;
        sv[c] = u;
        so[c] = dec * q + kq * u;
    }
    __syncthreads();
    if (live) {
        for (int c0 = cv; c0 < vq; c0 += cpt) {
            const float4 u = reinterpret_cast<const float4 *>(sv)[c0];
            auto put = [&](int r, float4 x) {
                const float kk = sk[r];
                x.x = fmaf(kk, u.x, dec * x.x), x.y = fmaf(kk, u.y, dec * x.y), x.z = fmaf(kk, u.z, dec * x.z), x.w = fmaf(kk, u.w, dec * x.w);
                reinterpret_cast<float4 *>(st + (int64_t)r * s.vs)[c0] = x;
            };
            if (c0 == cv) {
#pragma unroll
                for (int i = 0; i < DS_KEEP; i++)
                    if (rgid + i * groups < s.D) put(rgid + i * groups, keep[i]);
            }
            for (int r = rgid + (c0 == cv ? DS_KEEP * groups : 0); r < s.D; r += groups)
                put(r, pos > 0 ? __ldcg(reinterpret_cast<const float4 *>(st + (int64_t)r * s.vs) + c0) : make_float4(0.f, 0.f, 0.f, 0.f));
        }
    }
    float ss = 0.0f;
    for (int c = tid; c < s.V; c += DS_T) ss += so[c] * so[c];
    ss = pg_block_sum(ss, red);
    const float inv = __fdiv_rn(1.0f, sqrtf(__fdiv_rn(ss, (float)s.V) + s.eps));
#pragma unroll
    for (int i = 0; i < 4; i++) {
        const int c = tid + i * DS_T;
        if (c < s.V) pg_put(out + (int64_t)b * ldo + (int64_t)h * s.V + c, so[c] * inv * __ldg(s.norm + c) * pg_silu(in_gate[i]));
    }
}

// ---- longer portions ---------------------------------------------------------------------------------------------
// work rows: q [G D] | k [G D] | v [H V] | o [H V] per token; coef: 32 floats per block of four tokens and head.  With the
// decays g_a of a block's tokens, c_a = g_0 .. g_a and r_ab = g_{b+1} .. g_a:
//   u_a = beta_a (v_a - c_a S^T k_a - sum_{b<a} r_ab (k_b . k_a) u_b)
//   o_a = c_a S^T q_a + sum_{b<=a} r_ab (k_b . q_a) u_b
//   S <- c_3 S + sum_b r_3b k_b u_b^T
// coef: c [4] | beta [4] | r_3b [4] | r_ab (k_b . k_a) of the 6 pairs b < a | r_ab (k_b . q_a) of the 10 pairs b <= a
struct DeltaWork {
    float *q, *k, *v, *o, *coef;
};
constexpr int BT = 4;            // tokens of a block
// blocks of a sequence are numbered from here on
__device__ __forceinline__ int64_t first_block(int row0, int seq) { return row0 / BT + seq; }

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
template <int V>
__device__ __forceinline__ void store_lanes(float *p, const Lanes<V> &r)
{
    if constexpr (V == 4)
        *reinterpret_cast<float4 *>(p) = make_float4(r.v[0], r.v[1], r.v[2], r.v[3]);
    else
        *p = r.v[0];
}

// grid (ceil(longest / 4), seqs).  TAPS: the number of taps, 0 = any; V: channels per thread and round (4 where rows and
// groups of channels start on 16-byte boundaries)
template <int TAPS, int V>
__global__ void __launch_bounds__(256)
    delta_prep_kernel(const DeltaShape s, const pg_batch bt, const float *__restrict__ proj, int64_t ldp, const float *__restrict__ ring, const DeltaWork w)
{
    extern __shared__ __align__(16) float sm[];   // q and k channels [4][2 G D], then the pairs' products [G][16]
    pg_pdl_begin();
    const int seq = blockIdx.y, row0 = __ldcg(bt.d_seq_row0 + seq), T = __ldcg(bt.d_seq_row0 + seq + 1) - row0;
    const int t0 = blockIdx.x * BT, n = min(BT, T - t0), m0 = row0 + t0;
    if (n <= 0) return;
    const int pos0 = __ldcg(bt.d_pos + row0);
    const float *row = proj + (int64_t)m0 * ldp;
    const float *rg = ring + (int64_t)__ldcg(bt.d_seq_slot + seq) * s.taps * s.C;
    const int qk = 2 * s.G * s.D;
    float *dots = sm + (size_t)BT * qk;
    for (int c = threadIdx.x * V; c < s.C; c += 256 * V) {
        Lanes<V> y[BT];
        if constexpr (TAPS > 0) {
            Lanes<V> x[TAPS - 1 + BT], wt[TAPS];
#pragma unroll
            for (int j = 0; j < TAPS - 1 + BT; j++) {
                const int t = t0 + j - (TAPS - 1);        // of the sequence's tokens in this step
                x[j] = Lanes<V>{};
                if (t >= 0) {
                    if (t < T) x[j] = load_lanes<V>(row + (int64_t)(j - (TAPS - 1)) * ldp + c);
                } else if (pos0 + t >= 0) {
                    x[j] = load_lanes<V>(rg + (int64_t)((pos0 + t) % TAPS) * s.C + c);
                }
            }
#pragma unroll
            for (int j = 0; j < TAPS; j++) wt[j] = load_lanes<V>(s.conv + (int64_t)j * s.C + c);
#pragma unroll
            for (int a = 0; a < BT; a++)
#pragma unroll
                for (int i = 0; i < V; i++) {
                    float acc = 0.0f;
#pragma unroll
                    for (int j = 0; j < TAPS; j++) acc = fmaf(wt[j].v[i], x[a + j].v[i], acc);
                    y[a].v[i] = pg_silu(acc);
                }
        } else {
#pragma unroll
            for (int a = 0; a < BT; a++)
#pragma unroll
                for (int i = 0; i < V; i++) y[a].v[i] = a < n ? conv_at(s, row + (int64_t)a * ldp, ldp, rg, c + i, t0 + a, pos0 + t0 + a) : 0.0f;
        }
#pragma unroll
        for (int a = 0; a < BT; a++) {
            if (c < qk)
                store_lanes<V>(sm + (size_t)a * qk + c, a < n ? y[a] : Lanes<V>{});
            else if (a < n)
                store_lanes<V>(w.v + (int64_t)(m0 + a) * s.H * s.V + c - qk, y[a]);
        }
    }
    __syncthreads();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    for (int i = warp; i < BT * 2 * s.G; i += 8) {        // unit norms: (token, q or k, head)
        const int a = i / (2 * s.G), hd = i - a * 2 * s.G;
        float *x = sm + (size_t)a * qk + hd * s.D;
        float ss = 0.0f;
        for (int d = lane; d < s.D; d += 32) ss += x[d] * x[d];
        ss = pg_warp_sum(ss);
        const bool is_q = hd < s.G;
        const float inv = __fdiv_rn(is_q ? s.qscale : 1.0f, sqrtf(ss + s.unit_eps));
        float *dst = (is_q ? w.q : w.k) + ((int64_t)(m0 + a) * s.G + (is_q ? hd : hd - s.G)) * s.D;
        for (int d = lane; d < s.D; d += 32) {
            const float y = x[d] * inv;
            x[d] = y;
            if (a < n) dst[d] = y;
        }
    }
    __syncthreads();
    for (int g = warp; g < s.G; g += 8) {                 // the pairs' products
        float p[16] = {};
        for (int d = lane; d < s.D; d += 32) {
            float q[BT], k[BT];
#pragma unroll
            for (int a = 0; a < BT; a++) {
                q[a] = sm[(size_t)a * qk + g * s.D + d];
                k[a] = sm[(size_t)a * qk + (s.G + g) * s.D + d];
            }
#pragma unroll
            for (int a = 0, i = 0, j = 6; a < BT; a++)
#pragma unroll
                for (int b = 0; b <= a; b++) {
                    if (b < a) p[i] = fmaf(k[b], k[a], p[i]), i++;
                    p[j] = fmaf(k[b], q[a], p[j]), j++;
                }
        }
#pragma unroll
        for (int i = 0; i < 16; i++) {
            p[i] = pg_warp_sum(p[i]);
            if (lane == i) dots[g * 16 + i] = p[i];
        }
    }
    __syncthreads();
    for (int h = threadIdx.x; h < s.H; h += 256) {
        const float *dp = dots + h / (s.H / s.G) * 16;
        const float al = __ldg(s.a_log + h), db = __ldg(s.dt_bias + h);
        float g[BT], o[32];
#pragma unroll
        for (int a = 0; a < BT; a++) {
            const float *tail = row + (int64_t)a * ldp + s.C + (int64_t)s.H * s.V;
            g[a] = a < n ? expf(log_decay(__ldcg(tail + s.H + h), al, db)) : 1.0f;
            o[4 + a] = a < n ? pg_sigmoid(__ldcg(tail + h)) : 0.0f;
            o[a] = a ? o[a - 1] * g[a] : g[0];
        }
        o[11] = 1.0f;
#pragma unroll
        for (int b = BT - 2; b >= 0; b--) o[8 + b] = o[9 + b] * g[b + 1];
#pragma unroll
        for (int a = 0, i = 0, j = 6; a < BT; a++)
#pragma unroll
            for (int b = 0; b <= a; b++) {
                float r = 1.0f;
#pragma unroll
                for (int x = b + 1; x <= a; x++) r *= g[x];
                if (b < a) o[12 + i] = r * dp[i], i++;
                o[12 + j] = r * dp[j], j++;
            }
        float4 *dst = reinterpret_cast<float4 *>(w.coef + ((first_block(row0, seq) + blockIdx.x) * s.H + h) * 32);
        o[28] = o[29] = o[30] = o[31] = 0.0f;
#pragma unroll
        for (int i = 0; i < 8; i++) dst[i] = make_float4(o[4 * i], o[4 * i + 1], o[4 * i + 2], o[4 * i + 3]);
    }
}

typedef unsigned long long f32x2;    // two f32 in a register pair
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c)
{
    f32x2 d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b)
{
    f32x2 d;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}
__device__ __forceinline__ f32x2 pack2(float lo, float hi)
{
    f32x2 d;
    asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(lo), "f"(hi));
    return d;
}
__device__ __forceinline__ float sum2(f32x2 v)
{
    float lo, hi;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v));
    return lo + hi;
}
struct __align__(16) Quad {
    f32x2 lo, hi;
};

// grid (ceil(V / 32), H, seqs), 4 warps.  Warp w: columns 8 w .. 8 w + 7 of the CTA's 32.  Eight lanes share two columns:
// lane l = lane & 7 holds rows l * 4 + 32 i .. + 3 (i < NI) of columns 2 (lane >> 3) and 2 (lane >> 3) + 1, and does a block's
// algebra for the column of its parity.
template <int NI>
struct ScanTile {
    static constexpr int DP = NI * 32;
    static constexpr int TB = NI <= 4 ? 16 : 8;           // tokens per tile
    static constexpr int STAGES = 3;
    struct Stage {
        float k[TB][DP], q[TB][DP], v[TB][32], coef[TB / BT][32];
    };
};

template <int NI>
__global__ void __launch_bounds__(128) delta_scan_kernel(const DeltaShape s, const pg_batch bt, const DeltaWork w, float *state)
{
    using C = ScanTile<NI>;
    constexpr int DP = C::DP, TB = C::TB;
    extern __shared__ __align__(16) unsigned char smem[];
    typename C::Stage *stages = reinterpret_cast<typename C::Stage *>(smem);
    // (launched whole, and the successor is not let in early either)
    const int h = blockIdx.y, seq = blockIdx.z, g = h / (s.H / s.G), tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int row0 = __ldcg(bt.d_seq_row0 + seq), T = __ldcg(bt.d_seq_row0 + seq + 1) - row0;
    if (T <= 0) return;
    const int pos0 = __ldcg(bt.d_pos + row0);
    const int c0 = blockIdx.x * 32, col = warp * 8 + (lane >> 3) * 2, l = lane & 7, par = lane & 1;
    const int64_t block0 = first_block(row0, seq);
    float *st = state + ((int64_t)__ldcg(bt.d_seq_slot + seq) * s.H + h) * (int64_t)s.D * s.vs + c0 + col;
    f32x2 S[2][NI][2];
#pragma unroll
    for (int c = 0; c < 2; c++)
#pragma unroll
        for (int i = 0; i < NI; i++)
#pragma unroll
            for (int j = 0; j < 2; j++) {
                const int r = l * 4 + 32 * i + 2 * j;
                const bool in = pos0 > 0 && c0 + col + c < s.V;
                S[c][i][j] = pack2((in && r < s.D) ? __ldcg(st + (int64_t)r * s.vs + c) : 0.0f, (in && r + 1 < s.D) ? __ldcg(st + (int64_t)(r + 1) * s.vs + c) : 0.0f);
            }
    // A tile into shared memory; rows of q and k behind D, columns behind V and tokens behind T are zero.  (16-byte copies
    // that bypass L1 where the shape allows them.)
    const bool vec = ((s.D | s.V) & 3) == 0;
    auto fetch = [&](int tile) {
        typename C::Stage &e = stages[tile % C::STAGES];
        const int t0 = tile * TB, n = min(TB, T - t0);
        if (n > 0) {
            for (int i = tid; i < TB * DP / 4; i += 128) {
                const int t = i / (DP / 4), d = (i - t * (DP / 4)) * 4;
                const int64_t at = ((int64_t)(row0 + t0 + t) * s.G + g) * s.D + d;
                if (vec && t < n && d < s.D) {
                    pg_cp16(pg_smem(&e.k[t][d]), w.k + at);
                    pg_cp16(pg_smem(&e.q[t][d]), w.q + at);
                } else {
#pragma unroll
                    for (int j = 0; j < 4; j++) {
                        const bool in = t < n && d + j < s.D;
                        e.k[t][d + j] = in ? __ldcg(w.k + at + j) : 0.0f;
                        e.q[t][d + j] = in ? __ldcg(w.q + at + j) : 0.0f;
                    }
                }
            }
            for (int i = tid; i < TB * 8; i += 128) {
                const int t = i / 8, c = (i & 7) * 4;
                const float *v = w.v + (int64_t)(row0 + t0 + t) * s.H * s.V + (int64_t)h * s.V + c0 + c;
                if (vec && t < n && c0 + c < s.V) {
                    pg_cp16(pg_smem(&e.v[t][c]), v);
                } else {
#pragma unroll
                    for (int j = 0; j < 4; j++) e.v[t][c + j] = (t < n && c0 + c + j < s.V) ? __ldcg(v + j) : 0.0f;
                }
            }
            if (tid < TB / BT * 8) {
                const int bi = tid / 8;
                if (bi * BT < n) pg_cp16(pg_smem(&e.coef[bi][(tid & 7) * 4]), w.coef + ((block0 + t0 / BT + bi) * s.H + h) * 32 + (tid & 7) * 4);
            }
        }
        pg_cp_commit();
    };
    const int tiles = (T + TB - 1) / TB;
    fetch(0);
    fetch(1);
    for (int tile = 0; tile < tiles; tile++) {
        fetch(tile + 2);                                  // its stage was left behind the last barrier
        pg_cp_wait<2>();
        __syncthreads();
        const typename C::Stage &e = stages[tile % C::STAGES];
        const int t0 = tile * TB, blocks = (min(TB, T - t0) + BT - 1) / BT;
        for (int bi = 0; bi < blocks; bi++) {
            const float(*kt)[DP] = &e.k[bi * BT], (*qt)[DP] = &e.q[bi * BT];
            f32x2 ak[BT][2] = {}, aq[BT][2] = {};
#pragma unroll
            for (int i = 0; i < NI; i++) {
#pragma unroll
                for (int a = 0; a < BT; a++) {
                    const Quad k = *reinterpret_cast<const Quad *>(&kt[a][l * 4 + 32 * i]), q = *reinterpret_cast<const Quad *>(&qt[a][l * 4 + 32 * i]);
#pragma unroll
                    for (int c = 0; c < 2; c++) {
                        ak[a][c] = fma2(k.lo, S[c][i][0], ak[a][c]);
                        ak[a][c] = fma2(k.hi, S[c][i][1], ak[a][c]);
                        aq[a][c] = fma2(q.lo, S[c][i][0], aq[a][c]);
                        aq[a][c] = fma2(q.hi, S[c][i][1], aq[a][c]);
                    }
                }
            }
            const float4 *cf = reinterpret_cast<const float4 *>(e.coef[bi]);
            const float4 cc = cf[0], be = cf[1], r3 = cf[2], p0 = cf[3], p1 = cf[4], p2 = cf[5], p3 = cf[6];
            float v[BT];
#pragma unroll
            for (int a = 0; a < BT; a++) v[a] = e.v[bi * BT + a][col + par];
            // the column of this lane's parity, then the sums over the eight lanes
            float sk[BT], sq[BT];
#pragma unroll
            for (int a = 0; a < BT; a++) {
                const float k0 = sum2(ak[a][0]), k1 = sum2(ak[a][1]), q0 = sum2(aq[a][0]), q1 = sum2(aq[a][1]);
                sk[a] = (par ? k1 : k0) + __shfl_xor_sync(0xffffffffu, par ? k0 : k1, 1);
                sq[a] = (par ? q1 : q0) + __shfl_xor_sync(0xffffffffu, par ? q0 : q1, 1);
            }
#pragma unroll
            for (int o = 2; o < 8; o <<= 1)
#pragma unroll
                for (int a = 0; a < BT; a++) {
                    sk[a] += __shfl_xor_sync(0xffffffffu, sk[a], o);
                    sq[a] += __shfl_xor_sync(0xffffffffu, sq[a], o);
                }
            // pairs: p0 = kk10 kk20 kk21 kk30, p1 = kk31 kk32 qk00 qk10, p2 = qk11 qk20 qk21 qk22, p3 = qk30 qk31 qk32 qk33
            const float u0 = be.x * (v[0] - cc.x * sk[0]);
            const float u1 = be.y * (v[1] - cc.y * sk[1] - p0.x * u0);
            const float u2 = be.z * (v[2] - cc.z * sk[2] - p0.y * u0 - p0.z * u1);
            const float u3 = be.w * (v[3] - cc.w * sk[3] - p0.w * u0 - p1.x * u1 - p1.y * u2);
            const float o0 = cc.x * sq[0] + p1.z * u0;
            const float o1 = cc.y * sq[1] + p1.w * u0 + p2.x * u1;
            const float o2 = cc.z * sq[2] + p2.y * u0 + p2.z * u1 + p2.w * u2;
            const float o3 = cc.w * sq[3] + p3.x * u0 + p3.y * u1 + p3.z * u2 + p3.w * u3;
            // lane l stores token l >> 1 of its column
            const int a = l >> 1, t = t0 + bi * BT + a;
            if (t < T && c0 + col + par < s.V)
                w.o[(int64_t)(row0 + t) * s.H * s.V + (int64_t)h * s.V + c0 + col + par] = a == 0 ? o0 : (a == 1 ? o1 : (a == 2 ? o2 : o3));
            const float mine[BT] = {r3.x * u0, r3.y * u1, r3.z * u2, r3.w * u3};
            f32x2 uw[BT][2];
#pragma unroll
            for (int b = 0; b < BT; b++) {
                const float other = __shfl_xor_sync(0xffffffffu, mine[b], 1);
                const float x0 = par ? other : mine[b], x1 = par ? mine[b] : other;
                uw[b][0] = pack2(x0, x0);
                uw[b][1] = pack2(x1, x1);
            }
            const f32x2 dec = pack2(cc.w, cc.w);
#pragma unroll
            for (int i = 0; i < NI; i++) {
#pragma unroll
                for (int c = 0; c < 2; c++) {
                    S[c][i][0] = mul2(dec, S[c][i][0]);
                    S[c][i][1] = mul2(dec, S[c][i][1]);
                }
#pragma unroll
                for (int b = 0; b < BT; b++) {
                    const Quad k = *reinterpret_cast<const Quad *>(&kt[b][l * 4 + 32 * i]);
#pragma unroll
                    for (int c = 0; c < 2; c++) {
                        S[c][i][0] = fma2(k.lo, uw[b][c], S[c][i][0]);
                        S[c][i][1] = fma2(k.hi, uw[b][c], S[c][i][1]);
                    }
                }
            }
        }
        __syncthreads();
    }
    pg_cp_wait<0>();
#pragma unroll
    for (int c = 0; c < 2; c++) {
        if (c0 + col + c >= s.V) continue;
#pragma unroll
        for (int i = 0; i < NI; i++)
#pragma unroll
            for (int j = 0; j < 2; j++) {
                const int r = l * 4 + 32 * i + 2 * j;
                float lo, hi;
                asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(S[c][i][j]));
                if (r < s.D) st[(int64_t)r * s.vs + c] = lo;
                if (r + 1 < s.D) st[(int64_t)(r + 1) * s.vs + c] = hi;
            }
    }
}

template <int NI>
int32_t run_scan(pg_ctx *ctx, const DeltaShape &s, const pg_batch *bt, const DeltaWork &w, float *state)
{
    constexpr int smem = ScanTile<NI>::STAGES * (int)sizeof(typename ScanTile<NI>::Stage);
    static std::atomic<uint64_t> set{0};
    PG_CUDA(pg_max_smem_once(delta_scan_kernel<NI>, smem, ctx->device, set));
    return launch_whole(ctx, delta_scan_kernel<NI>, dim3((unsigned)((s.V + 31) / 32), (unsigned)s.H, (unsigned)bt->seqs), dim3(128), (size_t)smem, s, *bt, w, state);
}

template <int TAPS, int V>
int32_t run_prep_v(pg_ctx *ctx, const DeltaShape &s, const pg_batch *bt, const float *proj, int64_t ldp, const float *ring, const DeltaWork &w)
{
    const size_t smem = ((size_t)BT * 2 * s.G * s.D + 16 * s.G) * 4;
    PG_REQUIRE(smem <= 220 * 1024, "delta: too many query / key channels");
    static std::atomic<uint64_t> set{0};
    PG_CUDA(pg_max_smem_once(delta_prep_kernel<TAPS, V>, 220 * 1024, ctx->device, set));
    return launch_pdl(ctx, delta_prep_kernel<TAPS, V>, dim3((unsigned)((bt->max_len + BT - 1) / BT), (unsigned)bt->seqs), dim3(256), smem, s, *bt, proj, ldp, ring, w);
}

template <int TAPS>
int32_t run_prep(pg_ctx *ctx, const DeltaShape &s, const pg_batch *bt, const float *proj, int64_t ldp, const float *ring, const DeltaWork &w)
{
    const bool vec = ((2 * s.G * s.D) & 3) == 0 && ((s.H * s.V) & 3) == 0 && ldp % 4 == 0 &&
                     (((uintptr_t)proj | (uintptr_t)ring | (uintptr_t)s.conv | (uintptr_t)w.v) & 15) == 0;
    return vec ? run_prep_v<TAPS, 4>(ctx, s, bt, proj, ldp, ring, w) : run_prep_v<TAPS, 1>(ctx, s, bt, proj, ldp, ring, w);
}

// a CTA per token: o / rms(o) * norm * silu(gate) per head; the sequence's last taps - 1 tokens also store their
// convolution inputs (everything that read the ring has run)
template <typename TA>
__global__ void __launch_bounds__(256)
    delta_out_kernel(const DeltaShape s, const pg_batch bt, const float *__restrict__ proj, int64_t ldp, const DeltaWork w, float *ring, TA *__restrict__ out,
                     int64_t ldo, bool vec)
{
    pg_pdl_begin();
    const int m = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const float *row = proj + (int64_t)m * ldp;
    if (vec) {                                            // V a multiple of 4, at most 128: a quad per lane
        for (int h0 = warp; h0 < s.H; h0 += 16) {         // two heads at a time
            float4 o[2], gt[2];
#pragma unroll
            for (int i = 0; i < 2; i++) {
                const int h = h0 + 8 * i;
                o[i] = gt[i] = make_float4(0.f, 0.f, 0.f, 0.f);
                if (h < s.H && lane * 4 < s.V) {
                    o[i] = __ldcg(reinterpret_cast<const float4 *>(w.o + ((int64_t)m * s.H + h) * s.V) + lane);
                    gt[i] = __ldcg(reinterpret_cast<const float4 *>(row + s.C + (int64_t)h * s.V) + lane);
                }
            }
#pragma unroll
            for (int i = 0; i < 2; i++) {
                const int h = h0 + 8 * i;
                const float ss = pg_warp_sum(o[i].x * o[i].x + o[i].y * o[i].y + o[i].z * o[i].z + o[i].w * o[i].w);
                const float inv = __fdiv_rn(1.0f, sqrtf(__fdiv_rn(ss, (float)s.V) + s.eps));
                if (h < s.H && lane * 4 < s.V) {
                    const float4 nw = __ldg(reinterpret_cast<const float4 *>(s.norm) + lane);
                    TA *dst = out + (int64_t)m * ldo + (int64_t)h * s.V + lane * 4;
                    const float y[4] = {o[i].x * inv * nw.x * pg_silu(gt[i].x), o[i].y * inv * nw.y * pg_silu(gt[i].y),
                                        o[i].z * inv * nw.z * pg_silu(gt[i].z), o[i].w * inv * nw.w * pg_silu(gt[i].w)};
                    if constexpr (sizeof(TA) == 2)
                        *reinterpret_cast<uint2 *>(dst) = make_uint2(pg_pack_bf16(y[0], y[1]), pg_pack_bf16(y[2], y[3]));
                    else
                        *reinterpret_cast<float4 *>(dst) = make_float4(y[0], y[1], y[2], y[3]);
                }
            }
        }
    } else {
        for (int h = warp; h < s.H; h += 8) {
            const float *o = w.o + (int64_t)m * s.H * s.V + (int64_t)h * s.V;
            float ss = 0.0f;
            for (int c = lane; c < s.V; c += 32) {
                const float x = __ldcg(o + c);
                ss += x * x;
            }
            ss = pg_warp_sum(ss);
            const float inv = __fdiv_rn(1.0f, sqrtf(__fdiv_rn(ss, (float)s.V) + s.eps));
            for (int c = lane; c < s.V; c += 32)
                pg_put(out + (int64_t)m * ldo + (int64_t)h * s.V + c, __ldcg(o + c) * inv * __ldg(s.norm + c) * pg_silu(__ldcg(row + s.C + (int64_t)h * s.V + c)));
        }
    }
    const int seq = __ldcg(bt.d_row_seq + m);
    if (m >= __ldcg(bt.d_seq_row0 + seq + 1) - (s.taps - 1)) {
        float *rg = ring + ((int64_t)__ldcg(bt.d_seq_slot + seq) * s.taps + __ldcg(bt.d_pos + m) % s.taps) * s.C;
        for (int c = threadIdx.x; c < s.C; c += 256) rg[c] = __ldcg(row + c);
    }
}

DeltaShape shape_of(const pg_delta *p)
{
    DeltaShape s;
    s.H = p->heads, s.G = p->kv_heads, s.D = p->dim, s.V = p->vdim, s.taps = p->taps;
    s.C = 2 * s.G * s.D + s.H * s.V;
    s.vs = (s.V + 3) & ~3;
    s.eps = p->eps, s.unit_eps = p->unit_eps;
    s.qscale = 1.0f / sqrtf((float)s.D);
    s.conv = p->d_conv, s.a_log = p->d_a_log, s.dt_bias = p->d_dt_bias, s.norm = p->d_norm;
    return s;
}

}  // namespace

extern "C" {

PG_API int64_t pg_delta_work_floats(const pg_delta *p, int64_t max_rows)
{
    if (!p || max_rows < 0) return 0;
    const int64_t G = p->kv_heads, H = p->heads, D = p->dim, V = p->vdim;
    // (a block of four tokens per sequence may be a single token)
    return max_rows * (2 * G * D + 2 * H * V) + (max_rows + 8) * H * 32 + 64;
}

PG_API int32_t pg_delta_run(pg_ctx *ctx, const pg_delta *p, const pg_batch *batch, const float *d_proj, int64_t ldp, float *d_ring, float *d_state,
                            void *d_out, int32_t dtype, int64_t ldo)
{
    PG_ENTER(ctx);
    PG_REQUIRE(p && batch && d_proj && d_ring && d_state && d_out && p->d_work, "delta: null pointer");
    PG_REQUIRE(p->heads > 0 && p->kv_heads > 0 && p->heads % p->kv_heads == 0 && p->dim > 0 && p->dim <= 256 && p->vdim > 0 && p->vdim <= 1024 && p->taps >= 1,
               "delta: bad shape (heads %d / %d, dim %d <= 256, vdim %d <= 1024, taps %d)", p->heads, p->kv_heads, p->dim, p->vdim, p->taps);
    const DeltaShape s = shape_of(p);
    PG_REQUIRE(ldp >= s.C + (int64_t)s.H * s.V + 2 * s.H && ldo >= (int64_t)s.H * s.V, "delta: rows too short");
    const int M = batch->rows;
    if (M == 0) return PG_OK;
    if (batch->max_len == 1) {
        const int cpt = s.vs / 4 < DS_T ? s.vs / 4 : DS_T, groups = DS_T / cpt;
        const size_t smem = (size_t)(2 * ((s.D + 3) & ~3) + 2 * s.vs + 2 * groups * s.vs) * 4;
        PG_REQUIRE(smem <= 48 * 1024, "delta: shared memory");
        const dim3 g((unsigned)s.H, (unsigned)M);
#define PG_DS_CASE(N)                                                                                                                                   \
    return dtype == PG_BF16 ? launch_pdl(ctx, delta_step_kernel<N, bf16>, g, dim3(DS_T), smem, s, d_proj, ldp, batch->d_pos, batch->d_seq_slot, d_ring, \
                                         d_state, (bf16 *)d_out, ldo)                                                                                   \
                            : launch_pdl(ctx, delta_step_kernel<N, float>, g, dim3(DS_T), smem, s, d_proj, ldp, batch->d_pos, batch->d_seq_slot, d_ring, \
                                         d_state, (float *)d_out, ldo)
        if (s.taps == 2) PG_DS_CASE(2);
        if (s.taps == 3) PG_DS_CASE(3);
        if (s.taps == 4) PG_DS_CASE(4);
        PG_DS_CASE(0);
#undef PG_DS_CASE
    }
    DeltaWork w;
    float *at = p->d_work;
    w.q = at, at += pg_up((int64_t)M * s.G * s.D, 4);
    w.k = at, at += pg_up((int64_t)M * s.G * s.D, 4);
    w.v = at, at += pg_up((int64_t)M * s.H * s.V, 4);
    w.o = at, at += pg_up((int64_t)M * s.H * s.V, 4);
    w.coef = at;
    int32_t rc;
    if (s.taps == 2)
        rc = run_prep<2>(ctx, s, batch, d_proj, ldp, d_ring, w);
    else if (s.taps == 3)
        rc = run_prep<3>(ctx, s, batch, d_proj, ldp, d_ring, w);
    else if (s.taps == 4)
        rc = run_prep<4>(ctx, s, batch, d_proj, ldp, d_ring, w);
    else
        rc = run_prep<0>(ctx, s, batch, d_proj, ldp, d_ring, w);
    if (rc != PG_OK) return rc;
    if (s.D <= 32)
        rc = run_scan<1>(ctx, s, batch, w, d_state);
    else if (s.D <= 64)
        rc = run_scan<2>(ctx, s, batch, w, d_state);
    else if (s.D <= 96)
        rc = run_scan<3>(ctx, s, batch, w, d_state);
    else if (s.D <= 128)
        rc = run_scan<4>(ctx, s, batch, w, d_state);
    else if (s.D <= 192)
        rc = run_scan<6>(ctx, s, batch, w, d_state);
    else
        rc = run_scan<8>(ctx, s, batch, w, d_state);
    if (rc != PG_OK) return rc;
    const bool vec = s.V % 4 == 0 && s.V <= 128 && s.C % 4 == 0 && ldp % 4 == 0 && ldo % 4 == 0 &&
                     (((uintptr_t)d_proj | (uintptr_t)d_out | (uintptr_t)s.norm | (uintptr_t)w.o) & 15) == 0;
    if (dtype == PG_BF16)
        return launch_pdl(ctx, delta_out_kernel<bf16>, dim3((unsigned)M), dim3(256), 0, s, *batch, d_proj, ldp, w, d_ring, (bf16 *)d_out, ldo, vec);
    return launch_pdl(ctx, delta_out_kernel<float>, dim3((unsigned)M), dim3(256), 0, s, *batch, d_proj, ldp, w, d_ring, (float *)d_out, ldo, vec);
}

}  // extern "C"
