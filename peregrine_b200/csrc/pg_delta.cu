// Gated delta rule with short causal convolutions.
//
// Per token and head (S: dim x vdim, f32):  S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q.
// Both read-outs can be taken from the S the token finds:  S^T k and S^T q of the old state give
//   u = beta (v - g S^T k),   o = g S^T q + (k . q) u,
// so a token needs one pass of reductions over the state before the update.
//
//   one token per sequence   delta_step_kernel: convolution, unit norms, gates, the state update and the gated output
//                            norm of one (head, sequence) in one CTA; the state is read and written once
//   longer portions          delta_prep_kernel (convolution, unit norms, gates; a CTA per token), delta_scan_kernel (the
//                            recurrence; a warp holds four columns of a head's state in registers), delta_out_kernel
//                            (output norm and gate; also stores the convolution inputs that the next portion needs)
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

template <typename TA>
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

    // the state's rows are asked for first
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
    for (int i = tid; i < 2 * s.D + s.V; i += DS_T) {
        const int c = i < s.D ? cq + i : (i < 2 * s.D ? ck + i - s.D : cvv + i - 2 * s.D);
        const float y = conv_at(s, row, ldp, rg, c, 0, pos);
        if (i < s.D)
            sq[i] = y;
        else if (i < 2 * s.D)
            sk[i - s.D] = y;
        else
            sv[i - 2 * s.D] = y;
        // the entry this position takes is older than anything a convolution still reads
        if (i >= 2 * s.D || h % rep == 0) rg[(int64_t)(pos % s.taps) * s.C + c] = __ldcg(row + c);
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
        const float *tail = row + s.C + (int64_t)s.H * s.V;
        bc[0] = pg_sigmoid(__ldcg(tail + h));
        bc[1] = expf(log_decay(__ldcg(tail + s.H + h), __ldg(s.a_log + h), __ldg(s.dt_bias + h)));
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
    const float *gate = row + s.C + (int64_t)h * s.V;
    for (int c = tid; c < s.V; c += DS_T)
        pg_put(out + (int64_t)b * ldo + (int64_t)h * s.V + c, so[c] * inv * __ldg(s.norm + c) * pg_silu(__ldcg(gate + c)));
}

// ---- longer portions ---------------------------------------------------------------------------------------------
// work rows: q [G D] | k [G D] | v [H V] | o [H V], and per token: kq [G] | beta [H] | decay [H]
struct DeltaWork {
    float *q, *k, *v, *o, *kq, *beta, *dec;
};

__global__ void __launch_bounds__(256)
    delta_prep_kernel(const DeltaShape s, const pg_batch bt, const float *__restrict__ proj, int64_t ldp, const float *__restrict__ ring, const DeltaWork w)
{
    extern __shared__ __align__(16) float sm[];   // q and k channels
    pg_pdl_begin();
    const int m = blockIdx.x, seq = __ldcg(bt.d_row_seq + m);
    const int pos = __ldcg(bt.d_pos + m), t = m - __ldcg(bt.d_seq_row0 + seq);
    const float *row = proj + (int64_t)m * ldp;
    const float *rg = ring + (int64_t)__ldcg(bt.d_seq_slot + seq) * s.taps * s.C;
    const int qk = 2 * s.G * s.D;
    for (int c = threadIdx.x; c < s.C; c += 256) {
        const float y = conv_at(s, row, ldp, rg, c, t, pos);
        if (c < qk)
            sm[c] = y;
        else
            w.v[(int64_t)m * s.H * s.V + c - qk] = y;
    }
    __syncthreads();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    for (int g = warp; g < s.G; g += 8) {
        const float *q = sm + g * s.D, *k = sm + (s.G + g) * s.D;
        float a = 0.0f, b = 0.0f, d = 0.0f;
        for (int i = lane; i < s.D; i += 32) {
            a += q[i] * q[i];
            b += k[i] * k[i];
            d += q[i] * k[i];
        }
        a = pg_warp_sum(a);
        b = pg_warp_sum(b);
        d = pg_warp_sum(d);
        const float iq = __fdiv_rn(s.qscale, sqrtf(a + s.unit_eps)), ik = __fdiv_rn(1.0f, sqrtf(b + s.unit_eps));
        for (int i = lane; i < s.D; i += 32) {
            w.q[((int64_t)m * s.G + g) * s.D + i] = q[i] * iq;
            w.k[((int64_t)m * s.G + g) * s.D + i] = k[i] * ik;
        }
        if (lane == 0) w.kq[(int64_t)m * s.G + g] = d * iq * ik;
    }
    const float *tail = row + s.C + (int64_t)s.H * s.V;
    for (int h = threadIdx.x; h < s.H; h += 256) {
        w.beta[(int64_t)m * s.H + h] = pg_sigmoid(__ldcg(tail + h));
        w.dec[(int64_t)m * s.H + h] = expf(log_decay(__ldcg(tail + s.H + h), __ldg(s.a_log + h), __ldg(s.dt_bias + h)));
    }
}

// grid (ceil(V / 32), H, seqs), 8 warps.  Warp w: columns w * 4 .. w * 4 + 3 of the CTA's 32; of its lanes, eight share a
// column: lane l = lane & 7 holds rows l * 4 + 32 i .. + 3 (i < NI) of column lane >> 3.
template <int NI>
__global__ void __launch_bounds__(256)
    delta_scan_kernel(const DeltaShape s, const pg_batch bt, const DeltaWork w, float *state)
{
    constexpr int DP = NI * 32;
    constexpr int SC_TB = NI <= 4 ? 16 : 8;      // tokens per shared-memory tile
    __shared__ __align__(16) float tk[2][SC_TB][DP], tq[2][SC_TB][DP];
    __shared__ __align__(16) float tv[2][SC_TB][32];
    __shared__ float ts[2][SC_TB][4];            // kq, beta, decay
    pg_pdl_begin();
    const int h = blockIdx.y, seq = blockIdx.z, g = h / (s.H / s.G), tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int row0 = __ldcg(bt.d_seq_row0 + seq), T = __ldcg(bt.d_seq_row0 + seq + 1) - row0;
    if (T <= 0) return;
    const int pos0 = __ldcg(bt.d_pos + row0);
    const int c0 = blockIdx.x * 32, mycol = warp * 4 + (lane >> 3), l = lane & 7;
    const bool col_ok = c0 + mycol < s.V;
    float *st = state + ((int64_t)__ldcg(bt.d_seq_slot + seq) * s.H + h) * (int64_t)s.D * s.vs + c0 + mycol;
    float S[NI][4];
#pragma unroll
    for (int i = 0; i < NI; i++)
#pragma unroll
        for (int j = 0; j < 4; j++) {
            const int r = l * 4 + 32 * i + j;
            S[i][j] = (pos0 > 0 && col_ok && r < s.D) ? __ldcg(st + (int64_t)r * s.vs) : 0.0f;
        }
    // a tile into shared memory; rows of q and k behind D and columns behind V are zero
    auto fetch = [&](int buf, int t0) {
        const int n = min(SC_TB, T - t0);
        // (16-byte copies that bypass L1 where the shape allows them)
        const bool vec = ((s.D | s.V) & 3) == 0;
        for (int i = tid; i < SC_TB * DP / 4; i += 256) {
            const int t = i / (DP / 4), d = (i - t * (DP / 4)) * 4;
            const int64_t at = ((int64_t)(row0 + t0 + t) * s.G + g) * s.D + d;
            if (vec && t < n && d < s.D) {
                pg_cp16(pg_smem(&tk[buf][t][d]), w.k + at);
                pg_cp16(pg_smem(&tq[buf][t][d]), w.q + at);
            } else {
#pragma unroll
                for (int j = 0; j < 4; j++) {
                    const bool in = t < n && d + j < s.D;
                    tk[buf][t][d + j] = in ? __ldcg(w.k + at + j) : 0.0f;
                    tq[buf][t][d + j] = in ? __ldcg(w.q + at + j) : 0.0f;
                }
            }
        }
        for (int i = tid; i < SC_TB * 8; i += 256) {
            const int t = i / 8, c = (i & 7) * 4;
            const float *v = w.v + (int64_t)(row0 + t0 + t) * s.H * s.V + (int64_t)h * s.V + c0 + c;
            if (vec && t < n && c0 + c < s.V) {
                pg_cp16(pg_smem(&tv[buf][t][c]), v);
            } else {
#pragma unroll
                for (int j = 0; j < 4; j++) tv[buf][t][c + j] = (t < n && c0 + c + j < s.V) ? __ldcg(v + j) : 0.0f;
            }
        }
        if (tid < n) {
            const int64_t m = row0 + t0 + tid;
            ts[buf][tid][0] = __ldcg(w.kq + m * s.G + g);
            ts[buf][tid][1] = __ldcg(w.beta + m * s.H + h);
            ts[buf][tid][2] = __ldcg(w.dec + m * s.H + h);
        }
        pg_cp_commit();
    };
    fetch(0, 0);
    int buf = 0;
    for (int t0 = 0; t0 < T; t0 += SC_TB, buf ^= 1) {
        const int n = min(SC_TB, T - t0);
        if (t0 + SC_TB < T) {
            fetch(buf ^ 1, t0 + SC_TB);
            pg_cp_wait<1>();
        } else {
            pg_cp_wait<0>();
        }
        __syncthreads();
        float4 k[NI], q[NI];
#pragma unroll
        for (int i = 0; i < NI; i++) {
            k[i] = *reinterpret_cast<const float4 *>(&tk[buf][0][l * 4 + 32 * i]);
            q[i] = *reinterpret_cast<const float4 *>(&tq[buf][0][l * 4 + 32 * i]);
        }
        for (int t = 0; t < n; t++) {
            // the next token's rows are asked for before this one's chain of dependent steps
            float4 kn[NI], qn[NI];
            const int tn = min(t + 1, SC_TB - 1);
#pragma unroll
            for (int i = 0; i < NI; i++) {
                kn[i] = *reinterpret_cast<const float4 *>(&tk[buf][tn][l * 4 + 32 * i]);
                qn[i] = *reinterpret_cast<const float4 *>(&tq[buf][tn][l * 4 + 32 * i]);
            }
            const float kq = ts[buf][t][0], beta = ts[buf][t][1], dec = ts[buf][t][2], v = tv[buf][t][mycol];
            float a[4] = {0.f, 0.f, 0.f, 0.f}, b[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
            for (int i = 0; i < NI; i++) {
                a[0] = fmaf(k[i].x, S[i][0], a[0]), a[1] = fmaf(k[i].y, S[i][1], a[1]), a[2] = fmaf(k[i].z, S[i][2], a[2]), a[3] = fmaf(k[i].w, S[i][3], a[3]);
                b[0] = fmaf(q[i].x, S[i][0], b[0]), b[1] = fmaf(q[i].y, S[i][1], b[1]), b[2] = fmaf(q[i].z, S[i][2], b[2]), b[3] = fmaf(q[i].w, S[i][3], b[3]);
            }
            float sk = (a[0] + a[1]) + (a[2] + a[3]), sq = (b[0] + b[1]) + (b[2] + b[3]);
#pragma unroll
            for (int o = 1; o < 8; o <<= 1) {
                sk += __shfl_xor_sync(0xffffffffu, sk, o);
                sq += __shfl_xor_sync(0xffffffffu, sq, o);
            }
            const float u = beta * (v - dec * sk);
#pragma unroll
            for (int i = 0; i < NI; i++) {
                S[i][0] = fmaf(k[i].x, u, dec * S[i][0]);
                S[i][1] = fmaf(k[i].y, u, dec * S[i][1]);
                S[i][2] = fmaf(k[i].z, u, dec * S[i][2]);
                S[i][3] = fmaf(k[i].w, u, dec * S[i][3]);
            }
            if (l == 0 && col_ok) w.o[(int64_t)(row0 + t0 + t) * s.H * s.V + (int64_t)h * s.V + c0 + mycol] = dec * sq + kq * u;
#pragma unroll
            for (int i = 0; i < NI; i++) {
                k[i] = kn[i];
                q[i] = qn[i];
            }
        }
        __syncthreads();
    }
    if (col_ok) {
#pragma unroll
        for (int i = 0; i < NI; i++)
#pragma unroll
            for (int j = 0; j < 4; j++) {
                const int r = l * 4 + 32 * i + j;
                if (r < s.D) st[(int64_t)r * s.vs] = S[i][j];
            }
    }
}

// a CTA per token: o / rms(o) * norm * silu(gate) per head; the sequence's last taps - 1 tokens also store their
// convolution inputs (everything that read the ring has run)
template <typename TA>
__global__ void __launch_bounds__(256)
    delta_out_kernel(const DeltaShape s, const pg_batch bt, const float *__restrict__ proj, int64_t ldp, const DeltaWork w, float *ring, TA *__restrict__ out,
                     int64_t ldo)
{
    pg_pdl_begin();
    const int m = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const float *row = proj + (int64_t)m * ldp;
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
    return max_rows * (2 * G * D + 2 * H * V + G + 2 * H) + 32;
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
        if (dtype == PG_BF16)
            return launch_pdl(ctx, delta_step_kernel<bf16>, g, dim3(DS_T), smem, s, d_proj, ldp, batch->d_pos, batch->d_seq_slot, d_ring, d_state, (bf16 *)d_out, ldo);
        return launch_pdl(ctx, delta_step_kernel<float>, g, dim3(DS_T), smem, s, d_proj, ldp, batch->d_pos, batch->d_seq_slot, d_ring, d_state, (float *)d_out, ldo);
    }
    DeltaWork w;
    float *at = p->d_work;
    w.q = at, at += pg_up((int64_t)M * s.G * s.D, 4);
    w.k = at, at += pg_up((int64_t)M * s.G * s.D, 4);
    w.v = at, at += pg_up((int64_t)M * s.H * s.V, 4);
    w.o = at, at += pg_up((int64_t)M * s.H * s.V, 4);
    w.kq = at, at += pg_up((int64_t)M * s.G, 4);
    w.beta = at, at += pg_up((int64_t)M * s.H, 4);
    w.dec = at;
    const size_t smem = (size_t)2 * s.G * s.D * 4;
    PG_REQUIRE(smem <= 200 * 1024, "delta: too many query / key channels");
    static std::atomic<uint64_t> set{0};
    PG_CUDA(pg_max_smem_once(delta_prep_kernel, 200 * 1024, ctx->device, set));
    int32_t rc = launch_pdl(ctx, delta_prep_kernel, dim3((unsigned)M), dim3(256), smem, s, *batch, d_proj, ldp, (const float *)d_ring, w);
    if (rc != PG_OK) return rc;
    const dim3 g((unsigned)((s.V + 31) / 32), (unsigned)s.H, (unsigned)batch->seqs);
    if (s.D <= 32)
        rc = launch_pdl(ctx, delta_scan_kernel<1>, g, dim3(256), 0, s, *batch, w, d_state);
    else if (s.D <= 64)
        rc = launch_pdl(ctx, delta_scan_kernel<2>, g, dim3(256), 0, s, *batch, w, d_state);
    else if (s.D <= 96)
        rc = launch_pdl(ctx, delta_scan_kernel<3>, g, dim3(256), 0, s, *batch, w, d_state);
    else if (s.D <= 128)
        rc = launch_pdl(ctx, delta_scan_kernel<4>, g, dim3(256), 0, s, *batch, w, d_state);
    else if (s.D <= 192)
        rc = launch_pdl(ctx, delta_scan_kernel<6>, g, dim3(256), 0, s, *batch, w, d_state);
    else
        rc = launch_pdl(ctx, delta_scan_kernel<8>, g, dim3(256), 0, s, *batch, w, d_state);
    if (rc != PG_OK) return rc;
    if (dtype == PG_BF16)
        return launch_pdl(ctx, delta_out_kernel<bf16>, dim3((unsigned)M), dim3(256), 0, s, *batch, d_proj, ldp, w, d_ring, (bf16 *)d_out, ldo);
    return launch_pdl(ctx, delta_out_kernel<float>, dim3((unsigned)M), dim3(256), 0, s, *batch, d_proj, ldp, w, d_ring, (float *)d_out, ldo);
}

}  // extern "C"
