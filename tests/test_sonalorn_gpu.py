"""Every mechanism of the Sonalorn layers alone, whole models, and serving, on the GPU against oracle/sonalorn_oracle.py."""
import os
import subprocess
import sys

import numpy as np
import pytest

from oracle import sonalorn_oracle as so
from tests import _sonalorn as t

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DTYPES = ["float32", "bfloat16"]


@pytest.fixture(scope="module")
def lm():
    from peregrine_b200.runtime import GpuContext

    return GpuContext(component="lm")


def rng(seed):
    return np.random.Generator(np.random.PCG64(seed))


def device(lm, dtype, rows=64):
    from peregrine_b200.layers import Device

    return Device(lm, dtype, rows)


def act(d, a, k=None):
    """[rows, cols] -> the step's type on the device, columns padded with zeros to a multiple of 64."""
    x = np.zeros((a.shape[0], (a.shape[1] + 63) // 64 * 64), np.float32)
    x[:, :a.shape[1]] = a
    out = d.torch.from_numpy(x).to(d.dev).to(d.act)
    d.torch.cuda.synchronize()
    return out


def rounded(a, dtype):
    return (a if dtype == "float32" else t.bf16_values(a)).astype(np.float64)


def close(got, want, tol, what=""):
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    assert got.shape == want.shape and np.isfinite(got).all(), what
    rms = max(1e-30, np.sqrt(np.mean(want ** 2)))
    worst, mean = np.abs(got - want).max() / rms, np.sqrt(np.mean((got - want) ** 2)) / rms
    assert mean <= tol and worst <= 10 * tol, f"{what}: rms error {mean:.3g}, largest {worst:.3g} of the rms, tolerance {tol:.3g}"


# ---- products ------------------------------------------------------------------------------------------------------
SHAPES = [(4, 64), (24, 64), (41, 192), (200, 320), (513, 576), (48, 4160), (40, 9000), (1030, 130)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,k", SHAPES)
def test_product(lm, dtype, n, k):
    from peregrine_b200.layers import Linear, up

    d = device(lm, dtype, 320)
    g = rng(n + k)
    w = t.bf16_values(g.standard_normal((n, k)) / k ** 0.5)
    lin = Linear(d, d.bf16(w))
    for m in (1, 2, 7, 8, 9, 16, 17, 64, 129, 300):
        a = g.standard_normal((m, k)).astype(np.float32)
        x = act(d, a)
        want = rounded(a, dtype) @ w.T.astype(np.float64)
        for out in (["float32", "bfloat16"] if dtype == "bfloat16" else ["float32"]):
            y = d.torch.full((m, up(n, 8)), 7.0, dtype=getattr(d.torch, out), device=d.dev)
            d.torch.cuda.synchronize()
            lin.run(x, m, y)
            lm.sync()
            got = y.float().cpu().numpy()
            # (the tensor cores' sums lose a little more over a long K)
            close(got[:, :n], want, 1e-2 if out == "bfloat16" else 2e-5 if dtype == "bfloat16" else 5e-6, f"m {m} {out}")
            assert (got[:, n:] == 7.0).all()       # nothing behind the matrix's own columns
    assert lm.device_status() == 0
    lin.free()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("f,k", [(5, 64), (72, 130), (300, 384), (24, 4500)])
def test_gated_products(lm, dtype, f, k):
    from peregrine_b200 import _lib
    from peregrine_b200.layers import Linear, up

    d = device(lm, dtype, 200)
    g = rng(f * 7 + k)
    gate, upw = (t.bf16_values(g.standard_normal((f, k)) * 2 / k ** 0.5) for _ in range(2))
    lin = Linear(d, (d.bf16(gate), d.bf16(upw)), gated=True)
    for m in (1, 9, 16, 40, 170):
        a = g.standard_normal((m, k)).astype(np.float32)
        x, ar = act(d, a), rounded(a, dtype)
        G, U = ar @ gate.T.astype(np.float64), ar @ upw.T.astype(np.float64)
        for code, limit, want in ((_lib.ACT_GELU_TANH_GLU, 0.0, so.gelu_tanh(G) * U),
                                  (_lib.ACT_CLAMPED_SWISH_GLU, 0.9, np.minimum(G, .9) * so.sigmoid(1.702 * np.minimum(G, .9)) * (np.clip(U, -.9, .9) + 1))):
            y = d.torch.zeros(m, up(f, 64), dtype=d.act, device=d.dev)
            d.torch.cuda.synchronize()
            lin.run(x, m, y, code, limit)
            lm.sync()
            got = y.float().cpu().numpy()
            close(got[:, :f], want, 1e-2 * 3 if dtype == "bfloat16" else 1e-5, f"m {m} act {code}")
            assert (got[:, f:] == 0.0).all()
    lin.free()


# ---- residual rows ---------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [5, 70, 256, 1030, 4096])
def test_rows(lm, dtype, width):
    from peregrine_b200.layers import Batch, up

    d = device(lm, dtype, 400)
    t_ = d.torch
    g = rng(width)
    for m in (1, 3, 40, 330):
        table, pos = t.bf16_values(g.standard_normal((20, width))), t.bf16_values(g.standard_normal((400, width)))
        w, scale, eps = g.standard_normal(width).astype(np.float32), g.standard_normal(width).astype(np.float32), 0.01
        tokens = g.integers(0, 20, m)
        b = Batch(d, [(0, 7, tokens.tolist())] if m < 300 else [(0, 0, tokens[:200].tolist()), (1, 3, tokens[200:].tolist())], [m - 1, 0])
        where = np.arange(7, 7 + m) if m < 300 else np.concatenate([np.arange(200), np.arange(3, 3 + m - 200)])
        x = t_.zeros(m, width, device=d.dev)
        h = t_.zeros(m, up(width, 64), dtype=d.act, device=d.dev)
        dt, dp, dw, ds = d.bf16(table), d.bf16(pos), d.f32(w), d.f32(scale)
        y = g.standard_normal((m, width)).astype(np.float32)
        dy = t_.zeros(m, up(width, 4), device=d.dev)
        dy[:, :width] = d.f32(y)
        picked = t_.zeros(2, up(width, 64), dtype=d.act, device=d.dev)
        t_.cuda.synchronize()
        ck, lib, gh = d.check, d.lib, lm.handle
        import ctypes as C

        ck(lib.pg_embed_norm(gh, C.byref(b.c), dt.data_ptr(), dp.data_ptr(), width, dw.data_ptr(), eps, x.data_ptr(), h.data_ptr(), d.code, h.stride(0)))
        lm.sync()
        want = so.rms_norm(table[tokens].astype(np.float64) + pos[where], w, eps)
        close(x.cpu().numpy(), want, 3e-6, "embed")
        close(h[:, :width].float().cpu().numpy(), want, 2e-2 if dtype == "bfloat16" else 3e-6, "embed h")
        ck(lib.pg_norm_add(gh, dy.data_ptr(), dy.stride(0), x.data_ptr(), dw.data_ptr(), ds.data_ptr(), m, width, eps, h.data_ptr(), d.code, h.stride(0)))
        ck(lib.pg_norm_rows(gh, x.data_ptr(), b.d_wanted, 2, width, ds.data_ptr(), eps, picked.data_ptr(), d.code, picked.stride(0)))
        lm.sync()
        want = want + so.rms_norm(y.astype(np.float64), w, eps) * scale
        close(x.cpu().numpy(), want, 5e-6, "add")
        close(picked[:, :width].float().cpu().numpy(), so.rms_norm(want[[m - 1, 0]], scale, eps), 2e-2 if dtype == "bfloat16" else 5e-6, "pick")
        assert (h[:, width:] == 0).all() and (picked[:, width:] == 0).all()


# ---- router and experts ----------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("experts,identity,top,groups", [(5, 0, 1, None), (6, 3, 2, (3, 2)), (20, 12, 5, (8, 3)), (33, 1, 34, None), (40, 24, 8, (4, 4)),
                                                         (250, 6, 8, (16, 4)), (700, 0, 3, (7, 1))])
def test_router(lm, dtype, experts, identity, top, groups):
    import ctypes as C

    d = device(lm, dtype)
    n = experts + identity
    g = rng(n * 3 + top)
    h = C.c_void_p()
    d.check(d.lib.pg_route_create(lm.handle, 300, experts, identity, top, C.byref(h)))
    corr = (g.standard_normal(n) * 0.5).astype(np.float32)      # most choice scores are negative or far from the scores
    dc = d.f32(corr)
    for m in (1, 3, 16, 17, 300):
        z = (g.standard_normal((m, n)) * 3).astype(np.float32)
        dz = d.torch.zeros(m, n + 3, device=d.dev)
        dz[:, :n] = d.f32(z)
        d.torch.cuda.synchronize()
        d.check(d.lib.pg_route_run(lm.handle, h, d.code, dz.data_ptr(), n + 3, m, dc.data_ptr(), groups[0] if groups else 1, groups[1] if groups else 1))
        ids, w = np.zeros((m, top), np.int32), np.zeros((m, top), np.float32)
        d.check(d.lib.pg_route_read(lm.handle, h, ids.ctypes.data, w.ctypes.data))
        for i in range(m):
            idx, want = so.route(z[i].astype(np.float64), corr.astype(np.float64), top, {"count": groups[0], "keep": groups[1]} if groups else None)
            assert ids[i].tolist() == idx.tolist()
            assert np.allclose(w[i], want, rtol=1e-5, atol=1e-9)
    d.lib.pg_route_free(lm.handle, h)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,mlp", [(96, t.moe(24, 0.8, 6, 3, 2, (3, 2))), (70, t.moe(17, 2.5, 5, 0, 3)), (320, t.moe(136, 1.1, 12, 12, 6, (6, 2))),
                                       (64, t.moe(8, 0.5, 1, 1, 2))])
def test_experts(lm, dtype, width, mlp):
    from peregrine_b200.layers import Batch, MoeFF

    d = device(lm, dtype, 290)
    g = rng(width)
    W = {k: t.bf16_values(v) for k, v in t.mlp_weights(g, mlp, width).items()}
    ff = MoeFF(d, mlp, W, width)
    got = {}
    for m in (1, 5, 16, 17, 290):
        x = t.bf16_values(g.standard_normal((m, width)))
        b = Batch(d, [(0, 0, [0] * m)])
        dx, dw, ds = d.f32(x), d.f32(np.ones(width, np.float32)), d.f32(np.ones(width, np.float32))
        h = act(d, x)
        hh = h.clone()
        d.torch.cuda.synchronize()

        def add(out, route=None):
            d.check(d.lib.pg_routed_norm_add(lm.handle, route, out.data_ptr(), out.stride(0), dx.data_ptr(), dw.data_ptr(), ds.data_ptr(), m, width, 1e-5,
                                             hh.data_ptr(), d.code, hh.stride(0)))
        ff.run(b, h, None, add)
        lm.sync()
        want = x + so.rms_norm(so.moe_ff(x.astype(np.float64), {k: v.astype(np.float64) for k, v in W.items()}, mlp), 1.0, 1e-5)
        close(dx.cpu().numpy(), want, 1e-5 if dtype == "float32" else 5e-2, f"m {m}")
        got[m] = dx.cpu().numpy()
        ids, w = ff.chosen(m)
        assert ids.shape == (m, mlp["router"]["top"]) and (w >= 0).all()
    assert lm.device_status() == 0
    ff.free()


# ---- gated delta rule ------------------------------------------------------------------------------------------------
DELTAS = [t.delta(4, 2, 24, 40, 4), t.delta(2, 2, 128, 128, 2), t.delta(4, 1, 17, 5, 1), t.delta(2, 1, 160, 300, 5), t.delta(6, 3, 64, 36, 3),
          t.delta(3, 1, 256, 16, 2), t.delta(2, 1, 96, 100, 3)]


def run_mixer(lm, d, mixer, width, x, cuts, slot=1, between=None):
    """x [T, width] in portions -> [T, width] outputs; `between` is called before every portion."""
    from peregrine_b200.layers import Batch, up
    from peregrine_b200.state import SlotPool

    state = between[1] if between else mixer.new_state(SlotPool(3, 512, d.dev))
    y = d.torch.zeros(d.rows, up(width, 4), device=d.dev)
    out, at = [], 0
    for n in cuts:
        b = Batch(d, [(slot, at, [0] * n)])
        h = act(d, x[at:at + n])
        mixer.run(b, h, state, y)
        lm.sync()
        out.append(y[:n, :width].cpu().numpy())
        at += n
    assert at == len(x) and lm.device_status() == 0
    return np.concatenate(out), state


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("p", DELTAS)
def test_delta(lm, dtype, p):
    from peregrine_b200.layers import GatedDelta

    width, T = 80, 45
    d = device(lm, dtype)
    g = rng(p["dim"])
    W = {k: t.bf16_values(v) for k, v in t.mixer_weights(g, "delta", p, width).items()}
    mixer = GatedDelta(d, p, W, width, 1e-4)
    x = t.bf16_values(g.standard_normal((T, width)))
    W64 = {k: v.astype(np.float64) for k, v in W.items()}
    want, carried = so.delta_mixer(x.astype(np.float64), W64, p, 1e-4, so.delta_start(p))
    for cuts in ([45], [1] * 45, [2, 1, 3, 1, 1, 17, 16, 2, 2]):
        got, state = run_mixer(lm, d, mixer, width, x, cuts)
        close(got, want, 1e-4 if dtype == "float32" else 6e-2, f"cuts {cuts}")
        S = state["state"][1].cpu().numpy()
        close(S[:, :, :p["vdim"]], carried["S"], 1e-4 if dtype == "float32" else 6e-2, "state")
        assert (S[:, :, p["vdim"]:] == 0).all() and (state["state"][0] == 0).all() and (state["state"][2] == 0).all()
    mixer.free()


def test_delta_state_is_f32_over_a_long_sequence(lm):
    """Slow decay and small writes: a state kept in 16 bits, or a decay rounded to them, is far off after 600 tokens."""
    from peregrine_b200.layers import GatedDelta

    p, width, T = t.delta(2, 1, 32, 16, 3), 64, 500
    g = rng(77)
    W = {k: t.bf16_values(v) for k, v in t.mixer_weights(g, "delta", p, width).items()}
    W["A_log"], W["dt_bias"] = t.bf16_values(np.full(2, -5.0)), t.bf16_values(np.full(2, -2.0))
    W["b"] = t.bf16_values(W["b"] * 0.1)
    x = t.bf16_values(g.standard_normal((T, width)))
    want, carried = so.delta_mixer(x.astype(np.float64), {k: v.astype(np.float64) for k, v in W.items()}, p, 1e-4, so.delta_start(p))
    for dtype in DTYPES:
        d = device(lm, dtype, 512)
        mixer = GatedDelta(d, p, W, width, 1e-4)
        for cuts in ([T], [300] + [1] * (T - 300)):
            got, state = run_mixer(lm, d, mixer, width, x, cuts)
            close(state["state"][1].cpu().numpy(), carried["S"], 1e-4 if dtype == "float32" else 1e-2, dtype)
        mixer.free()


# ---- attention ---------------------------------------------------------------------------------------------------------
ATTENTIONS = [t.attention(6, 2, 40, 24, 0.3, (0.7, 16)), t.attention(8, 1, 64, 64, 0.2), t.attention(2, 2, 128, 128, 0.1, (1.5, 1)),
              t.attention(34, 2, 16, 80, 0.4, (0.2, 9)), t.attention(4, 4, 200, 256, 0.08), t.attention(3, 1, 5, 7, 1.0, (0.9, 33)),
              t.attention(8, 2, 64, 128, 0.15, (0.3, 40)), t.attention(4, 1, 128, 64, 0.12), t.attention(6, 2, 128, 128, 0.1)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("p", ATTENTIONS)
def test_attention(lm, dtype, p):
    from peregrine_b200.layers import Attention

    width, T = 80, 150
    d = device(lm, dtype, 160)
    g = rng(p["dim"])
    W = {k: t.bf16_values(v) for k, v in t.mixer_weights(g, "attention", p, width).items()}
    mixer = Attention(d, p, W, width, 1e-4, 200, 3)
    x = t.bf16_values(g.standard_normal((T, width)))
    want, _ = so.attention_mixer(x.astype(np.float64), {k: v.astype(np.float64) for k, v in W.items()}, p, 1e-4, so.attention_start(p), 0)
    for cuts in ([T], [1] * 20 + [2, 60, 3, 64] + [1], [70] + [1] * 70 + [2, 8]):
        got, _state = run_mixer(lm, d, mixer, width, x, cuts)
        close(got, want, 3e-5 if dtype == "float32" else 6e-2, f"cuts {cuts[:4]}")
    mixer.free()


def planted(p, width, T, far, at):
    """An input and weights with which the query of position `at` picks the key of position `far` out of all others."""
    g = rng(T + far)
    W = {k: t.bf16_values(v) for k, v in t.mixer_weights(g, "attention", p, width).items()}
    x = (g.standard_normal((T, width)) * 0.2).astype(np.float32)
    x[:, -2:] = 0.0
    x[at, -2] = 40.0                      # only this query ...
    x[far, -1] = 40.0                     # ... and only this key lie along one direction of every head
    for name, col in (("q", -2), ("k", -1)):
        W[name][:, -2:] = 0.0
        W[name].reshape(-1, p["dim"], width)[:, 0, col] = 4.0
    W["v"][:, -2] = 0.0
    W["q.norm"][:], W["k.norm"][:] = 1.0, 1.0
    return t.bf16_values(x), W


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads", [(4, 2, 32, 32, 0.5), (4, 2, 64, 64, 0.25), (8, 1, 128, 128, 0.13)])
@pytest.mark.parametrize("far", [0, 1, 63, 64, 65, 127, 128, 300, 440, 447])
def test_attention_far_key(lm, dtype, far, heads):
    """One key among hundreds carries the answer: at tile and slice borders, at the start, just in front of the query."""
    from peregrine_b200.layers import Attention

    p, width, T = t.attention(*heads, (0.5, 100)), 64, 448
    d = device(lm, dtype, T)
    x, W = planted(p, width, T, far, T - 1)
    W64 = {k: v.astype(np.float64) for k, v in W.items()}
    want, _ = so.attention_mixer(x.astype(np.float64), W64, p, 1e-4, so.attention_start(p), 0)
    x2 = x.copy()
    x2[far, -1] = 0.0
    without, _ = so.attention_mixer(x2.astype(np.float64), W64, p, 1e-4, so.attention_start(p), 0)
    if far != T - 1:
        assert np.abs(want[-1] - without[-1]).max() > 0.5 * np.sqrt(np.mean(want[-1] ** 2))     # the key matters
    mixer = Attention(d, p, W, width, 1e-4, 500, 3)
    for cuts in ([T], [T - 1, 1], [100, 2, 3, T - 108, 2, 1]):
        got, _ = run_mixer(lm, d, mixer, width, x, cuts)
        close(got[-1], want[-1], 3e-5 if dtype == "float32" else 4e-2, f"cuts {cuts}")
    mixer.free()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads", [(4, 1, 128, 128, 1.0), (2, 2, 64, 64, 1.5), (2, 1, 40, 48, 2.0)])
@pytest.mark.parametrize("rising", [True, False])
def test_attention_scores_that_rise_or_fall_along_the_sequence(lm, dtype, heads, rising):
    """The largest score moves by far more than 2^8 from one tile of keys to the next."""
    from peregrine_b200.layers import Attention

    p, width, T = t.attention(*heads), 64, 400
    d = device(lm, dtype, T)
    x, W = planted(p, width, T, 0, 0)
    x[:, -2] = 10.0
    ramp = np.linspace(0, 3, T) if rising else np.linspace(3, 0, T)
    x[:, -1] = ramp
    x = t.bf16_values(x)
    want, _ = so.attention_mixer(x.astype(np.float64), {k: v.astype(np.float64) for k, v in W.items()}, p, 1e-4, so.attention_start(p), 0)
    mixer = Attention(d, p, W, width, 1e-4, 500, 3)
    for cuts in ([T], [T - 40] + [1] * 40, [130, 2, 268]):
        got, _ = run_mixer(lm, d, mixer, width, x, cuts)
        # (scores up to 128: rounding q and k to 16 bits moves them by a third)
        close(got, want, 2e-4 if dtype == "float32" else 0.25, f"cuts {cuts[:2]}")
    mixer.free()


@pytest.mark.parametrize("dtype", DTYPES)
def test_attention_sink(lm, dtype):
    """All scores far below 0: nearly everything goes to the sink; the first token has only itself and the sink."""
    from peregrine_b200.layers import Attention

    p, width, T = t.attention(2, 1, 16, 16, 0.6), 64, 70
    d = device(lm, dtype, 80)
    x, W = planted(p, width, T, 0, 0)
    for name, sign in (("q", 1.0), ("k", -1.0)):
        W[name].reshape(-1, p["dim"], width)[:, 0, :] = 0.0
        W[name].reshape(-1, p["dim"], width)[:, 0, 0] = sign * 4.0
    x[:, 0] = 10.0
    x = t.bf16_values(x)
    W64 = {k: v.astype(np.float64) for k, v in W.items()}
    want, _ = so.attention_mixer(x.astype(np.float64), W64, p, 1e-4, so.attention_start(p), 0)
    v = x.astype(np.float64) @ W64["v"].T @ W64["o"].reshape(width, 2, 16).sum(1).T
    assert np.abs(want).max() < 0.2 * np.abs(v).max()     # without the sink the weights would add up to one
    mixer = Attention(d, p, W, width, 1e-4, 128, 3)
    for cuts in ([T], [1] * T):
        got, _ = run_mixer(lm, d, mixer, width, x, cuts)
        close(got, want, 3e-5 if dtype == "float32" else 0.1)
    mixer.free()


def test_attention_refuses_positions_behind_its_cache(lm):
    from peregrine_b200 import _lib
    from peregrine_b200.layers import Attention, Batch
    from peregrine_b200.state import SlotPool

    p, width = ATTENTIONS[0], 64
    W = {k: t.bf16_values(v) for k, v in t.mixer_weights(rng(1), "attention", p, width).items()}
    for dtype in DTYPES:
        d = device(lm, dtype)
        mixer = Attention(d, p, W, width, 1e-4, 8, 1)
        state = mixer.new_state(SlotPool(1, 8, d.dev))
        y = d.torch.zeros(64, width, device=d.dev)
        for n in (1, 3):
            h = act(d, np.zeros((n, width), np.float32))
            mixer.run(Batch(d, [(0, 8, [0] * n)]), h, state, y)
            assert lm.device_status() == _lib.PG_ERR_INVALID
        assert not state["k"].any() and not state["v"].any()
        mixer.free()


# ---- whole models --------------------------------------------------------------------------------------------------------
def make_engine(lm, cfg, W, dtype, slots=3, portion=0, step_rows=64):
    from peregrine_b200.engine import Engine
    from peregrine_b200.sonalorn import SonalornConfig, SonalornModel

    bits = {k: t.to_bits(v) for k, v in W.items()}
    return Engine(SonalornModel(SonalornConfig.from_dict(cfg), bits, lm, dtype=dtype, slots=slots, step_rows=step_rows, max_wanted=16), portion=portion)


# the error of logits, rms over the vocabulary relative to the reference's rms, that rounding causes in these models
MODEL_TOL = {"float32": 2e-4, "bfloat16": 8e-2}


def logit_error(got, want):
    e = np.asarray(got, np.float64) - want
    e -= e.mean(-1, keepdims=True)
    return np.sqrt((e ** 2).mean(-1)) / np.sqrt((want ** 2).mean())


@pytest.mark.parametrize("make", [t.small_config, t.other_config])
@pytest.mark.parametrize("dtype", DTYPES)
def test_model_however_a_prompt_is_cut(lm, dtype, make):
    cfg = make()
    W = t.weights(cfg, 11)
    oracle = so.Model(cfg, W)
    g = rng(12)
    e = make_engine(lm, cfg, W, dtype)
    for T in (1, 2, 37, 150):
        tokens = g.integers(0, cfg["vocab"], T).tolist()
        want = oracle.forward(tokens, oracle.start())
        for cuts in ([T], [1] * T, [2] * (T // 2) + [1] * (T % 2), [T - T // 3] + [1] * (T // 3)):
            at, got = 0, []
            for n in cuts:
                got.append(e.step([("r", tokens[at:at + n], list(range(n)))]))
                at += n
            e.end("r")
            err = logit_error(np.concatenate(got), want)
            assert np.median(err) < MODEL_TOL[dtype] / 2 and err.max() < MODEL_TOL[dtype] * (1 if dtype == "float32" else 6), (T, cuts[:3], err.max())
    # (a bf16 router can choose differently at a close call: single positions may be further off)
    e.close()


def ragged_config():
    """Widths at which prompts run on the tcgen05 attention kernel and the delta rule in its 16-byte forms."""
    return t.config(83, 128, [t.layer("attention", t.attention(4, 1, 64, 64, 0.2, (0.4, 50)), t.dense(72)),
                              t.layer("delta", t.delta(4, 2, 64, 32, 4), None),
                              t.layer("attention", t.attention(4, 2, 128, 64, 0.1), None)], max_positions=500)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("make,lengths,cuts", [
    (t.small_config, {"a": 90, "b": 7, "c": 41}, {"a": [30, 1, 1, 40, 18], "b": [2, 1, 1, 1, 2], "c": [1, 1, 30, 1, 8]}),
    (ragged_config, {"a": 370, "b": 8, "c": 180}, {"a": [200, 1, 60, 1, 108], "b": [2, 1, 2, 1, 2], "c": [33, 1, 130, 1, 15]})])
def test_unequal_requests_together_equal_each_alone(lm, dtype, make, lengths, cuts):
    cfg = make()
    W = t.weights(cfg, 21)
    oracle = so.Model(cfg, W)
    g = rng(22)
    prompts = {k: g.integers(0, 83, n).tolist() for k, n in lengths.items()}
    alone, together = {}, {k: [] for k in prompts}
    e = make_engine(lm, cfg, W, dtype, step_rows=400)
    for k, x in prompts.items():
        alone[k] = e.step([(k, x, list(range(len(x))))])
        e.end(k)
    # in mixed steps, each with slots that others have used
    at = dict.fromkeys(prompts, 0)
    for i in range(5):
        entries = []
        for k, x in prompts.items():
            n = cuts[k][i]
            entries.append((k, x[at[k]:at[k] + n], list(range(n))))
            at[k] += n
        out = e.step(entries)
        o = 0
        for k, x, want in entries:
            together[k].append(out[o:o + len(want)])
            o += len(want)
    for k, x in prompts.items():
        assert at[k] == len(x)
        err = logit_error(np.concatenate(together[k]), alone[k].astype(np.float64))
        assert np.median(err) < MODEL_TOL[dtype] / 4 and (dtype == "bfloat16" or err.max() < 1e-4), k
        err = logit_error(alone[k], oracle.forward(x, oracle.start()))
        assert np.median(err) < MODEL_TOL[dtype] / 2, k
    e.close()


def test_a_slot_used_again_starts_from_nothing(lm):
    cfg = t.small_config()
    e = make_engine(lm, cfg, t.weights(cfg, 31), "bfloat16", slots=1)
    g = rng(32)
    x, other = g.integers(0, 83, 40).tolist(), g.integers(0, 83, 120).tolist()
    for first in (x[:1], x[:3], x):
        fresh = e.step([("x", first, [len(first) - 1])])
        e.end("x")
        e.step([("y", other, [])])
        for tok in other[:5]:
            e.step([("y", [tok], [])])
        e.end("y")
        again = e.step([("x", first, [len(first) - 1])])
        assert np.array_equal(fresh, again)
        e.end("x")
    e.close()


def test_a_layer_with_another_layers_weights_has_its_own_state(lm):
    cfg = t.small_config()
    W = t.weights(cfg, 41)
    e = make_engine(lm, cfg, W, "float32")
    m = e.model
    assert m.layers[1]["mixer"] is m.layers[2]["mixer"] and m.layers[1]["state"]["state"].data_ptr() != m.layers[2]["state"]["state"].data_ptr()
    # the same model with the tensors written out twice
    cfg2 = t.small_config()
    cfg2["layers"][2].pop("weights_of")
    W2 = dict(W, **{k.replace("l1.", "l2."): v for k, v in W.items() if k.startswith("l1.")})
    e2 = make_engine(lm, cfg2, W2, "float32")
    tokens = rng(42).integers(0, 83, 30).tolist()
    assert np.array_equal(e.step([("r", tokens, [0, 29])]), e2.step([("r", tokens, [0, 29])]))
    e.close()
    e2.close()


def greedy(oracle, prompt, n):
    """The oracle's continuation and the smallest lead of a chosen token over the next best."""
    state, out, lead = oracle.start(), [], np.inf
    logits = oracle.forward(prompt, state)[-1]
    while True:
        two = np.sort(logits)[-2:]
        lead = min(lead, two[1] - two[0])
        out.append(int(logits.argmax()))
        if len(out) == n:
            return out, lead
        logits = oracle.forward(out[-1:], state)[-1]


def test_greedy_generation_through_the_scheduler(lm):
    """Five prompts in three slots, portions of 16 tokens, decoding as recorded graphs: what the oracle gives for each."""
    cfg = t.small_config()
    W = t.weights(cfg, 51)
    W["head"] = t.bf16_values(W["head"] * 2)
    oracle = so.Model(cfg, W)
    g = rng(52)
    prompts = [g.integers(0, 83, n).tolist() for n in (1, 33, 5, 18, 64)]
    want = [greedy(oracle, p, 12) for p in prompts]
    e = make_engine(lm, cfg, W, "float32", portion=16)
    for _ in range(2):
        got = e.generate(prompts, 12)
        for a, (b, lead) in zip(got, want):
            assert a == b or lead < 1e-3
    stop = want[1][0][3]
    assert e.generate([prompts[1]], 12, stop=[stop])[0] == want[1][0][:want[1][0].index(stop) + 1]
    e.close()


def test_long_decoding_in_bf16(lm):
    """180 tokens fed one by one through the decode path, against the oracle on the same tokens."""
    cfg = t.other_config()
    W = t.weights(cfg, 61)
    oracle = so.Model(cfg, W)
    tokens = rng(62).integers(0, 61, 190).tolist()
    want = oracle.forward(tokens, oracle.start())
    e = make_engine(lm, cfg, W, "bfloat16")
    got = [e.step([("r", tokens[:3], [0, 1, 2])])] + [e.step([("r", [x], [0])]) for x in tokens[3:]]
    err = logit_error(np.concatenate(got), want)
    assert np.median(err) < MODEL_TOL["bfloat16"] / 2 and np.median(err[-40:]) < MODEL_TOL["bfloat16"]
    e.close()


def test_wider_layers(lm):
    """Sizes at which the kernels take their other forms: clusters over K, 128-wide heads, many experts."""
    cfg = t.config(300, 640, [t.layer("delta", t.delta(8, 4, 128, 128, 4), t.dense(4300)),
                              t.layer("attention", t.attention(16, 2, 128, 64, 0.09, (0.4, 32)), t.moe(200, 1.2, 40, 8, 6, (8, 4)))], max_positions=260)
    W = t.weights(cfg, 71)
    oracle = so.Model(cfg, W, np.float32)
    tokens = rng(72).integers(0, 300, 70).tolist()
    want = oracle.forward(tokens, oracle.start()).astype(np.float64)
    for dtype in DTYPES:
        e = make_engine(lm, cfg, W, dtype)
        got = np.concatenate([e.step([("r", tokens[:50], list(range(50)))])] + [e.step([("r", [x], [0])]) for x in tokens[50:]])
        err = logit_error(got, want)
        assert np.median(err) < (1e-4 if dtype == "float32" else 4e-2)
        e.close()


# ---- the command line ------------------------------------------------------------------------------------------------------
def test_command_line(lm, tmp_path):
    cfg = t.small_config()
    W = t.weights(cfg, 81)
    t.save(str(tmp_path / "model"), cfg, W)
    e = make_engine(lm, cfg, W, "bfloat16")
    prompts = [[1, 2, 3, 4, 5], [80, 7]]
    want = e.generate(prompts, 5)
    r = subprocess.run([sys.executable, "-m", "peregrine_b200", "generate", "--model", str(tmp_path / "model"), "--max-new", "5", "--prompt", "1,2,3,4,5",
                        "--prompt", "80,7"], cwd=ROOT, capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert [[int(x) for x in line.split(",")] for line in r.stdout.split()] == want
    steps = '{"step": 0, "entries": [{"id": "a", "tokens": [1, 2, 3], "want": [0, 2]}], "end": []}\n' \
            '{"step": 1, "entries": [{"id": "a", "tokens": [4], "want": []}], "end": ["a"]}\n' \
            '{"step": 2, "entries": [{"id": "b", "tokens": [1], "want": [0]}], "end": ["b"]}\n'
    out = tmp_path / "out"
    out.mkdir()
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path / "model"), "--dtype", "bfloat16", "--out", str(out), "--max-tokens", "64"],
                       input=steps, cwd=str(tmp_path), capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert r.stdout.split("\n")[:3] == ["done 0", "done 1", "done 2"] and sorted(os.listdir(out)) == ["0.f32", "2.f32"]
    a = np.fromfile(out / "0.f32", "<f4").reshape(2, 83)
    assert np.array_equal(a, e.step([("a", [1, 2, 3], [0, 2])]))
    # one position, whatever else ran: the same logits up to the rounding of another kernel's sums
    assert logit_error(np.fromfile(out / "2.f32", "<f4")[None], a[:1].astype(np.float64)).max() < MODEL_TOL["bfloat16"]
    e.close()
