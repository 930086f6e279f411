"""Every mechanism of the Bubotar layers alone, whole models, and serving, on the GPU against oracle/bubotar_oracle.py."""
import ctypes as C
import os
import subprocess
import sys

import numpy as np
import pytest

from oracle import bubotar_oracle as bo
from tests import _bubotar as t

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


def act(d, a):
    """[rows, cols] -> the step's type on the device, columns padded with zeros to a multiple of 64."""
    x = np.zeros((a.shape[0], (a.shape[1] + 63) // 64 * 64), np.float32)
    x[:, :a.shape[1]] = a
    out = d.torch.from_numpy(x).to(d.dev).to(d.act)
    d.torch.cuda.synchronize()
    return out


def wide(W):
    return {k: v.astype(np.float64) for k, v in W.items()}


def close(got, want, tol, what=""):
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    assert got.shape == want.shape and np.isfinite(got).all(), what
    rms = max(1e-30, np.sqrt(np.mean(want ** 2)))
    worst, mean = np.abs(got - want).max() / rms, np.sqrt(np.mean((got - want) ** 2)) / rms
    assert mean <= tol and worst <= 10 * tol, f"{what}: rms error {mean:.3g}, largest {worst:.3g} of the rms, tolerance {tol:.3g}"


def tensors(kind, p, width, seed):
    return {k: t.bf16_values(v) for k, v in t.mixer_weights(rng(seed), kind, p, width).items()}


def run_mixer(lm, d, mixer, width, x, cuts, state, slot=1):
    """x [T, width] in portions -> [T, width] outputs."""
    from peregrine_b200.layers import Batch, up

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
    return np.concatenate(out)


def new_state(d, mixer, slots=3, capacity=512):
    from peregrine_b200.state import SlotPool

    s = mixer.new_state(SlotPool(slots, capacity, d.dev))
    d.torch.cuda.synchronize()
    return s


# ---- residual rows and products ----------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [5, 70, 256, 1030, 4096])
def test_rows_with_norms_on_both_sides(lm, dtype, width):
    from peregrine_b200.layers import Batch, up

    d = device(lm, dtype, 400)
    t_ = d.torch
    g = rng(width)
    tol = 2e-2 if dtype == "bfloat16" else 5e-6
    for m in (1, 3, 40, 330):
        table = t.bf16_values(g.standard_normal((20, width)) * 3)
        w, nxt, eps = g.standard_normal(width).astype(np.float32), g.standard_normal(width).astype(np.float32), 0.01
        tokens = g.integers(0, 20, m)
        b = Batch(d, [(0, 7, tokens.tolist())])
        x = t_.zeros(m, width, device=d.dev)
        h = t_.zeros(m, up(width, 64), dtype=d.act, device=d.dev)
        dt, dw, dn = d.bf16(table), d.f32(w), d.f32(nxt)
        y = g.standard_normal((m, width)).astype(np.float32)
        dy = t_.zeros(m, up(width, 4), device=d.dev)
        dy[:, :width] = d.f32(y)
        t_.cuda.synchronize()
        ck, lib, gh = d.check, d.lib, lm.handle
        ck(lib.pg_embed_prenorm(gh, C.byref(b.c), dt.data_ptr(), width, dn.data_ptr(), eps, x.data_ptr(), h.data_ptr(), d.code, h.stride(0)))
        lm.sync()
        want = table[tokens].astype(np.float64)
        assert np.array_equal(x.cpu().numpy(), want.astype(np.float32))
        close(h[:, :width].float().cpu().numpy(), bo.rms_norm(want, nxt, eps), tol, "embed h")
        for following in (dn, None):
            ck(lib.pg_norm_add_prenorm(gh, dy.data_ptr(), dy.stride(0), x.data_ptr(), dw.data_ptr(), following.data_ptr() if following is not None else 0, m, width,
                                       eps, h.data_ptr(), d.code, h.stride(0)))
            lm.sync()
            want = want + bo.rms_norm(y.astype(np.float64), w, eps)
            close(x.cpu().numpy(), want, 5e-6, "add")
            close(h[:, :width].float().cpu().numpy(), bo.rms_norm(want, nxt, eps) if following is not None else want, tol, "add h")
        assert (h[:, width:] == 0).all()


@pytest.mark.parametrize("dtype", DTYPES)
def test_product_of_rows_that_lie_apart(lm, dtype):
    from peregrine_b200.layers import Linear

    d = device(lm, dtype, 300)
    g = rng(4)
    n, k, ld = 90, 128, 168
    w = t.bf16_values(g.standard_normal((n, k)) / k ** 0.5)
    lin = Linear(d, d.bf16(w))
    for m in (1, 9, 16, 40, 300):
        a = t.bf16_values(g.standard_normal((m, ld)))
        x = d.torch.from_numpy(a).to(d.dev).to(d.act)
        y = d.torch.zeros(m, 96, device=d.dev)
        d.torch.cuda.synchronize()
        lin.run_ld(x.data_ptr(), ld, m, y)
        lm.sync()
        close(y[:, :n].cpu().numpy(), a[:, :k].astype(np.float64) @ w.T, 2e-5, f"m {m}")
    lin.free()


@pytest.mark.parametrize("dtype", DTYPES)
def test_clamped_feed_forward(lm, dtype):
    from peregrine_b200.layers import Batch, DenseFF, up

    d = device(lm, dtype, 200)
    g = rng(8)
    for width, ff, limit in ((96, 40, 0.7), (70, 133, 2.2), (256, 520, 1.0)):
        W = {k: t.bf16_values(v) for k, v in t.mlp_weights(g, t.dense(ff, limit), width).items()}
        layer = DenseFF(d, t.dense(ff, limit), W, width)
        for m in (1, 16, 150):
            x = t.bf16_values(g.standard_normal((m, width)))
            y = d.torch.zeros(m, up(width, 4), device=d.dev)
            layer.run(Batch(d, [(0, 0, [0] * m)]), act(d, x), y, lambda out: None)
            lm.sync()
            close(y[:, :width].cpu().numpy(), bo.dense_ff(x.astype(np.float64), wide(W), limit), 1e-5 if dtype == "float32" else 2e-2, f"{width} {m}")
        layer.free()


# ---- selective scan ------------------------------------------------------------------------------------------------------
SCANS = [t.mamba(72, 5, 7, 3), t.mamba(192, 16, 8, 4), t.mamba(40, 18, 70, 4), t.mamba(33, 1, 1, 1), t.mamba(130, 64, 64, 2), t.mamba(64, 100, 5, 5),
         t.mamba(36, 200, 3, 4), t.mamba(31, 32, 130, 7), t.mamba(520, 13, 20, 4)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("p", SCANS)
def test_scan(lm, dtype, p):
    from peregrine_b200.layers import SelectiveScan

    width, T = 80, 45
    d = device(lm, dtype)
    W = tensors("mamba1", p, width, p["inner"])
    mixer = SelectiveScan(d, p, W, width)
    x = t.bf16_values(rng(1).standard_normal((T, width)))
    want, carried = bo.mamba_mixer(x.astype(np.float64), wide(W), p, bo.mamba_start(p))
    N = p["state"]
    for cuts in ([45], [1] * 45, [2, 1, 3, 1, 1, 17, 16, 2, 2], [16, 16, 13]):
        state = new_state(d, mixer)
        state["ring"].normal_(), state["state"][:, :, :N].normal_()      # what a slot held before is not seen
        before = state["state"].clone()
        d.torch.cuda.synchronize()
        got = run_mixer(lm, d, mixer, width, x, cuts, state)
        close(got, want, 1e-5 if dtype == "float32" else 2.5e-2, f"cuts {cuts}")
        S = state["state"][1].cpu().numpy()
        close(S[:, :N], carried["S"], 1e-5 if dtype == "float32" else 2.5e-2, "state")
        assert (S[:, N:] == 0).all() and (state["state"][0] == before[0]).all() and (state["state"][2] == before[2]).all()
    mixer.free()


def test_scan_state_is_f32_over_a_long_sequence(lm):
    """Slow decay and small writes: a state or a decay rounded to 16 bits is far off after 500 tokens."""
    from peregrine_b200.layers import SelectiveScan

    p, width, T = t.mamba(48, 12, 4, 3), 64, 500
    W = tensors("mamba1", p, width, 3)
    W["A_log"], W["dt.b"] = t.bf16_values(np.full((48, 12), -3.0)), t.bf16_values(np.full(48, -3.0))
    W["dt"] = t.bf16_values(W["dt"] * 0.2)
    x = t.bf16_values(rng(78).standard_normal((T, width)))
    want, carried = bo.mamba_mixer(x.astype(np.float64), wide(W), p, bo.mamba_start(p))
    for dtype in DTYPES:
        d = device(lm, dtype, 512)
        mixer = SelectiveScan(d, p, W, width)
        for cuts in ([T], [300] + [1] * (T - 300)):
            state = new_state(d, mixer)
            run_mixer(lm, d, mixer, width, x, cuts, state)
            close(state["state"][1].cpu().numpy(), carried["S"], 2e-5 if dtype == "float32" else 1e-2, dtype)
        mixer.free()


# ---- chunked attention with a distance bias --------------------------------------------------------------------------------
def chunked(d, p, W, width, capacity=512, seqs=3):
    from peregrine_b200.layers import Attention, halving_slopes

    return Attention(d, p, W, width, 1e-4, capacity, seqs, sink=False, norms=False, slopes=halving_slopes(p["heads"]), chunk=p["mask"]["size"])


ATTENTIONS = [t.attention(6, 2, 40, 24, 0.3, 11), t.attention(8, 1, 64, 64, 0.2, 64), t.attention(2, 2, 128, 128, 0.1, 100), t.attention(34, 2, 16, 80, 0.4, 130),
              t.attention(4, 4, 200, 256, 0.08, 33), t.attention(3, 1, 5, 7, 1.0, 1), t.attention(8, 2, 80, 112, 0.15, 129), t.attention(4, 1, 128, 64, 0.12, 500),
              t.attention(5, 5, 48, 36, 0.2, 3), t.attention(4, 2, 72, 20, 0.2, 128)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("p", ATTENTIONS)
def test_chunked_attention(lm, dtype, p):
    width, T = 80, 300
    d = device(lm, dtype, 300)
    W = tensors("attention", p, width, p["dim"])
    mixer = chunked(d, p, W, width)
    x = t.bf16_values(rng(2).standard_normal((T, width)))
    want, _ = bo.attention_mixer(x.astype(np.float64), wide(W), p, bo.attention_start(p), 0)
    for cuts in ([T], [1] * 20 + [2, 60, 3, 64] + [1] + [150], [170] + [1] * 120 + [2, 8], [2] * 30 + [129, 111]):
        state = new_state(d, mixer)
        state["k"].normal_(), state["v"].normal_()
        d.torch.cuda.synchronize()
        got = run_mixer(lm, d, mixer, width, x, cuts, state)
        close(got, want, 1e-5 if dtype == "float32" else 2e-2, f"cuts {cuts[:4]}")
    mixer.free()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size,rows", [(16, 64), (7, 24), (50, 64), (64, 130)])
def test_a_ring_of_chunks_is_used_again(lm, dtype, size, rows):
    """More positions than the cache has rows: only the chunks that a step can touch are kept."""
    p, width, T = t.attention(4, 2, 64, 64, 0.2, size), 64, 700
    d = device(lm, dtype, rows)
    W = tensors("attention", p, width, size)
    mixer = chunked(d, p, W, width, capacity=T)
    assert mixer.cap % size == 0 and mixer.cap < T / 2
    x = t.bf16_values(rng(3).standard_normal((T, width)))
    want, _ = bo.attention_mixer(x.astype(np.float64), wide(W), p, bo.attention_start(p), 0)
    cuts, g, left = [], rng(4), T
    while left:
        cuts.append(min(left, int(g.choice([1, 1, 2, 5, rows // 2, rows - 1, rows]))))
        left -= cuts[-1]
    for c in (cuts, [rows] * (T // rows) + ([T % rows] if T % rows else [])):
        got = run_mixer(lm, d, mixer, width, x, c, new_state(d, mixer, capacity=T))
        close(got, want, 1e-5 if dtype == "float32" else 2e-2, f"cuts {c[:6]}")
    mixer.free()


def plant(x, W, columns, far, at, strength=40.0):
    """The query of position `at` and the key of position `far`, and no others, lie along one direction of every head.
    columns: (tensor, rows of it that make the direction, input column)."""
    x[:, -2:] = 0.0
    x[at, -2] = strength
    x[far, -1] = strength
    for name, rows, col in columns:
        W[name][:, -2:] = 0.0
        W[name][rows, col] = 4.0
    return t.bf16_values(x)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads", [(4, 2, 32, 32, 0.5), (4, 1, 64, 128, 0.25), (6, 2, 96, 40, 0.3)])
@pytest.mark.parametrize("size,at,far", [(50, 399, 350), (50, 399, 349), (50, 350, 349), (50, 350, 350), (50, 351, 350), (128, 383, 256), (128, 383, 255),
                                         (128, 256, 255), (100, 299, 200), (100, 299, 199), (400, 399, 0), (130, 389, 260), (130, 389, 259)])
def test_chunk_edges(lm, dtype, heads, size, at, far):
    """One key carries the answer if it is just inside the query's chunk, and nothing of it shows if it is just outside."""
    p, width = t.attention(*heads, size), 64
    T = at + 3
    d = device(lm, dtype, T)
    W = tensors("attention", p, width, at + far)
    x = (rng(far).standard_normal((T, width)) * 0.2).astype(np.float32)
    x = plant(x, W, [("q", slice(0, None, p["dim"]), -2), ("k", slice(0, None, p["dim"]), -1)], far, at)
    W["v"][:, -2] = 0.0
    W["v"][:, -1] = t.bf16_values(rng(9).standard_normal(len(W["v"])))
    want, _ = bo.attention_mixer(x.astype(np.float64), wide(W), p, bo.attention_start(p), 0)
    x2 = x.copy()
    x2[far, -1] = 0.0
    without, _ = bo.attention_mixer(x2.astype(np.float64), wide(W), p, bo.attention_start(p), 0)
    change = np.abs(want[at] - without[at]).max() / np.sqrt(np.mean(want[at] ** 2))
    assert (change > 0.5) if far // size == at // size else change == 0
    mixer = chunked(d, p, W, width)
    for cuts in ([T], [at, 1, 2], [at - 1, 2, 2], [100, 2, 3, T - 108, 2, 1]):
        got = run_mixer(lm, d, mixer, width, x, cuts, new_state(d, mixer))
        close(got[at:at + 1], want[at:at + 1], 2e-5 if dtype == "float32" else 4e-2, f"cuts {cuts}")
        close(got[at + 1:], want[at + 1:], 2e-5 if dtype == "float32" else 4e-2, f"behind, cuts {cuts}")
    mixer.free()


@pytest.mark.parametrize("dtype", DTYPES)
def test_distance_bias(lm, dtype):
    """Without scores of their own, the weights are the bias alone: steep for the first heads, nearly flat for the last."""
    p, width, T = t.attention(8, 4, 64, 64, 0.5, 300), 64, 290
    d = device(lm, dtype, T)
    W = tensors("attention", p, width, 5)
    W["q"][:] = 0.0
    x = t.bf16_values(rng(6).standard_normal((T, width)))
    want, _ = bo.attention_mixer(x.astype(np.float64), wide(W), p, bo.attention_start(p), 0)
    mixer = chunked(d, p, W, width)
    for cuts in ([T], [200] + [1] * 90, [30] * 9 + [20]):
        got = run_mixer(lm, d, mixer, width, x, cuts, new_state(d, mixer))
        close(got, want, 1e-5 if dtype == "float32" else 1e-2, f"cuts {cuts[:2]}")
    mixer.free()


def test_chunked_attention_refuses_what_its_ring_does_not_hold(lm):
    from peregrine_b200 import _lib
    from peregrine_b200.layers import Batch, Device

    p, width = t.attention(4, 2, 32, 32, 0.3, 8), 64
    W = tensors("attention", p, width, 1)
    for dtype in DTYPES:
        d = device(lm, dtype, 16)
        mixer = chunked(d, p, W, width, capacity=100)
        state = new_state(d, mixer)
        big = Device(lm, dtype, 64)
        y = d.torch.zeros(64, width, device=d.dev)
        h = act(d, np.zeros((40, width), np.float32))
        mixer.proj.d = mixer.out.d = mixer.d = big
        for name, cols, dt in (("proj", mixer.proj.n, d.torch.float32), ("mixed", mixer.out.k, None), ("attn.q", 4 * mixer.dp, None),
                               ("attn.part", 1, d.torch.float32), ("attn.tickets", 1, d.torch.int32)):
            big.buffer(name, cols, dtype=dt)
        d.torch.cuda.synchronize()
        with pytest.raises(_lib.InvalidArgument):
            mixer.run(Batch(big, [(0, 0, [0] * 40)]), h, state, y)
        mixer.free()


# ---- latent attention ----------------------------------------------------------------------------------------------------
LATENTS = [t.latent(6, 20, 6, 12, 40, 0.25, 500.0), t.latent(4, 64, 32, 64, 128, 0.1), t.latent(17, 8, 2, 5, 70, 0.35), t.latent(2, 128, 64, 128, 512, 0.08, 2e5),
           t.latent(32, 48, 16, 80, 64, 0.15), t.latent(1, 33, 18, 17, 1, 0.4), t.latent(3, 96, 64, 40, 200, 0.1), t.latent(40, 16, 4, 24, 320, 0.2),
           t.latent(2, 160, 16, 200, 96, 0.1), t.latent(16, 32, 128, 32, 448, 0.1)]


def latent_layers(d, p, width, seed, capacity=512):
    """A layer with latents of its own and one of other heads that reads its cache; their weights."""
    from peregrine_b200.layers import LatentAttention

    q = dict(p, heads=p["heads"] + 1, dim=p["dim"] + 8, vdim=max(1, p["vdim"] - 4), scale=p["scale"] * 0.7, kv_from=0)
    W, V = tensors("latent_attention", p, width, seed), tensors("latent_attention", q, width, seed + 1)
    return (p, W, LatentAttention(d, p, W, width, 1e-4, capacity, 3)), (q, V, LatentAttention(d, q, V, width, 1e-4, capacity, 3, own=False))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("p", LATENTS)
def test_latent_attention(lm, dtype, p):
    from peregrine_b200.layers import Batch, up

    width, T = 80, 230
    d = device(lm, dtype, 240)
    (p, W, own), (q, V, reader) = latent_layers(d, p, width, p["dim"])
    x = t.bf16_values(rng(2).standard_normal((T, width)))
    want, carried = bo.latent_mixer(x.astype(np.float64), wide(W), p, 1e-4, bo.latent_start(p), 0)
    want2, _ = bo.latent_mixer(x.astype(np.float64), wide(V), q, 1e-4, bo.latent_start(q), 0, carried)
    tol = 1e-5 if dtype == "float32" else 2.5e-2
    for cuts in ([T], [1] * 20 + [2, 60, 3, 64, 1, 80], [130] + [1] * 66 + [2, 32], [70, 70, 65, 25], [63, 64, 65, 38]):
        state = new_state(d, own)
        state["latent"][:, :, :p["kv_rank"]].normal_()
        other = state["latent"][[0, 2]].clone()
        y = d.torch.zeros(d.rows, up(width, 4), device=d.dev)
        d.torch.cuda.synchronize()
        got, got2, at = [], [], 0
        for n in cuts:
            b, h = Batch(d, [(1, at, [0] * n)]), act(d, x[at:at + n])
            for mixer, out in ((own, got), (reader, got2)):
                mixer.run(b, h, state, y)
                lm.sync()
                out.append(y[:n, :width].cpu().numpy())
            at += n
        close(np.concatenate(got), want, tol, f"cuts {cuts[:4]}")
        close(np.concatenate(got2), want2, tol, f"shared latents, cuts {cuts[:4]}")
        cache = state["latent"][1, :T].float().cpu().numpy()
        close(cache[:, :p["kv_rank"]], carried["c"], 1e-5 if dtype == "float32" else 1e-2, "latents")
        close(cache[:, own.cp:own.cp + p["rot_dim"]], carried["kr"], 1e-5 if dtype == "float32" else 1e-2, "key parts")
        assert (state["latent"][[0, 2]] == other).all() and lm.device_status() == 0
    own.free()
    reader.free()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [(4, 24, 8, 16, 48, 0.5), (17, 64, 16, 64, 64, 0.2), (2, 128, 64, 128, 256, 0.1)])
@pytest.mark.parametrize("far", [0, 1, 63, 64, 65, 127, 128, 300, 440, 446])
def test_latent_attention_far_key(lm, dtype, sizes, far):
    """One latent among hundreds carries the answer: at tile and slice borders, at the start, just in front of the query."""
    from peregrine_b200.layers import LatentAttention

    p, width, T = t.latent(*sizes, base=800.0), 64, 448
    d = device(lm, dtype, T)
    W = tensors("latent_attention", p, width, far)
    x = (rng(far).standard_normal((T, width)) * 0.2).astype(np.float32)
    x = plant(x, W, [("q", slice(0, None, p["dim"] + p["rot_dim"]), -2), ("dkv", slice(0, 1), -1)], far, T - 1)
    W["dkv"][0, :-1], W["dkv"][1:, -1] = 0.0, 0.0            # the first latent column is the planted token's alone
    W["dkv.norm"][:] = 1.0
    W["uk"][:, 0] = 0.0
    W["uk"][::p["dim"], 0] = 4.0
    W["g"][:, -2] = 0.0
    want, _ = bo.latent_mixer(x.astype(np.float64), wide(W), p, 1e-4, bo.latent_start(p), 0)
    x2 = x.copy()
    x2[far, -1] = 0.0
    without, _ = bo.latent_mixer(x2.astype(np.float64), wide(W), p, 1e-4, bo.latent_start(p), 0)
    assert np.abs(want[-1] - without[-1]).max() > 0.5 * np.sqrt(np.mean(want[-1] ** 2))     # the key matters
    mixer = LatentAttention(d, p, W, width, 1e-4, 500, 3)
    for cuts in ([T], [T - 1, 1], [100, 2, 3, T - 108, 2, 1], [T - 40, 40], [T - 90, 90]):
        got = run_mixer(lm, d, mixer, width, x, cuts, new_state(d, mixer, capacity=500))
        close(got[-1:], want[-1:], 2e-5 if dtype == "float32" else 4e-2, f"cuts {cuts}")
    mixer.free()


@pytest.mark.parametrize("dtype", DTYPES)
def test_latent_attention_rotation_decides(lm, dtype):
    """Scores come from the rotated parts alone, so the answer depends on the distance, for near and far keys."""
    from peregrine_b200.layers import LatentAttention

    p, width, T = t.latent(4, 16, 8, 32, 32, 0.6, 60.0), 64, 260
    d = device(lm, dtype, T)
    W = tensors("latent_attention", p, width, 12)
    W["uk"][:] = 0.0
    W["q"] = t.bf16_values(W["q"] * 2)
    x = t.bf16_values(rng(13).standard_normal((T, width)))
    want, _ = bo.latent_mixer(x.astype(np.float64), wide(W), p, 1e-4, bo.latent_start(p), 0)
    mixer = LatentAttention(d, p, W, width, 1e-4, 500, 3)
    for cuts in ([T], [200] + [1] * 60, [30] * 8 + [20]):
        got = run_mixer(lm, d, mixer, width, x, cuts, new_state(d, mixer, capacity=500))
        close(got, want, 2e-5 if dtype == "float32" else 4e-2, f"cuts {cuts[:2]}")
    mixer.free()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rising", [True, False])
def test_latent_scores_that_rise_or_fall_along_the_sequence(lm, dtype, rising):
    """The largest score moves by far more than 2^8 from one tile of keys to the next (through the rotated part, which is not
    normed)."""
    from peregrine_b200.layers import LatentAttention

    p, width, T = t.latent(4, 64, 16, 64, 64, 1.0, 1e9), 64, 400
    d = device(lm, dtype, T)
    W = tensors("latent_attention", p, width, 14)
    x = (rng(15).standard_normal((T, width)) * 0.2).astype(np.float32)
    W["q"][:, -2:], W["dkv"][:, -2:] = 0.0, 0.0
    R, D = p["rot_dim"], p["dim"]
    W["q"].reshape(4, D + R, width)[:, D + R - 2, -2] = 4.0     # the slowest pair hardly turns
    W["dkv"][p["kv_rank"] + R - 2, -1] = 4.0
    x[:, -2], x[:, -1] = 8.0, np.linspace(0, 2, T) if rising else np.linspace(2, 0, T)
    x = t.bf16_values(x)
    want, _ = bo.latent_mixer(x.astype(np.float64), wide(W), p, 1e-4, bo.latent_start(p), 0)
    mixer = LatentAttention(d, p, W, width, 1e-4, 500, 3)
    for cuts in ([T], [T - 40] + [1] * 40, [130, 2, 268]):
        got = run_mixer(lm, d, mixer, width, x, cuts, new_state(d, mixer, capacity=500))
        # (scores up to 256: rounding q and k to 16 bits moves them by more than a half)
        close(got, want, 3e-4 if dtype == "float32" else 0.3, f"cuts {cuts[:2]}")
    mixer.free()


def test_latent_attention_refuses_positions_behind_its_cache(lm):
    from peregrine_b200 import _lib
    from peregrine_b200.layers import Batch, LatentAttention

    p, width = LATENTS[1], 64
    W = tensors("latent_attention", p, width, 1)
    for dtype in DTYPES:
        d = device(lm, dtype)
        mixer = LatentAttention(d, p, W, width, 1e-4, 8, 1)
        state = new_state(d, mixer, 1, 8)
        y = d.torch.zeros(64, width, device=d.dev)
        for n in (1, 3):
            mixer.run(Batch(d, [(0, 8, [0] * n)]), act(d, np.zeros((n, width), np.float32)), state, y)
            assert lm.device_status() == _lib.PG_ERR_INVALID
        assert not state["latent"].any()
        mixer.free()


# ---- whole models --------------------------------------------------------------------------------------------------------
def make_engine(lm, cfg, W, dtype, slots=3, portion=0, step_rows=64, capacity=400):
    from peregrine_b200.bubotar import BubotarConfig, BubotarModel
    from peregrine_b200.engine import Engine

    bits = {k: t.to_bits(v) for k, v in W.items()}
    return Engine(BubotarModel(BubotarConfig.from_dict(cfg), bits, lm, dtype=dtype, slots=slots, capacity=capacity, step_rows=step_rows, max_wanted=16),
                  portion=portion)


# the error of logits, rms over the vocabulary relative to the reference's rms, that rounding causes in these models: of most
# positions, and of the worst (in 16 bits single positions, where small differences decide, are several times further off)
TYPICAL = {"float32": 3e-5, "bfloat16": 2e-2}
WORST = {"float32": 1e-4, "bfloat16": 1e-1}


def logit_error(got, want):
    e = np.asarray(got, np.float64) - want
    e -= e.mean(-1, keepdims=True)
    return np.sqrt((e ** 2).mean(-1)) / np.sqrt((want ** 2).mean())


def check_logits(got, want, dtype, what=None):
    err = logit_error(got, want)
    assert np.median(err) < TYPICAL[dtype] and err.max() < WORST[dtype], (what, np.median(err), err.max())


@pytest.mark.parametrize("make", t.CONFIGS)
@pytest.mark.parametrize("dtype", DTYPES)
def test_model_however_a_prompt_is_cut(lm, dtype, make):
    cfg = make()
    W = t.weights(cfg, 11)
    oracle = bo.Model(cfg, W)
    g = rng(12)
    for step_rows in (64, 256):
        e = make_engine(lm, cfg, W, dtype, step_rows=step_rows)
        for T in (1, 2, 37, 211):
            tokens = g.integers(0, cfg["vocab"], T).tolist()
            want = oracle.forward(tokens, oracle.start())
            for cuts in ([T], [1] * T, [2] * (T // 2) + [1] * (T % 2), [T - T // 3] + [1] * (T // 3)):
                at, got = 0, []
                for n in cuts:
                    got.append(e.step([("r", tokens[at:at + n], list(range(n)))]))
                    at += n
                e.end("r")
                check_logits(np.concatenate(got), want, dtype, (T, cuts[:3]))
        e.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("make", t.CONFIGS)
def test_unequal_requests_together_equal_each_alone(lm, dtype, make):
    cfg = make()
    W = t.weights(cfg, 21)
    oracle = bo.Model(cfg, W)
    g = rng(22)
    lengths = {"a": 370, "b": 8, "c": 180}
    cuts = {"a": [200, 1, 60, 1, 108], "b": [2, 1, 2, 1, 2], "c": [33, 1, 130, 1, 15]}
    prompts = {k: g.integers(0, cfg["vocab"], n).tolist() for k, n in lengths.items()}
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
        check_logits(np.concatenate(together[k]), alone[k].astype(np.float64), dtype, k)
        check_logits(alone[k], oracle.forward(x, oracle.start()), dtype, k)
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
        assert np.array_equal(fresh, e.step([("x", first, [len(first) - 1])]))
        e.end("x")
    e.close()


def test_layers_that_share_latents_share_a_cache(lm):
    cfg = t.small_config()
    e = make_engine(lm, cfg, t.weights(cfg, 41), "float32")
    m = e.model
    assert m.layers[3]["state"] is m.layers[0]["state"] and m.layers[4]["state"] is not m.layers[1]["state"]
    assert m.pool.bytes == sum(v.numel() * 4 for i in (0, 1, 2, 4) for v in m.layers[i]["state"].values())
    e.close()


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


@pytest.mark.parametrize("make", t.CONFIGS)
def test_greedy_generation_through_the_scheduler(lm, make):
    """Six prompts in three slots, portions of 70 tokens, decoding as recorded graphs: what the oracle gives for each."""
    cfg = make()
    W = t.weights(cfg, 51)
    oracle = bo.Model(cfg, W)
    g = rng(52)
    prompts = [g.integers(0, cfg["vocab"], n).tolist() for n in (1, 33, 5, 18, 64, 150)]
    want = [greedy(oracle, p, 12) for p in prompts]
    e = make_engine(lm, cfg, W, "float32", portion=70, step_rows=80)
    for _ in range(2):
        got = e.generate(prompts, 12)
        for a, (b, lead) in zip(got, want):
            assert a == b or lead < 1e-3
    stop = want[1][0][3]
    assert e.generate([prompts[1]], 12, stop=[stop])[0] == want[1][0][:want[1][0].index(stop) + 1]
    e.close()


def test_decoding_is_recorded_without_a_small_product_before_it(lm):
    """A fresh context whose first steps are a long prompt and a recorded decode step with a K that is divided over CTAs."""
    from peregrine_b200.runtime import GpuContext

    gpu = GpuContext(component="lm")
    cfg = t.config(50, 64, [t.layer("attention", t.attention(2, 1, 32, 32, 0.2, 50), t.dense(4400, 1.0))])
    W = t.weights(cfg, 55)
    oracle = bo.Model(cfg, W)
    prompt = rng(56).integers(0, 50, 40).tolist()
    e = make_engine(gpu, cfg, W, "bfloat16")
    out = e.generate([prompt], 6)[0]
    logits = oracle.forward(prompt + out[:-1], oracle.start())[len(prompt) - 1:]
    assert all(row[tok] > np.sort(row)[-1] - 0.1 * np.abs(row).max() for row, tok in zip(logits, out))
    e.close()
    e.model.free()
    gpu.close()


@pytest.mark.parametrize("make", [t.other_config, t.even_config])
def test_long_decoding_in_bf16(lm, make):
    """Hundreds of tokens fed one by one through the decode path, across many chunks, against the oracle on the same tokens."""
    cfg = make()
    W = t.weights(cfg, 61)
    oracle = bo.Model(cfg, W)
    tokens = rng(62).integers(0, cfg["vocab"], 330).tolist()
    want = oracle.forward(tokens, oracle.start())
    e = make_engine(lm, cfg, W, "bfloat16")
    got = [e.step([("r", tokens[:3], [0, 1, 2])])] + [e.step([("r", [x], [0])]) for x in tokens[3:]]
    check_logits(np.concatenate(got), want, "bfloat16")
    check_logits(np.concatenate(got)[-40:], want[-40:], "bfloat16")
    e.close()


def test_wider_layers(lm):
    """Sizes at which the kernels take their other forms: K divided over CTAs, two row tiles, 192-column keys."""
    cfg = t.config(300, 640, [t.layer("mamba1", t.mamba(1280, 16, 40, 4), None),
                              t.layer("latent_attention", t.latent(20, 128, 64, 128, 512, 0.07), t.dense(4300, 1.2)),
                              t.layer("attention", t.attention(16, 2, 128, 64, 0.09, 90), t.dense(300, 3.0))])
    W = t.weights(cfg, 71)
    oracle = bo.Model(cfg, W, np.float32)
    tokens = rng(72).integers(0, 300, 150).tolist()
    want = oracle.forward(tokens, oracle.start()).astype(np.float64)
    for dtype in DTYPES:
        e = make_engine(lm, cfg, W, dtype, step_rows=150)
        for cuts in ([130] + [1] * 20, [30, 100, 20]):
            at, got = 0, []
            for n in cuts:
                got.append(e.step([("r", tokens[at:at + n], list(range(n)))]))
                at += n
            e.end("r")
            assert logit_error(np.concatenate(got), want).max() < (1e-4 if dtype == "float32" else 4e-2)
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
    assert logit_error(np.fromfile(out / "2.f32", "<f4")[None], a[:1].astype(np.float64)).max() < WORST["bfloat16"]
    e.close()
