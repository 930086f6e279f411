"""`bench.py --workload sonalorn` and `--workload bubotar`: throughput of a model's layers at sizes that resemble a real model's
(random weights), and of their kernels one by one, beside the closest other model at equal size: for Sonalorn the Llama int8
decode step and its kernels, for Bubotar Sonalorn's `dense` and its kernels.

Sonalorn models (bf16, 128256 tokens of vocabulary for `dense`, like the Llama step):
    dense  8 layers of width 4096: three delta layers (32 heads on 16 query/key heads, 128 x 128 states, 4 taps) to one
           attention layer (32 heads on 8, 128 wide), feed-forward 14336
    moe    8 layers of width 2048: delta 16 / 8 heads, attention 16 / 4 heads, 64 experts of 1024 and 16 identity experts,
           top 8 of the best 4 of 8 groups
Bubotar model (the same vocabulary and width 4096):
    bubotar  8 layers: scan (8192 channels, 16 states, rank 256, 4 taps) without a feed-forward, latent attention (32 heads of
           128 + 64, values of 128, latents of 512), scan, attention (32 heads on 8, 128 wide, chunks of 4096); then the same,
           the second latent layer with the first one's latents; feed-forward 14336 behind the attention layers
Decoding: batch 1 and 16 behind a context of 2048, one recorded graph per step.  Prompts: 4096 tokens in one step.

Every kernel is timed on its own memory: a graph of enough launches over different weights, states or caches that one
pass exceeds L2 several times over, replayed, CUDA events on the stream.
"""
from __future__ import annotations

import ctypes as C
import json
import os
import time

ROOT = os.path.dirname(os.path.abspath(__file__))


def sonalorn_config(kind: str, layers: int = 8, vocab: int = 128256, max_positions: int = 8192) -> dict:
    if kind == "dense":
        width = 4096
        delta = {"heads": 32, "kv_heads": 16, "dim": 128, "vdim": 128, "conv": 4}
        attn = {"heads": 32, "kv_heads": 8, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "q_temp": {"coef": 0.1, "every": 4096}}
        mlp = {"kind": "dense", "ff": 14336}
    else:
        width, vocab = 2048, 32768
        delta = {"heads": 16, "kv_heads": 8, "dim": 128, "vdim": 128, "conv": 4}
        attn = {"heads": 16, "kv_heads": 4, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "q_temp": {"coef": 0.1, "every": 4096}}
        mlp = {"kind": "moe", "expert": {"ff": 1024, "limit": 7.0}, "router": {"experts": 64, "identity": 16, "top": 8, "groups": {"count": 8, "keep": 4}}}
    return {"architecture": "Sonalorn", "vocab": vocab, "width": width, "max_positions": max_positions, "norm": {"eps": 1e-5},
            "layers": [{"type": "attention" if i % 4 == 3 else "delta", "mixer": attn if i % 4 == 3 else delta, "mlp": mlp} for i in range(layers)]}


def bubotar_config(layers: int = 8, vocab: int = 128256) -> dict:
    latent = {"heads": 32, "dim": 128, "rot_dim": 64, "vdim": 128, "kv_rank": 512, "scale": 192 ** -0.5, "rot": {"base": 10000.0, "dims": 64}}
    attn = {"heads": 32, "kv_heads": 8, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "mask": {"size": 4096}}
    scan = {"inner": 8192, "state": 16, "dt_rank": 256, "conv": 4}
    mlp = {"kind": "dense", "ff": 14336, "limit": 7.0}
    four = [("mamba1", scan, None), ("latent_attention", latent, mlp), ("mamba1", scan, None), ("attention", attn, mlp)]
    out = [{"type": k, "mixer": dict(p), "mlp": m} for i in range(layers) for k, p, m in [four[i % 4]]]
    for i, L in enumerate(out):
        if L["type"] == "latent_attention" and i > 1:
            L["mixer"]["kv_from"] = 1
    return {"architecture": "Bubotar", "vocab": vocab, "width": 4096, "norm": {"eps": 1e-5}, "logit_scale": 1.0, "layers": out}


def bubotar_mixer_shape(kind: str, p: dict, N: int, name: str):
    if kind == "mamba1":
        I, S, R = p["inner"], p["state"], p["dt_rank"]
        return {"in": (2 * I, N), "conv": (I, p["conv"]), "conv.b": (I,), "x": (R + 2 * S, I), "dt": (I, R), "dt.b": (I,), "A_log": (I, S), "D": (I,),
                "o": (N, I)}[name]
    H, D, V = p["heads"], p["dim"], p["vdim"]
    if kind == "attention":
        G = p["kv_heads"]
        return {"q": (H * D, N), "k": (G * D, N), "v": (G * V, N), "o": (N, H * V)}[name]
    K, R = p["kv_rank"], p["rot_dim"]
    return {"q": (H * (D + R), N), "dkv": (K + R, N), "dkv.norm": (K,), "uk": (H * D, K), "uv": (H * V, K), "g": (H * V, N), "o": (N, H * V)}[name]


class RandomWeights:
    """Draws a tensor on the device when the model asks for it."""

    def __init__(self, torch, cfg: dict, dev):
        self.torch, self.cfg, self.dev = torch, cfg, dev
        self.gen = torch.Generator(device=dev)
        self.gen.manual_seed(17)

    def shape(self, name):
        c = self.cfg
        N = c["width"]
        if name in ("embed", "head"):
            return (c["vocab"], N)
        if name == "pos":
            return (c["max_positions"], N)
        if not name.startswith("l"):
            return (N,)
        i, rest = name[1:].split(".", 1)
        L = c["layers"][int(i)]
        p = L["mixer"]
        if rest.startswith("mix."):
            rest = rest[4:]
            if c["architecture"] == "Bubotar":
                return bubotar_mixer_shape(L["type"], p, N, rest)
            G, H, D, V = p["kv_heads"], p["heads"], p["dim"], p["vdim"]
            if L["type"] == "delta":
                return {"q": (G * D, N), "k": (G * D, N), "v": (H * V, N), "g": (H * V, N), "b": (H, N), "a": (H, N), "o": (N, H * V),
                        "q.conv": (G * D, p["conv"]), "k.conv": (G * D, p["conv"]), "v.conv": (H * V, p["conv"]), "A_log": (H,), "dt_bias": (H,), "norm": (V,)}[rest]
            return {"q": (H * D, N), "k": (G * D, N), "v": (G * V, N), "o": (N, H * V), "q.norm": (D,), "k.norm": (D,)}[rest]
        if rest.startswith("mlp."):
            m = L["mlp"]
            F = m["ff"] if m["kind"] == "dense" else m["expert"]["ff"]
            last = rest.split(".")[-1]
            if last in ("router", "correction"):
                n = m["router"]["experts"] + m["router"]["identity"]
                return (n, N) if last == "router" else (n,)
            return {"gate": (F, N), "up": (F, N), "down": (N, F)}[last]
        return (N,)

    def __getitem__(self, name):
        t, s = self.torch, self.shape(name)
        if len(s) == 1:
            if name.endswith("correction"):
                return t.zeros(s, device=self.dev)
            return t.full(s, -2.0 if name.endswith(("A_log", "dt_bias", "dt.b")) else 1.0, device=self.dev)
        return (t.randn(*s, generator=self.gen, device=self.dev, dtype=t.bfloat16) * (1.0 if name in ("embed", "pos") else s[1] ** -0.5)).to(t.bfloat16)


class Timer:
    """Microseconds per call of a list of calls that touch different memory."""

    def __init__(self, gpu, torch):
        self.gpu, self.torch = gpu, torch
        self.stream = torch.cuda.ExternalStream(gpu.stream)

    def __call__(self, calls, reps: int = 20, per: int = 0) -> float:
        for f in calls:
            f()
        self.gpu.sync()
        with self.gpu.record() as g:
            for f in calls:
                f()
        for _ in range(3):
            g.launch()
        e0, e1 = (self.torch.cuda.Event(enable_timing=True) for _ in range(2))
        self.gpu.sync()
        e0.record(self.stream)
        for _ in range(reps):
            g.launch()
        e1.record(self.stream)
        self.gpu.sync()
        us = e0.elapsed_time(e1) * 1e3 / reps / (per or len(calls))
        if self.gpu.device_status():
            raise SystemExit("a kernel reported an error while it was timed")
        g.free()
        return us


def model_figures(torch, gpu, kind: str, hbm: float, tflops: float, layers: int = 8) -> dict:
    from peregrine_b200.bubotar import BubotarModel
    from peregrine_b200.sonalorn import SonalornModel

    Model, cfg = (BubotarModel, bubotar_config(layers)) if kind == "bubotar" else (SonalornModel, sonalorn_config(kind, layers))
    dev = torch.device("cuda", gpu.device)
    ctx0, T, steps = 2048, 4096, 64
    m = Model(Model.Config.from_dict(cfg), RandomWeights(torch, cfg, dev), gpu, slots=16, capacity=T + 128, step_rows=T)
    for L in m.layers:
        for v in L["state"].values():
            v.normal_()
    torch.cuda.synchronize()
    stream = torch.cuda.ExternalStream(gpu.stream)
    out = {"layers": layers, "width": cfg["width"], "vocab": cfg["vocab"], "prompt_tokens": T, "context": ctx0}
    # prompts: one step of T tokens from host ids, greedy choice read back
    ids = torch.randint(0, cfg["vocab"], (T,)).tolist()
    for _ in range(3):
        m.run_greedy([(0, 0, ids)], [T - 1])
    ms = []
    for _ in range(5):
        t0 = time.perf_counter()
        m.run_greedy([(0, 0, ids)], [T - 1])
        ms.append((time.perf_counter() - t0) * 1e3)
    ms.sort()
    flops = 0.0
    for L in m.layers:
        mx, f = L["mixer"], L["ff"]
        flops += 2.0 * T * (mx.proj.n * mx.proj.k + mx.out.n * mx.out.k)
        if hasattr(mx, "dp"):
            flops += 2.0 * T * T / 2 * mx.H * (mx.D + mx.V)
        if hasattr(mx, "unfold"):
            flops += 2.0 * T * T / 2 * mx.H * (mx.D + mx.R + mx.V) + 2.0 * T * mx.unfold.n * mx.unfold.k
        if hasattr(mx, "dtp"):
            flops += 2.0 * T * (mx.low.n * mx.low.k + mx.dt.n * mx.dt.k)
        if f is None:
            pass
        elif hasattr(f, "route"):
            flops += 2.0 * T * f.top * f.E / (f.E + f.I) * (f.gate_up.n * f.gate_up.k + f.down.n * f.down.k)
        else:
            flops += 2.0 * T * (f.gate_up.n * f.gate_up.k + f.down.n * f.down.k)
    out["prompt"] = {"e2e_ms": ms[2], "e2e_tok_s": T / ms[2] * 1e3, "tflops": flops / ms[2] * 1e-9, "frac_of_bf16_peak": flops / ms[2] * 1e-9 / tflops}
    for B in (1, 16):
        d = m.decoder(B)
        entries = [(s, ctx0, 5 + s) for s in range(B)]
        d.load(entries)
        d.enqueue()
        gpu.sync()
        d.load(entries)
        for _ in range(4):
            d.run()
        gpu.sync()
        d.load(entries)
        e0, e1 = (torch.cuda.Event(enable_timing=True) for _ in range(2))
        gpu.sync()
        e0.record(stream)
        for _ in range(steps):
            d.run()
        e1.record(stream)
        gpu.sync()
        us = e0.elapsed_time(e1) * 1e3 / steps
        d.load(entries)
        gpu.sync()
        t0 = time.perf_counter()
        for _ in range(steps):
            d.run()
            d.tokens()
        e2e = (time.perf_counter() - t0) / steps
        kv = sum(B * mx.G * (ctx0 + steps / 2) * (mx.dp + mx.vp) * 2 for mx in (L["mixer"] for L in m.layers) if hasattr(mx, "dp"))
        kv += sum(B * (ctx0 + steps / 2) * mx.ck * 2 for mx in (L["mixer"] for L in m.layers) if hasattr(mx, "ck"))
        st = sum(2 * B * L["state"]["state"][0].numel() * 4 for L in m.layers if "state" in L["state"])
        moe_rows = 0.0
        nbytes = kv + st + m.head.bytes()
        for L in m.layers:
            mx, f = L["mixer"], L["ff"]
            nbytes += mx.bytes()
            if f is None:
                continue
            if hasattr(f, "route"):
                used = len(set(f.chosen(B)[0].ravel().tolist()) & set(range(f.E)))
                moe_rows += used
                nbytes += f.router.bytes() + (f.gate_up.bytes() + f.down.bytes()) * used / f.E
            else:
                nbytes += f.gate_up.bytes() + f.down.bytes()
        out[f"decode_b{B}"] = {"us_per_step": us, "tok_s": B / us * 1e6, "e2e_tok_s": B / e2e, "kernels_per_step": d.graph.kernels, "bytes": nbytes,
                               "hbm_gbs": nbytes / us * 1e-3, "frac_of_hbm": nbytes / us * 1e-3 / hbm}
        if moe_rows:
            out[f"decode_b{B}"]["experts_read_per_layer"] = moe_rows / layers
        d.free()
    m.free()
    return out


def kernel_figures(torch, gpu, hbm: float, tflops: float) -> dict:
    """New kernels at the sizes of `dense` and `moe`."""
    from peregrine_b200 import _lib
    from peregrine_b200.layers import Attention, Batch, Device, GatedDelta, Linear, MoeFF
    from peregrine_b200.state import SlotPool

    dev = torch.device("cuda", gpu.device)
    time_us = Timer(gpu, torch)
    T = 4096
    d = Device(gpu, "bfloat16", T)
    out = {}

    def note(name, us, nbytes=None, flops=None):
        e = out[name] = {"us": us}
        if nbytes:
            e.update(gbs=nbytes / us * 1e-3, frac_of_hbm=nbytes / us * 1e-3 / hbm)
        if flops:
            e.update(tflops=flops / us * 1e-6, frac_of_bf16_peak=flops / us * 1e-6 / tflops)

    rnd = lambda *s: torch.randn(*s, device=dev, dtype=torch.bfloat16) * s[-1] ** -0.5

    def linears(n, k, gated=False):
        copies = max(2, int(400e6 / (n * k * 2)) + 1)
        return [Linear(d, (rnd(n // 2, k), rnd(n // 2, k)) if gated else rnd(n, k), gated=gated) for _ in range(copies)]

    for name, n, k, gated in (("delta_proj", 12352, 4096, False), ("attn_proj", 6144, 4096, False), ("o", 4096, 4096, False), ("gate_up", 28672, 4096, True),
                              ("down", 4096, 14336, False)):
        ls = linears(n, k, gated)
        for M in (1, 16, 64, T):
            a = torch.randn(M, k, device=dev).to(torch.bfloat16)
            y = torch.zeros(M, n // 2 if gated else n, device=dev, dtype=torch.bfloat16 if gated else torch.float32)
            torch.cuda.synchronize()
            act = _lib.ACT_GELU_TANH_GLU if gated else _lib.ACT_NONE
            us = time_us([(lambda l=l: l.run(a, M, y, act)) for l in (ls if M <= 64 else ls[:2])], reps=10)
            if M <= 64:
                note(f"product.{name}.m{M}", us, nbytes=n * k * 2 + M * k * 2 + y.numel() * y.element_size())
            else:
                note(f"product.{name}.m{M}", us, flops=2.0 * M * n * k)
        for l in ls:
            l.free()
        del ls

    dense, sparse = sonalorn_config("dense"), sonalorn_config("moe")
    W = RandomWeights(torch, dense, dev)

    class Sub:
        def __init__(self, W, prefix):
            self.W, self.p = W, prefix

        def __getitem__(self, n):
            return self.W[self.p + n]

    # decode: states and caches of sixteen sequences, several layers' worth
    x = torch.randn(T, 4096, device=dev).to(torch.bfloat16)
    for B in (1, 16):
        batch = Batch(d, [(s, 2048, [1]) for s in range(B)], fixed=True)
        mx = GatedDelta(d, dense["layers"][0]["mixer"], Sub(W, "l0.mix."), 4096, 1e-5)
        pool = SlotPool(16, 2304, dev)
        states = [mx.new_state(pool) for _ in range(10)]
        proj = torch.randn(T, mx.proj.n, device=dev)
        mixed = d.buffer("mixed", mx.out.k)
        torch.cuda.synchronize()

        def delta(state, b):
            mx.c.d_work = d.buffer("delta.work", 1, 1, torch.float32).data_ptr()
            d.check(d.lib.pg_delta_run(gpu.handle, C.byref(mx.c), C.byref(b.c), proj.data_ptr(), proj.stride(0), state["ring"].data_ptr(),
                                       state["state"].data_ptr(), mixed.data_ptr(), d.code, mixed.stride(0)))
        note(f"delta.step.b{B}", time_us([(lambda s=s: delta(s, batch)) for s in states]), nbytes=B * 2 * 32 * 128 * 128 * 4)
        if B == 16:
            long = Batch(d, [(0, 0, [1] * T)], fixed=True)
            us = time_us([(lambda s=s: delta(s, long)) for s in states[:2]], reps=5)
            note(f"delta.prompt.t{T}", us, nbytes=T * (mx.channels * 3 + 32 * 128 * 4) * 4)
        mx.free()
        del states
        att = Attention(d, dense["layers"][3]["mixer"], Sub(W, "l3.mix."), 4096, 1e-5, 2304, 16)
        states = [att.new_state(pool) for _ in range(6)]
        for s in states:
            s["k"].normal_()
            s["v"].normal_()
        torch.cuda.synchronize()

        def attend(a, state, b):
            a.c.d_q = d.buffer("attn.q", a.H * a.dp).data_ptr()
            a.c.d_part = d.buffer("attn.part", 1, 1, torch.float32).data_ptr()
            a.c.d_tickets = d.buffer("attn.tickets", 1, 1, torch.int32).data_ptr()
            a.c.slots = state["k"].shape[0]
            d.check(d.lib.pg_attention_run(gpu.handle, C.byref(a.c), C.byref(b.c), proj.data_ptr(), proj.stride(0), state["k"].data_ptr(), state["v"].data_ptr(),
                                           mixed.data_ptr(), d.code, mixed.stride(0)))
        note(f"attention.step.b{B}", time_us([(lambda s=s: attend(att, s, batch)) for s in states]), nbytes=B * 8 * 2049 * 256 * 2)
        att.free()
        if B == 16:
            att = Attention(d, dense["layers"][3]["mixer"], Sub(W, "l3.mix."), 4096, 1e-5, T, 1)
            st = att.new_state(SlotPool(1, T, dev))
            torch.cuda.synchronize()
            note(f"attention.prompt.t{T}", time_us([lambda: attend(att, st, long)] * 2, reps=5), flops=4.0 * T * T / 2 * 32 * 128)
            att.free()
    # residual rows
    xs = torch.randn(T, 4096, device=dev)
    y = torch.randn(T, 4096, device=dev)
    one = torch.ones(4096, device=dev)
    h = torch.zeros(T, 4096, device=dev, dtype=torch.bfloat16)
    torch.cuda.synchronize()
    for M in (1, 16, T):
        f = lambda: d.check(d.lib.pg_norm_add(gpu.handle, y.data_ptr(), 4096, xs.data_ptr(), one.data_ptr(), one.data_ptr(), M, 4096, 1e-5, h.data_ptr(), d.code, 4096))
        note(f"norm_add.m{M}", time_us([f] * 8), nbytes=M * 4096 * 14)
    # experts
    W = RandomWeights(torch, sparse, dev)
    ff = [MoeFF(d, sparse["layers"][0]["mlp"], Sub(W, "l0.mlp."), 2048) for _ in range(3)]
    xs, hh = torch.randn(T, 2048, device=dev), torch.zeros(T, 2048, device=dev, dtype=torch.bfloat16)
    x = torch.randn(T, 2048, device=dev).to(torch.bfloat16)
    torch.cuda.synchronize()
    for M in (1, 16, T):
        class Rows:
            rows = M

        def add(o, route=None):
            d.check(d.lib.pg_routed_norm_add(gpu.handle, route, o.data_ptr(), o.stride(0), xs.data_ptr(), one.data_ptr(), one.data_ptr(), M, 2048, 1e-5, hh.data_ptr(),
                                             d.code, 2048))
        us = time_us([(lambda f=f: f.run(Rows, x, None, add)) for f in ff], reps=5)
        ids, _w = ff[0].chosen(M)
        real = ids < ff[0].E
        if M <= 16:
            note(f"experts.m{M}", us, nbytes=len(set(ids[real].tolist())) * 3 * 2048 * 1024 * 2)
        else:
            note(f"experts.m{M}", us, flops=2.0 * real.sum() * 3 * 2048 * 1024)
        if M <= 16:
            act = d.buffer("expert.act", ff[0].down.k, ff[0].max_rows)
            o = d.buffer("expert.out", 2048, ff[0].max_rows)
            used = len(set(ids[real].tolist()))
            us = time_us([(lambda f=f: f.gate_up.run_routed(f.route, x, True, act, _lib.ACT_CLAMPED_SWISH_GLU, 7.0)) for f in ff])
            note(f"experts.gate_up.m{M}", us, nbytes=used * 2 * 2048 * 1024 * 2)
            us = time_us([(lambda f=f: f.down.run_routed(f.route, act, False, o)) for f in ff])
            note(f"experts.down.m{M}", us, nbytes=used * 2048 * 1024 * 2)
    for f in ff:
        f.free()
    return out


def bubotar_kernel_figures(torch, gpu, hbm: float, tflops: float) -> dict:
    """The kernels of Bubotar's layers at the sizes of `bubotar`."""
    from peregrine_b200 import _lib
    from peregrine_b200.layers import Attention, Batch, Device, LatentAttention, Linear, SelectiveScan, halving_slopes
    from peregrine_b200.slot_model import Below
    from peregrine_b200.state import SlotPool

    dev = torch.device("cuda", gpu.device)
    time_us = Timer(gpu, torch)
    T, N, ctx0 = 4096, 4096, 2048
    d = Device(gpu, "bfloat16", T)
    out = {}

    def note(name, us, nbytes=None, flops=None):
        e = out[name] = {"us": us}
        if nbytes:
            e.update(gbs=nbytes / us * 1e-3, frac_of_hbm=nbytes / us * 1e-3 / hbm)
        if flops:
            e.update(tflops=flops / us * 1e-6, frac_of_bf16_peak=flops / us * 1e-6 / tflops)

    rnd = lambda *s: torch.randn(*s, device=dev, dtype=torch.bfloat16) * s[-1] ** -0.5
    for name, n, k, gated in (("scan_in", 16384, N, False), ("scan_low", 288, 8192, False), ("scan_low_dt", 256, 8192, False), ("scan_low_bc", 32, 8192, False), ("scan_dt", 8192, 256, False), ("latent_proj", 10816, N, False),
                              ("latent_unfold", 8192, 512, False), ("o", N, 4096, False), ("scan_o", N, 8192, False), ("gate_up", 28672, N, True),
                              ("down", N, 14336, False)):
        ls = [Linear(d, (rnd(n // 2, k), rnd(n // 2, k)) if gated else rnd(n, k), gated=gated) for _ in range(min(80, max(2, int(400e6 / (n * k * 2)) + 1)))]
        # (decoding takes the low-rank product whole, prompts in its two parts)
        for M in {"scan_low": (1, 16), "scan_low_dt": (64, T), "scan_low_bc": (64, T), "scan_dt": (64, T), "latent_unfold": (T,)}.get(name, (1, 16, 64, T)):
            a = torch.randn(M, k, device=dev).to(torch.bfloat16)
            narrow = gated or name in ("latent_unfold", "scan_low_dt")
            y = torch.zeros(M, n // 2 if gated else n, device=dev, dtype=torch.bfloat16 if narrow else torch.float32)
            torch.cuda.synchronize()
            act = _lib.ACT_CLAMPED_SWISH_GLU if gated else _lib.ACT_NONE
            us = time_us([(lambda l=l: l.run(a, M, y, act, 7.0)) for l in (ls if M <= 64 else ls[:2])], reps=10)
            note(f"product.{name}.m{M}", us, nbytes=(n * k + M * k) * 2 + y.numel() * y.element_size(), flops=2.0 * M * n * k if M > 64 else None)
        for l in ls:
            l.free()
        del ls

    cfg = bubotar_config()
    W = RandomWeights(torch, cfg, dev)
    cap = T + 64
    pool = SlotPool(16, cap, dev)
    steps = {B: Batch(d, [(s, ctx0, [1]) for s in range(B)], fixed=True) for B in (1, 16)}
    long = Batch(d, [(0, 0, [1] * T)], fixed=True)
    part = Batch(d, [(0, ctx0, [1] * 16)], fixed=True)
    ptr = lambda t: t.data_ptr()
    f32 = torch.float32

    # scan
    mx = [SelectiveScan(d, cfg["layers"][0]["mixer"], Below(W, "l0.mix."), N) for _ in range(16)]
    states = [m.new_state(pool) for m in mx]
    proj, mixed = torch.randn(T, mx[0].proj.n, device=dev), d.buffer("mixed", mx[0].out.k)
    x, low = d.buffer("scan.x", mx[0].low.k), d.buffer("scan.low", mx[0].low.n, dtype=f32)
    dt, bc = d.buffer("scan.dt", mx[0].I, dtype=f32), d.buffer("scan.bc", mx[0].low_bc.n, dtype=f32)
    for v in (low, dt, bc, x):
        v.normal_()
    torch.cuda.synchronize()
    ck, lib, gh, I, S = d.check, d.lib, gpu.handle, mx[0].I, mx[0].ss

    def conv(m, s, b):
        ck(lib.pg_scan_conv(gh, C.byref(m.c), C.byref(b.c), ptr(proj), proj.stride(0), ptr(s["ring"]), ptr(x), d.code, x.stride(0)))

    def step(m, s, b):
        ck(lib.pg_scan_step(gh, C.byref(m.c), C.byref(b.c), ptr(proj), proj.stride(0), ptr(x), x.stride(0), ptr(low), low.stride(0), ptr(s["state"]), ptr(mixed),
                            d.code, mixed.stride(0)))

    def scan(m, s, b):
        ck(lib.pg_scan_run(gh, C.byref(m.c), C.byref(b.c), ptr(proj), proj.stride(0), ptr(s["ring"]), ptr(x), x.stride(0), ptr(dt), dt.stride(0), ptr(bc),
                           bc.stride(0), ptr(s["state"]), ptr(mixed), d.code, mixed.stride(0)))
    pairs = list(zip(mx, states))
    for B, b in steps.items():
        note(f"scan.conv.b{B}", time_us([(lambda m=m, s=s: conv(m, s, b)) for m, s in pairs]), nbytes=B * I * (4 * 4 + 4 + 2))
        note(f"scan.step.b{B}", time_us([(lambda m=m, s=s: step(m, s, b)) for m, s in pairs]), nbytes=B * I * (2 * S * 4 + 8) + I * (256 * 2 + S * 4))
    note(f"scan.conv.t{T}", time_us([(lambda m=m, s=s: conv(m, s, long)) for m, s in pairs[:2]], reps=5), nbytes=T * I * 6)
    # an exponential per channel, state and token, on a unit of 16 per SM and clock, bounds the recurrence
    us = time_us([(lambda m=m, s=s: scan(m, s, long)) for m, s in pairs[:2]], reps=5)
    note(f"scan.run.t{T}", us, nbytes=T * I * (4 + 2 + 4 + 2))
    out[f"scan.run.t{T}"]["frac_of_exponentials_at_1965_mhz"] = T * I * S / (148 * 16 * 1965.0) / us
    for m in mx:
        m.free()
    del mx, states, pairs, proj
    # latent attention
    mx = [LatentAttention(d, cfg["layers"][1]["mixer"], Below(W, "l1.mix."), N, 1e-5, cap, 16) for _ in range(6)]
    states = [m.new_state(pool) for m in mx]
    for s in states:
        s["latent"].normal_()
    m0 = mx[0]
    proj, mixed = torch.randn(T, m0.proj.n, device=dev), d.buffer("mixed", m0.out.k)
    for m in mx:
        m.c.d_q, m.c.d_part, m.c.part_floats, m.c.slots = ptr(d.buffer("latent.q", m.H * m.qd)), ptr(d.buffer("latent.part", 1, 1, f32)), m.part_rows, 16
    kv = d.buffer("latent.kv", m0.unfold.n, cap)
    torch.cuda.synchronize()

    def short(m, s, b, n, longest):
        ck(lib.pg_latent_run(gh, C.byref(m.c), C.byref(b.c), m.LONG, n, longest, ptr(proj), proj.stride(0), ptr(s["latent"]), ptr(mixed), d.code, mixed.stride(0)))

    def prep(m, s):
        ck(lib.pg_latent_prompt_prep(gh, C.byref(m.c), C.byref(long.c), 0, T, 0, ptr(proj), proj.stride(0), ptr(s["latent"])))

    def attend(m, s):
        ck(lib.pg_latent_prompt(gh, C.byref(m.c), C.byref(long.c), 0, T, T, 0, ptr(proj), proj.stride(0), ptr(s["latent"]), ptr(kv), kv.stride(0), ptr(mixed),
                                mixed.stride(0)))

    def whole(m, s):
        prep(m, s)
        m.unfold.run_ld(ptr(s["latent"][0]), m.ck, T, kv)
        attend(m, s)
    pairs = list(zip(mx, states))
    wb = 2 * m0.H * 128 * 512 * 2
    for B, b in steps.items():
        note(f"latent.step.b{B}", time_us([(lambda m=m, s=s: short(m, s, b, B, 1)) for m, s in pairs]), nbytes=B * (ctx0 + 1) * m0.ck * 2 + wb,
             flops=2.0 * B * m0.H * ((ctx0 + 1) * (m0.ck + 512) + 2 * 128 * 512))
    note("latent.portion.t16", time_us([(lambda m=m, s=s: short(m, s, part, 16, 16)) for m, s in pairs]), nbytes=(ctx0 + 16) * m0.ck * 2 + wb,
         flops=2.0 * 16 * m0.H * ((ctx0 + 8) * (m0.ck + 512) + 2 * 128 * 512))
    fl = 2.0 * T * T / 2 * m0.H * (m0.D + m0.R + m0.V)
    note(f"latent.prompt.prep.t{T}", time_us([(lambda m=m, s=s: prep(m, s)) for m, s in pairs[:2]], reps=5), nbytes=T * (m0.H * 192 * 6 + 576 * 6))
    note(f"latent.prompt.attend.t{T}", time_us([(lambda m=m, s=s: attend(m, s)) for m, s in pairs[:2]], reps=5), flops=fl)
    note(f"latent.prompt.t{T}", time_us([(lambda m=m, s=s: whole(m, s)) for m, s in pairs[:2]], reps=5), flops=fl + 2.0 * T * 8192 * 512)
    for m in mx:
        m.free()
    del mx, states, pairs, proj
    # chunked attention
    proj = torch.randn(T, 6144, device=dev)
    for size in (4096, 1024):
        p = dict(cfg["layers"][3]["mixer"], mask={"size": size})
        att = Attention(d, p, Below(W, "l3.mix."), N, 1e-5, cap, 16, sink=False, norms=False, slopes=halving_slopes(32), chunk=size)
        states = [att.new_state(pool) for _ in range(4)]
        for s in states:
            s["k"].normal_(), s["v"].normal_()
        mixed = d.buffer("mixed", att.out.k)
        att.c.d_q, att.c.d_part = ptr(d.buffer("attn.q", att.H * att.dp)), ptr(d.buffer("attn.part", 1, 1, f32))
        att.c.d_tickets, att.c.slots = ptr(d.buffer("attn.tickets", 1, 1, torch.int32)), 16
        torch.cuda.synchronize()

        def run(s, b):
            ck(lib.pg_attention_run(gh, C.byref(att.c), C.byref(b.c), ptr(proj), proj.stride(0), ptr(s["k"]), ptr(s["v"]), ptr(mixed), d.code, mixed.stride(0)))
        if size > ctx0:
            for B, b in steps.items():
                note(f"attention.chunk{size}.step.b{B}", time_us([(lambda s=s: run(s, b)) for s in states]), nbytes=B * 8 * (ctx0 + 1) * 256 * 2)
        note(f"attention.chunk{size}.prompt.t{T}", time_us([(lambda s=s: run(s, long)) for s in states[:2]], reps=5), flops=4.0 * T * size / 2 * 32 * 128)
        att.free()
        del states
    xs, y, one = torch.randn(T, N, device=dev), torch.randn(T, N, device=dev), torch.ones(N, device=dev)
    h = torch.zeros(T, N, device=dev, dtype=torch.bfloat16)
    torch.cuda.synchronize()
    for M in (1, 16, T):
        f = lambda: ck(lib.pg_norm_add_prenorm(gh, ptr(y), N, ptr(xs), ptr(one), ptr(one), M, N, 1e-5, ptr(h), d.code, N))
        note(f"norm_add_prenorm.m{M}", time_us([f] * 8), nbytes=M * N * 14)
    return out


def llama_kernel_figures(torch, hbm: float, tflops: float) -> dict:
    """The like kernels of the Llama int8 path at equal size."""
    from peregrine_b200 import _lib
    from peregrine_b200.runtime import GpuContext

    gpu = GpuContext()
    lib, dev = gpu.lib, torch.device("cuda", gpu.device)
    time_us = Timer(gpu, torch)
    out = {}
    ck = _lib.check
    for name, n, k in (("qkv", 6144, 4096), ("o", 4096, 4096), ("gate_up", 28672, 4096), ("down", 4096, 14336)):
        hs = []
        for _ in range(max(2, int(400e6 / (n * k)) + 1)):
            w = torch.randn(k, n, device=dev) * 0.02
            torch.cuda.synchronize()
            h = C.c_void_p()
            ck(lib.pg_qtensor_from_f32(gpu.handle, w.data_ptr(), k, n, 0, C.byref(h)))
            gpu.sync()
            hs.append(h)
        for M in (1, 16, 64, 4096):
            q = torch.randint(-127, 127, (M, k), device=dev, dtype=torch.int8)
            s = torch.ones(M, device=dev)
            y = torch.zeros(M, n, device=dev)
            torch.cuda.synchronize()
            us = time_us([(lambda h=h: ck(lib.pg_gemm_i8(gpu.handle, q.data_ptr(), s.data_ptr(), M, k, h, y.data_ptr(), None, _lib.ALGO_AUTO))) for h in (hs if M <= 64 else hs[:2])], reps=10)
            b = n * k + M * k + M * n * 4
            out[f"product.{name}.m{M}"] = {"us": us, "gbs": b / us * 1e-3, "frac_of_hbm": b / us * 1e-3 / hbm} if M <= 64 else \
                {"us": us, "tops": 2.0 * M * n * k / us * 1e-6, "frac_of_twice_bf16_peak": 2.0 * M * n * k / us * 1e-6 / (2 * tflops)}
        for h in hs:
            lib.pg_qtensor_free(gpu.handle, h)
    for B in (1, 16):
        cap = 2304
        pos = torch.full((1,), 2048, dtype=torch.int32, device=dev)
        cos, sin = torch.ones(cap, 64, device=dev), torch.zeros(cap, 64, device=dev)
        qkv = torch.randn(B, 48 * 128, device=dev)
        kv = [(torch.randn(B, 8, cap, 128, device=dev), torch.randn(B, 8, cap, 128, device=dev)) for _ in range(4)]
        work = torch.zeros(B * 32 * 64 * 130, device=dev)
        q8, q8s = torch.zeros(B * 4096 + 64, dtype=torch.int8, device=dev), torch.zeros(B, device=dev)
        torch.cuda.synchronize()
        us = time_us([(lambda k=k, v=v: ck(lib.pg_gqa_attention_decode_fused(gpu.handle, qkv.data_ptr(), pos.data_ptr(), cos.data_ptr(), sin.data_ptr(), k.data_ptr(),
                                                                             v.data_ptr(), B, 32, 8, 128, cap, work.data_ptr(), None, q8.data_ptr(), q8s.data_ptr())))
                      for k, v in kv])
        b = B * 8 * 2049 * 256 * 4
        out[f"attention.step.b{B}"] = {"us": us, "gbs": b / us * 1e-3, "frac_of_hbm": b / us * 1e-3 / hbm}
    x, y, w = torch.randn(16, 4096, device=dev), torch.randn(16, 4096, device=dev), torch.ones(4096, device=dev)
    q8, q8s = torch.zeros(16 * 4096 + 64, dtype=torch.int8, device=dev), torch.zeros(16, device=dev)
    torch.cuda.synchronize()
    for M in (1, 16):
        us = time_us([lambda: ck(lib.pg_add_rmsnorm_quantize(gpu.handle, x.data_ptr(), y.data_ptr(), w.data_ptr(), M, 4096, 1e-5, q8.data_ptr(), q8s.data_ptr(), None))] * 8)
        out[f"norm_add.m{M}"] = {"us": us}
    gpu.close()
    return out


def run(args, result_out, clocks) -> None:
    """clocks: class of the sampler that bench.py uses."""
    import torch

    from peregrine_b200.runtime import GpuContext

    peaks = {}
    try:
        with open(os.path.join(ROOT, "MEASURED_PEAKS.json")) as f:
            peaks = json.load(f)
    except (OSError, ValueError):
        pass
    hbm, tflops = float(peaks.get("hbm_gbs", 6650.0)), float(peaks.get("bf16_tflops", 1590.0))
    out = {"workload": args.workload, "data": "synthetic", "dtype": "bf16", "peaks": {"hbm_gbs": hbm, "bf16_tflops": tflops, "source": "measured" if peaks else "fallback"}}
    gpu = GpuContext(component="lm")
    sampler = clocks(gpu.device)
    sampler.mark()
    usual = ["bubotar", "bubotar_kernels", "dense", "kernels"] if args.workload == "bubotar" else ["dense", "moe", "kernels", "llama"]
    parts = args.parts.split(",") if args.parts else usual
    if "bubotar_kernels" in parts:
        out["bubotar_kernels"] = bubotar_kernel_figures(torch, gpu, hbm, tflops)
        torch.cuda.empty_cache()
    for kind in ("bubotar", "dense", "moe"):
        if kind in parts:
            out[kind] = model_figures(torch, gpu, kind, hbm, tflops)
            torch.cuda.empty_cache()
    if "kernels" in parts:
        out["kernels"] = kernel_figures(torch, gpu, hbm, tflops)
        torch.cuda.empty_cache()
    if "llama" in parts:
        out["llama_kernels"] = llama_kernel_figures(torch, hbm, tflops)
        import bench

        g8 = GpuContext()
        out["llama_8_layers"] = bench.llama_decode_measurement(g8, torch, torch.cuda.ExternalStream(g8.stream), torch.device("cuda", g8.device), hbm, steps=64, layers=8)
    out["clocks"] = sampler.stop(time.time())
    print(json.dumps(out), file=result_out, flush=True)
