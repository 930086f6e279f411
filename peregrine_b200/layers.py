"""The layer mechanisms of the bf16 / f32 language models: device weights and state of each, and its calls into
libperegrine_b200_lm.  A model puts a list of them together (peregrine_b200/sonalorn.py); constants are parameters.

    Linear        y = a W^T, plain or gated, one matrix or one per expert
    GatedDelta    gated delta rule with short convolutions (recurrent state)
    SelectiveScan selective scan with a short convolution (recurrent state)
    Attention     per-head norms, query temperature, softmax sink, distance bias, chunks (key / value cache)
    LatentAttention  keys and values from a latent per position, rotated key part (latent cache, which layers may share)
    DenseFF       gated feed-forward, clamped or not
    MoeFF         router with corrected, grouped choice and identity experts; clamped gated experts

torch holds device memory and lays weights out at load time; every computation of a step is a kernel of the library.
"""
from __future__ import annotations

import ctypes as C
from typing import Optional

import numpy as np

from . import _lib


def up(v: int, to: int) -> int:
    return (v + to - 1) // to * to


class Device:
    """The context, the step's type and the buffers that the layers of one model share.

    Activation buffers are kept per width, zero behind the true width: products read K rounded up to 64."""

    def __init__(self, gpu, dtype: str, step_rows: int):
        import torch

        if dtype not in ("bfloat16", "float32"):
            raise ValueError(f"dtype {dtype!r}: bfloat16 or float32")
        self.torch, self.gpu, self.lib = torch, gpu, gpu.lib
        self.dev = torch.device("cuda", gpu.device)
        self.code = _lib.BF16 if dtype == "bfloat16" else _lib.F32
        self.act = torch.bfloat16 if dtype == "bfloat16" else torch.float32
        self.rows = int(step_rows)
        self._buffers = {}

    def f32(self, a):
        """Host array (f32, or bf16 bits as uint16) or torch tensor -> f32 on the device."""
        if isinstance(a, self.torch.Tensor):
            return a.to(self.dev).float().contiguous()
        return self.bf16(a).float().contiguous() if a.dtype == np.uint16 else self.torch.from_numpy(np.array(a, np.float32)).to(self.dev)

    def bf16(self, a):
        """Host array (bf16 bits as uint16, or f32) or torch tensor -> bf16 on the device."""
        t = self.torch
        if isinstance(a, t.Tensor):
            return a.to(self.dev).to(t.bfloat16)
        if a.dtype == np.uint16:
            return t.from_numpy(np.array(a).view(np.int16)).to(self.dev).view(t.bfloat16)
        return t.from_numpy(np.array(a, np.float32)).to(self.dev).to(t.bfloat16)

    def buffer(self, name: str, cols: int, rows: int = 0, dtype=None):
        """[rows, cols] zeroed; the same (name, cols) is the same memory."""
        rows, dtype = rows or self.rows, dtype or self.act
        key = (name, cols, dtype)
        t = self._buffers.get(key)
        if t is None or t.shape[0] < rows:
            t = self._buffers[key] = self.torch.zeros(rows, cols, dtype=dtype, device=self.dev)
        return t

    def rotation(self, base: float, dims: int, positions: int):
        """[positions, dims / 2, 2] f32: cosine and sine of p * base^(-2 i / dims); angles are computed in 64 bits."""
        key = ("rotation", float(base), int(dims), int(positions))
        if key not in self._buffers:
            a = np.arange(positions, dtype=np.float64)[:, None] * float(base) ** (-2.0 * np.arange(dims // 2) / dims)
            self._buffers[key] = self.f32(np.stack([np.cos(a), np.sin(a)], axis=-1))
        return self._buffers[key]

    def check(self, code: int) -> None:
        _lib.check(code, self.lib)


def expect(what: str, W, shapes: dict) -> None:
    """The tensors of a mixer or feed-forward have the shapes that the configuration says."""
    for name, shape in shapes.items():
        if tuple(W[name].shape) != tuple(shape):
            raise ValueError(f"{what}: {name} is {list(W[name].shape)}, the configuration says {list(shape)}")


class Linear:
    """w: bf16 [N, K] or [experts, N, K] on the device; K is padded to 64 with zero columns.  `gated`: w is the pair
    (gate, up), whose rows are laid out in alternating blocks of eight; F is then padded to 8 with zero rows."""

    def __init__(self, d: Device, w, gated: bool = False):
        t = d.torch
        self.d = d
        if gated:
            gate, upw = (x if x.dim() == 3 else x[None] for x in w)
            E, F, K = gate.shape
            both = t.zeros(E, up(F, 8), 2, up(K, 64), dtype=t.bfloat16, device=d.dev)
            both[:, :F, 0, :K], both[:, :F, 1, :K] = gate, upw
            w = both.view(E, -1, 8, 2, both.shape[-1]).transpose(2, 3).reshape(E, 2 * up(F, 8), -1).contiguous()
            self.cols = up(F, 8)
        else:
            w = w if w.dim() == 3 else w[None]
            E, N, K = w.shape
            if K % 64:
                w = t.nn.functional.pad(w, (0, up(K, 64) - K))
            w = w.contiguous()
            self.cols = N
        self.w = w
        self.experts, self.n, self.k = w.shape
        h = C.c_void_p()
        d.check(d.lib.pg_linear_wrap(d.gpu.handle, w.data_ptr(), self.n, self.k, self.experts, C.byref(h)))
        self.handle = h

    def run(self, a, rows: int, y, act: int = _lib.ACT_NONE, limit: float = 0.0) -> None:
        d = self.d
        d.check(d.lib.pg_linear_run(d.gpu.handle, self.handle, a.data_ptr(), d.code, rows, act, limit, y.data_ptr(),
                                    _lib.F32 if y.dtype == d.torch.float32 else _lib.BF16, y.stride(0)))

    def run_ld(self, a_ptr: int, lda: int, rows: int, y) -> None:
        """Rows of a at the device address a_ptr, lda elements apart."""
        d = self.d
        d.check(d.lib.pg_linear_run_ld(d.gpu.handle, self.handle, a_ptr, lda, d.code, rows, _lib.ACT_NONE, 0.0, y.data_ptr(),
                                       _lib.F32 if y.dtype == d.torch.float32 else _lib.BF16, y.stride(0)))

    def run_routed(self, route, a, by_token: bool, y, act: int = _lib.ACT_NONE, limit: float = 0.0) -> None:
        d = self.d
        d.check(d.lib.pg_linear_run_routed(d.gpu.handle, self.handle, route, a.data_ptr(), d.code, int(by_token), act, limit, y.data_ptr(),
                                           _lib.F32 if y.dtype == d.torch.float32 else _lib.BF16, y.stride(0)))

    def free(self) -> None:
        if self.handle is not None:
            self.d.lib.pg_linear_free(self.d.gpu.handle, self.handle)
            self.handle = None

    def bytes(self) -> int:
        return self.w.numel() * 2


def stack_rows(d: Device, parts, multiple: int = 4):
    """Matrices that read the same input as one, rows padded with zeros to `multiple`."""
    t = d.torch
    w = t.cat(parts, dim=0)
    return t.nn.functional.pad(w, (0, 0, 0, up(w.shape[0], multiple) - w.shape[0]))


# ---- mixers: weights are shared by layers that name another layer's; state is per layer ---------------------------
class GatedDelta:
    """p: heads, kv_heads, dim, vdim, conv (taps).  W: name -> host array, the tensors of one mixer."""

    UNIT_EPS = 1e-6

    def __init__(self, d: Device, p: dict, W, width: int, eps: float):
        self.d, self.p, self.eps = d, p, float(eps)
        H, G, D, V, taps = (int(p[k]) for k in ("heads", "kv_heads", "dim", "vdim", "conv"))
        self.H, self.G, self.D, self.V, self.taps = H, G, D, V, taps
        self.channels = 2 * G * D + H * V
        expect("delta mixer", W, {"q": (G * D, width), "k": (G * D, width), "v": (H * V, width), "g": (H * V, width), "b": (H, width), "a": (H, width),
                                  "o": (width, H * V), "q.conv": (G * D, taps), "k.conv": (G * D, taps), "v.conv": (H * V, taps), "A_log": (H,), "dt_bias": (H,),
                                  "norm": (V,)})
        self.proj = Linear(d, stack_rows(d, [d.bf16(W[n]) for n in ("q", "k", "v", "g", "b", "a")]))
        self.out = Linear(d, d.bf16(W["o"]))
        self.conv = d.torch.cat([d.f32(W[n + ".conv"]) for n in ("q", "k", "v")], dim=0).t().contiguous()
        self.a_log, self.dt_bias, self.norm = d.f32(W["A_log"]), d.f32(W["dt_bias"]), d.f32(W["norm"])
        self.c = _lib.PgDelta(H, G, D, V, taps, self.eps, self.UNIT_EPS, self.conv.data_ptr(), self.a_log.data_ptr(), self.dt_bias.data_ptr(),
                              self.norm.data_ptr(), 0)
        # shared buffers exist before the first step: torch fills them on a stream of its own
        d.buffer("delta.work", 1, d.lib.pg_delta_work_floats(C.byref(self.c), d.rows), d.torch.float32)
        d.buffer("proj", self.proj.n, dtype=d.torch.float32)
        d.buffer("mixed", self.out.k)

    def new_state(self, pool):
        t = self.d.torch
        return {"ring": pool.tensor((self.taps, self.channels), t.float32), "state": pool.tensor((self.H, self.D, up(self.V, 4)), t.float32)}

    def run(self, batch, h, state, y) -> None:
        """h [rows, K] -> y [rows, width] f32."""
        d = self.d
        rows = batch.rows
        proj = d.buffer("proj", self.proj.n, dtype=d.torch.float32)
        mixed = d.buffer("mixed", self.out.k)
        self.proj.run(h, rows, proj)
        self.c.d_work = d.buffer("delta.work", 1, 1, d.torch.float32).data_ptr()
        d.check(d.lib.pg_delta_run(d.gpu.handle, C.byref(self.c), C.byref(batch.c), proj.data_ptr(), proj.stride(0), state["ring"].data_ptr(),
                                   state["state"].data_ptr(), mixed.data_ptr(), d.code, mixed.stride(0)))
        self.out.run(mixed, rows, y)

    def bytes(self) -> int:
        return self.proj.bytes() + self.out.bytes()

    def free(self) -> None:
        self.proj.free()
        self.out.free()


def halving_slopes(heads: int) -> np.ndarray:
    """Slopes of a distance bias: 2^(-8 (h + 1) / heads) for head h."""
    return (2.0 ** (-8.0 * np.arange(1, heads + 1) / heads)).astype(np.float32)


class Attention:
    """p: heads, kv_heads, dim, vdim, scale and, if the query temperature grows, q_temp {coef, every}.  norms: per-head query
    and key norms; slopes: [heads] of a bias slope * distance that is taken off the score; chunk: a position sees the
    positions of its own chunk only, and the cache keeps the chunks that a step can touch."""

    def __init__(self, d: Device, p: dict, W, width: int, eps: float, capacity: int, max_seqs: int, sink: bool = True, norms: bool = True, slopes=None,
                 chunk: int = 0):
        self.d, self.p = d, p
        H, G, D, V = (int(p[k]) for k in ("heads", "kv_heads", "dim", "vdim"))
        if H % G:
            raise ValueError(f"attention mixer: {H} heads on {G} key/value heads")
        self.H, self.G, self.D, self.V, self.cap = H, G, D, V, int(capacity)
        if chunk:
            # whole chunks: what the longest step can touch, or the whole sequence
            self.cap = chunk * min((chunk + d.rows - 2) // chunk + 1, (int(capacity) + chunk - 1) // chunk)
        expect("attention mixer", W, {"q": (H * D, width), "k": (G * D, width), "v": (G * V, width), "o": (width, H * V),
                                      **({"q.norm": (D,), "k.norm": (D,)} if norms else {})})
        self.proj = Linear(d, stack_rows(d, [d.bf16(W[n]) for n in ("q", "k", "v")]))
        self.out = Linear(d, d.bf16(W["o"]))
        self.qn, self.kn = (d.f32(W["q.norm"]), d.f32(W["k.norm"])) if norms else (None, None)
        self.slopes = d.f32(slopes) if slopes is not None else None
        ptr = lambda t: t.data_ptr() if t is not None else 0
        temp = p.get("q_temp") or {}
        self.dp, self.vp = up(D, 16), up(V, 16)
        f32 = d.torch.float32
        self.c = _lib.PgAttention(H, G, D, V, self.cap, 0, float(eps), float(p["scale"]), float(temp.get("coef", 0.0)), float(temp.get("every", 0.0)), int(sink),
                                  int(chunk), int(capacity), ptr(self.qn), ptr(self.kn), ptr(self.slopes), 0, 0, 0)
        d.buffer("attn.part", 1, max(1, d.lib.pg_attention_part_floats(d.gpu.handle, C.byref(self.c), max_seqs)), f32)
        d.buffer("attn.tickets", 1, max_seqs * G * ((H // G + 15) // 16), d.torch.int32)
        d.buffer("attn.q", H * self.dp)
        d.buffer("proj", self.proj.n, dtype=f32)
        d.buffer("mixed", self.out.k)

    def new_state(self, pool):
        a = self.d.act
        return {"k": pool.tensor((self.G, self.cap, self.dp), a), "v": pool.tensor((self.G, self.cap, self.vp), a)}

    def run(self, batch, h, state, y) -> None:
        d = self.d
        rows = batch.rows
        proj = d.buffer("proj", self.proj.n, dtype=d.torch.float32)
        mixed = d.buffer("mixed", self.out.k)
        self.proj.run(h, rows, proj)
        self.c.d_q = d.buffer("attn.q", self.H * self.dp).data_ptr()
        self.c.d_part = d.buffer("attn.part", 1, 1, d.torch.float32).data_ptr()
        self.c.d_tickets = d.buffer("attn.tickets", 1, 1, d.torch.int32).data_ptr()
        self.c.slots = state["k"].shape[0]
        d.check(d.lib.pg_attention_run(d.gpu.handle, C.byref(self.c), C.byref(batch.c), proj.data_ptr(), proj.stride(0), state["k"].data_ptr(),
                                       state["v"].data_ptr(), mixed.data_ptr(), d.code, mixed.stride(0)))
        self.out.run(mixed, rows, y)

    def bytes(self) -> int:
        return self.proj.bytes() + self.out.bytes()

    def free(self) -> None:
        self.proj.free()
        self.out.free()


class LatentAttention:
    """p: heads, dim, rot_dim, vdim, kv_rank, scale, rot {base, dims}.  own: the layer projects latents of its own and keeps
    them; else it reads the state of a layer that does, which has run before it in the same step.

    Short portions attend over the latents themselves, with W_uk on the queries and W_uv on the sums; longer ones unfold
    keys and values of their sequence's whole context first (csrc/pg_latent.cu)."""

    LONG = 64      # tokens from which unfolding is the shorter way

    def __init__(self, d: Device, p: dict, W, width: int, eps: float, capacity: int, max_seqs: int, own: bool = True):
        t = d.torch
        self.d, self.p, self.own = d, p, own
        H, D, R, V, K = (int(p[k]) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
        self.H, self.D, self.R, self.V, self.K, self.cap = H, D, R, V, K, int(capacity)
        if int(p["rot"]["dims"]) != R or R % 2:
            raise ValueError(f"latent attention mixer: {p['rot']['dims']} rotated dimensions of {R}")
        expect("latent attention mixer", W, {"q": (H * (D + R), width), "uk": (H * D, K), "uv": (H * V, K), "g": (H * V, width), "o": (width, H * V),
                                             **({"dkv": (K + R, width), "dkv.norm": (K,)} if own else {})})
        self.proj = Linear(d, stack_rows(d, [d.bf16(W[n]) for n in (("q", "dkv", "g") if own else ("q", "g"))]))
        self.out = Linear(d, d.bf16(W["o"]))
        self.norm = d.f32(W["dkv.norm"]) if own else None
        self.cp, self.ck = up(K, 64), up(K, 64) + up(R, 16)
        bf, dev = t.bfloat16, d.dev
        uk, uv = d.bf16(W["uk"]).view(H, D, K), d.bf16(W["uv"]).view(H, V, K)
        self.uk = t.zeros(H, self.cp, up(D, 32), dtype=bf, device=dev)
        self.uk[:, :K, :D] = uk.transpose(1, 2)
        self.uv = t.zeros(H * V + 7, self.cp, dtype=bf, device=dev)
        self.uv[:H * V, :K] = uv.reshape(H * V, K)
        self.rot = d.rotation(p["rot"]["base"], R, self.cap)
        qd = max(self.ck, up(D, 64) + up(R, 64))
        f32 = t.float32
        self.c = _lib.PgLatent(H, D, R, V, K, self.cap, 0, int(own), float(eps), float(p["scale"]), self.rot.data_ptr(),
                               self.norm.data_ptr() if own else 0, self.uk.data_ptr(), self.uv.data_ptr(), 0, 0, 0)
        self.unfold = None
        if d.code == _lib.BF16 and d.lib.pg_latent_prompt_supports(C.byref(self.c)):
            dn, vn = up(D, 16), up(V, 16)
            w = t.zeros(H * (dn + vn), self.cp, dtype=bf, device=dev)
            w[:H * dn].view(H, dn, self.cp)[:, :D, :K] = uk
            w[H * dn:].view(H, vn, self.cp)[:, :V, :K] = uv
            self.unfold = Linear(d, w)
            d.buffer("latent.kv", self.unfold.n, self.cap)
        d.buffer("latent.q", H * qd)
        self.qd = qd
        self.part_rows = d.lib.pg_latent_part_floats(d.gpu.handle, C.byref(self.c), d.code, d.rows, max_seqs)
        d.buffer("latent.part", 1, self.part_rows, f32)
        d.buffer("proj", self.proj.n, dtype=f32)
        d.buffer("mixed", self.out.k)

    def new_state(self, pool):
        return {"latent": pool.tensor((self.cap, self.ck), self.d.act)}

    def run(self, batch, h, state, y) -> None:
        d, c = self.d, self.c
        rows, lib, gh = batch.rows, d.lib, d.gpu.handle
        proj = d.buffer("proj", self.proj.n, dtype=d.torch.float32)
        mixed = d.buffer("mixed", self.out.k)
        cache = state["latent"]
        self.proj.run(h, rows, proj)
        c.d_q = d.buffer("latent.q", self.H * self.qd).data_ptr()
        c.d_part, c.part_floats = d.buffer("latent.part", 1, 1, d.torch.float32).data_ptr(), self.part_rows
        c.slots = cache.shape[0]
        long_from = self.LONG if self.unfold is not None else 1 << 30
        lens = [n for _slot, _pos, n in batch.parts if n < long_from]
        d.check(lib.pg_latent_run(gh, C.byref(c), C.byref(batch.c), long_from, sum(lens), max(lens, default=0), proj.data_ptr(), proj.stride(0),
                                  cache.data_ptr(), mixed.data_ptr(), d.code, mixed.stride(0)))
        row0 = 0
        for seq, (slot, pos, n) in enumerate(batch.parts):
            if n >= long_from:
                d.check(lib.pg_latent_prompt_prep(gh, C.byref(c), C.byref(batch.c), row0, n, slot, proj.data_ptr(), proj.stride(0), cache.data_ptr()))
                kv = d.buffer("latent.kv", self.unfold.n, self.cap)
                self.unfold.run_ld(cache[slot].data_ptr(), self.ck, pos + n, kv)
                d.check(lib.pg_latent_prompt(gh, C.byref(c), C.byref(batch.c), seq, n, pos + n, slot, proj.data_ptr(), proj.stride(0), cache.data_ptr(),
                                             kv.data_ptr(), kv.stride(0), mixed.data_ptr(), mixed.stride(0)))
            row0 += n
        self.out.run(mixed, rows, y)

    def bytes(self) -> int:
        return self.proj.bytes() + self.out.bytes() + (self.uk.numel() + self.uv.numel()) * 2

    def free(self) -> None:
        for x in (self.proj, self.out, self.unfold):
            if x is not None:
                x.free()


class SelectiveScan:
    """p: inner, state, dt_rank, conv (taps).  Per channel and state S <- exp(dt A) S + dt x B, read out with C."""

    def __init__(self, d: Device, p: dict, W, width: int):
        t = d.torch
        self.d, self.p = d, p
        I, N, R, taps = (int(p[k]) for k in ("inner", "state", "dt_rank", "conv"))
        self.I, self.N, self.taps = I, N, taps
        expect("scan mixer", W, {"in": (2 * I, width), "conv": (I, taps), "conv.b": (I,), "x": (R + 2 * N, I), "dt": (I, R), "dt.b": (I,), "A_log": (I, N),
                                 "D": (I,), "o": (width, I)})
        self.proj = Linear(d, stack_rows(d, [d.bf16(W["in"])]))
        self.out = Linear(d, d.bf16(W["o"]))
        # [dt, padded to 64 rows | B | C]: one product where a token decodes, two where a prompt needs dt as an operand
        self.dtp = up(R, 64)
        x = d.bf16(W["x"])
        low = t.zeros(up(self.dtp + 2 * N, 4), up(I, 64), dtype=t.bfloat16, device=d.dev)
        low[:R, :I], low[self.dtp:self.dtp + 2 * N, :I] = x[:R], x[R:]
        self.low, self.low_dt, self.low_bc = Linear(d, low), Linear(d, low[:self.dtp]), Linear(d, low[self.dtp:])
        self.dt = Linear(d, d.bf16(W["dt"]))
        self.conv = d.f32(W["conv"]).t().contiguous()
        self.conv_b, self.dt_b, self.skip = d.f32(W["conv.b"]), d.f32(W["dt.b"]), d.f32(W["D"])
        self.ss = up(N, 4)
        self.a = t.zeros(I, self.ss, device=d.dev)
        self.a[:, :N] = (-t.exp(d.f32(W["A_log"]).double()) * 1.4426950408889634).float()
        self.c = _lib.PgScan(I, N, R, taps, self.conv.data_ptr(), self.conv_b.data_ptr(), self.a.data_ptr(), self.skip.data_ptr(), self.dt_b.data_ptr(),
                             self.dt.w.data_ptr())
        f32 = t.float32
        d.buffer("proj", self.proj.n, dtype=f32)
        d.buffer("mixed", self.out.k)
        d.buffer("scan.x", self.low.k)
        d.buffer("scan.low", self.low.n, dtype=f32)
        d.buffer("scan.dt_low", self.dtp)
        d.buffer("scan.dt", up(I, 4), dtype=f32)
        d.buffer("scan.bc", self.low_bc.n, dtype=f32)

    def new_state(self, pool):
        t = self.d.torch
        return {"ring": pool.tensor((self.taps, self.I), t.float32), "state": pool.tensor((self.I, self.ss), t.float32)}

    def run(self, batch, h, state, y) -> None:
        d, c, b = self.d, C.byref(self.c), C.byref(batch.c)
        rows, lib, gh, f32 = batch.rows, d.lib, d.gpu.handle, d.torch.float32
        proj = d.buffer("proj", self.proj.n, dtype=f32)
        mixed = d.buffer("mixed", self.out.k)
        x = d.buffer("scan.x", self.low.k)
        self.proj.run(h, rows, proj)
        d.check(lib.pg_scan_conv(gh, c, b, proj.data_ptr(), proj.stride(0), state["ring"].data_ptr(), x.data_ptr(), d.code, x.stride(0)))
        if batch.c.max_len == 1:
            low = d.buffer("scan.low", self.low.n, dtype=f32)
            self.low.run(x, rows, low)
            d.check(lib.pg_scan_step(gh, c, b, proj.data_ptr(), proj.stride(0), x.data_ptr(), x.stride(0), low.data_ptr(), low.stride(0),
                                     state["state"].data_ptr(), mixed.data_ptr(), d.code, mixed.stride(0)))
        else:
            dt_low, dt = d.buffer("scan.dt_low", self.dtp), d.buffer("scan.dt", up(self.I, 4), dtype=f32)
            bc = d.buffer("scan.bc", self.low_bc.n, dtype=f32)
            self.low_dt.run(x, rows, dt_low)
            self.dt.run(dt_low, rows, dt)
            self.low_bc.run(x, rows, bc)
            d.check(lib.pg_scan_run(gh, c, b, proj.data_ptr(), proj.stride(0), state["ring"].data_ptr(), x.data_ptr(), x.stride(0), dt.data_ptr(), dt.stride(0),
                                    bc.data_ptr(), bc.stride(0), state["state"].data_ptr(), mixed.data_ptr(), d.code, mixed.stride(0)))
        self.out.run(mixed, rows, y)

    def bytes(self) -> int:
        return sum(x.bytes() for x in (self.proj, self.out, self.low, self.dt)) + self.a.numel() * 4

    def free(self) -> None:
        for x in (self.proj, self.out, self.low, self.low_dt, self.low_bc, self.dt):
            x.free()


# ---- feed-forwards: `run` ends with the residual update, which for experts also adds up their outputs --------------
class DenseFF:
    """gelu_tanh(gate) * up; where `mlp` has a limit, the clamped swish form of the experts."""

    def __init__(self, d: Device, mlp: dict, W, width: int):
        self.d = d
        F = int(mlp["ff"])
        expect("feed-forward", W, {"gate": (F, width), "up": (F, width), "down": (width, F)})
        self.limit = float(mlp.get("limit", 0.0))
        self.act = _lib.ACT_CLAMPED_SWISH_GLU if "limit" in mlp else _lib.ACT_GELU_TANH_GLU
        self.gate_up = Linear(d, (d.bf16(W["gate"]), d.bf16(W["up"])), gated=True)
        self.down = Linear(d, d.bf16(W["down"]))
        d.buffer("act", self.down.k)

    def run(self, batch, h, y, add) -> None:
        """add(y): the model's residual update from a plain output."""
        act = self.d.buffer("act", self.down.k)
        self.gate_up.run(h, batch.rows, act, self.act, self.limit)
        self.down.run(act, batch.rows, y)
        add(y)

    def bytes(self, tokens: int = 1) -> int:
        return self.gate_up.bytes() + self.down.bytes()

    def free(self) -> None:
        self.gate_up.free()
        self.down.free()


class MoeFF:
    def __init__(self, d: Device, mlp: dict, W, width: int):
        self.d = d
        r = mlp["router"]
        self.E, self.I, self.top = int(r["experts"]), int(r.get("identity", 0)), int(r["top"])
        groups = r.get("groups") or {"count": 1, "keep": 1}
        self.groups, self.keep = int(groups["count"]), int(groups["keep"])
        F = int(mlp["expert"]["ff"])
        self.limit = float(mlp["expert"]["limit"])
        for e in range(self.E):
            for name, shape in {"gate": (F, width), "up": (F, width), "down": (width, F)}.items():
                if tuple(W[f"e{e}.{name}"].shape) != shape:
                    raise ValueError(f"expert {e}: {name} is {list(W[f'e{e}.{name}'].shape)}, the configuration says {list(shape)}")
        if tuple(W["router"].shape) != (self.E + self.I, width) or tuple(W["correction"].shape) != (self.E + self.I,):
            raise ValueError("router: the tensors do not fit the configuration")
        every = lambda name: d.torch.stack([d.bf16(W[f"e{e}.{name}"]) for e in range(self.E)])
        self.router = Linear(d, stack_rows(d, [d.bf16(W["router"])]))
        self.correction = d.f32(W["correction"])
        self.gate_up = Linear(d, (every("gate"), every("up")), gated=True)
        self.down = Linear(d, every("down"))
        h = C.c_void_p()
        d.check(d.lib.pg_route_create(d.gpu.handle, d.rows, self.E, self.I, self.top, C.byref(h)))
        self.route = h
        self.max_rows = int(d.lib.pg_route_max_rows(h))
        d.buffer("expert.act", self.down.k, self.max_rows)
        d.buffer("expert.out", up(self.down.n, 8), self.max_rows)
        d.buffer("router", self.router.n, dtype=d.torch.float32)

    def run(self, batch, h, y, add) -> None:
        """add(route, outputs): the model's residual update from routed outputs."""
        d = self.d
        logits = d.buffer("router", self.router.n, dtype=d.torch.float32)
        self.router.run(h, batch.rows, logits)
        d.check(d.lib.pg_route_run(d.gpu.handle, self.route, d.code, logits.data_ptr(), logits.stride(0), batch.rows, self.correction.data_ptr(), self.groups,
                                   self.keep))
        act = d.buffer("expert.act", self.down.k, self.max_rows)
        out = d.buffer("expert.out", up(self.down.n, 8), self.max_rows)
        self.gate_up.run_routed(self.route, h, True, act, _lib.ACT_CLAMPED_SWISH_GLU, self.limit)
        self.down.run_routed(self.route, act, False, out)
        add(out, self.route)

    def bytes(self, tokens: int = 1) -> int:
        """Read by a step of `tokens` tokens at most: every expert that can be chosen, once."""
        return self.router.bytes() + (self.gate_up.bytes() + self.down.bytes()) * min(self.E, tokens * self.top) // self.E

    def chosen(self, rows: int):
        """(ids, weights) [rows, top] of the last step, on the host."""
        ids, w = np.zeros((rows, self.top), np.int32), np.zeros((rows, self.top), np.float32)
        self.d.check(self.d.lib.pg_route_read(self.d.gpu.handle, self.route, ids.ctypes.data, w.ctypes.data))
        return ids, w

    def free(self) -> None:
        for x in (self.router, self.gate_up, self.down):
            x.free()
        if self.route is not None:
            self.d.lib.pg_route_free(self.d.gpu.handle, self.route)
            self.route = None


def BATCH_WORDS(rows: int) -> int:
    return 6 * rows + 64


class Batch:
    """The rows of one step on the device (pg_batch).  entries: (slot, first position, tokens) per sequence; `rows`: rows
    whose logits are wanted.  With `fixed` the arrays keep their addresses, so that a recorded graph can be replayed."""

    def __init__(self, d: Device, entries, wanted=(), fixed: bool = False):
        seqs = len(entries)
        lens = [len(e[2]) for e in entries]
        self.rows, self.seqs, self.wanted = sum(lens), seqs, len(wanted)
        self.parts = [(e[0], e[1], n) for e, n in zip(entries, lens)]     # slot, first position, tokens
        n = self.rows
        host = np.zeros(3 * n + 2 * seqs + 1 + self.wanted, np.int32)
        at = 0
        for i, (slot, pos0, tokens) in enumerate(entries):
            k = lens[i]
            host[at:at + k] = tokens
            host[n + at:n + at + k] = np.arange(pos0, pos0 + k)
            host[2 * n + at:2 * n + at + k] = i
            host[3 * n + i + 1] = at + k
            host[3 * n + seqs + 1 + i] = slot
            at += k
        host[3 * n + 2 * seqs + 1:] = wanted
        if fixed:
            self.mem = d.torch.zeros(host.size, dtype=d.torch.int32, device=d.dev)
            d.torch.cuda.synchronize()
        else:
            self.mem = d.buffer("batch", 1, BATCH_WORDS(d.rows), d.torch.int32)
            if host.size > self.mem.shape[0]:
                raise ValueError(f"a step of {n} rows, more than the {d.rows} the model was made for")
        self.d = d
        self.write(host)
        p = self.mem.data_ptr()
        self.c = _lib.PgBatch(n, seqs, max(lens, default=0), p, p + 4 * n, p + 8 * n, p + 12 * n, p + 4 * (3 * n + seqs + 1))
        self.d_tokens, self.d_pos = p, p + 4 * n
        self.d_wanted = p + 4 * (3 * n + 2 * seqs + 1)

    def write(self, host: np.ndarray) -> None:
        # pageable host memory: the copy has left `host` when the call returns
        self.d.gpu.check(self.d.lib.pg_mem_upload(self.d.gpu.handle, self.mem.data_ptr(), host.ctypes.data, host.nbytes))
