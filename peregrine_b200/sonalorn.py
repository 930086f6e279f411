"""Sonalorn: a decoder-only language model of gated delta rule and attention layers.

    x = norm(embed[token] + pos[p])
    per layer:  x += ls1 * norm1(mixer(x));  x += ls2 * norm2(ff(x))        (norms on the sublayers' outputs)
    logits = head norm(x)

The configuration lists the layers: the type of mixer and its sizes, a dense or mixture-of-experts feed-forward or none,
and optionally the index of an earlier layer whose tensors it uses (with a cache or state of its own).  The mechanisms
are in peregrine_b200/layers.py.
"""
from __future__ import annotations

import ctypes as C
import json
import os
from dataclasses import dataclass
from typing import Iterator, List

from .layers import BATCH_WORDS, Attention, Batch, DenseFF, Device, GatedDelta, Linear, MoeFF, up
from .safetensors_file import SafetensorsFile
from .slot_model import SlotModel
from .state import SlotPool

ARCHITECTURE = "Sonalorn"


@dataclass
class SonalornConfig:
    vocab: int
    width: int
    max_positions: int
    eps: float
    layers: List[dict]

    @staticmethod
    def from_dict(c: dict) -> "SonalornConfig":
        cfg = SonalornConfig(vocab=int(c["vocab"]), width=int(c["width"]), max_positions=int(c["max_positions"]), eps=float(c["norm"]["eps"]),
                             layers=list(c["layers"]))
        for i, L in enumerate(cfg.layers):
            if L["type"] not in ("delta", "attention"):
                raise ValueError(f"layer {i}: unknown mixer type {L['type']!r}")
            if L.get("mlp") and L["mlp"]["kind"] not in ("dense", "moe"):
                raise ValueError(f"layer {i}: unknown feed-forward kind {L['mlp']['kind']!r}")
            if L["type"] != cfg.layers[cfg.tensors_of(i)]["type"]:
                raise ValueError(f"layer {i}: another type than layer {cfg.tensors_of(i)}, whose tensors it uses")
        return cfg

    def tensors_of(self, i: int) -> int:
        """The layer whose tensors layer i uses."""
        j = i
        for _ in self.layers:
            k = self.layers[j].get("weights_of")
            if k is None:
                return j
            if not 0 <= k < len(self.layers):
                break
            j = k
        raise ValueError(f"layer {i}: weights_of leads to no layer with tensors")

    @staticmethod
    def load(path: str) -> "SonalornConfig":
        with open(os.path.join(path, "config.json")) as f:
            return SonalornConfig.from_dict(json.load(f))


class Below:
    """The tensors whose names start with a prefix, by the rest of their names."""

    def __init__(self, weights, prefix: str):
        self.weights, self.prefix = weights, prefix

    def __getitem__(self, name: str):
        return self.weights[self.prefix + name]


class SonalornModel(SlotModel):
    """weights: mapping name -> host array (bf16 bits as uint16, or f32, which is rounded to bf16 where a product reads it).
    slots / capacity: sequences alive at once and positions of each; step_rows: most tokens of one step; max_wanted: most
    rows of logits of one `head` call."""

    def __init__(self, cfg: SonalornConfig, weights, gpu, dtype: str = "bfloat16", slots: int = 1, capacity: int = 0, step_rows: int = 2048,
                 max_wanted: int = 64):
        self.cfg, self.gpu, self.lib = cfg, gpu, gpu.lib
        self.dtype, self.vocab, self.step_rows = dtype, cfg.vocab, max(int(step_rows), slots + 1)
        d = self.d = Device(gpu, dtype, self.step_rows)
        torch = self.torch = d.torch
        f32 = torch.float32

        def matrix(name, rows):
            t = d.bf16(weights[name]).contiguous()
            if tuple(t.shape) != (rows, cfg.width):
                raise ValueError(f"{name} is {list(t.shape)}, the configuration says [{rows}, {cfg.width}]")
            return t

        def vector(name):
            t = d.f32(weights[name])
            if tuple(t.shape) != (cfg.width,):
                raise ValueError(f"{name} is {list(t.shape)}, the configuration says [{cfg.width}]")
            return t

        self.embed, self.pos = matrix("embed", cfg.vocab), matrix("pos", cfg.max_positions)
        self.embed_norm, self.final_norm = vector("embed.norm"), vector("final.norm")
        self.head = Linear(d, matrix("head", cfg.vocab))
        self.capacity = min(int(capacity or cfg.max_positions), cfg.max_positions)
        self.pool = SlotPool(slots, self.capacity, d.dev)

        def tensors(i, L):
            W = Below(weights, f"l{i}.")
            mix = Below(weights, f"l{i}.mix.")
            out = {"norm1": vector(f"l{i}.norm1"), "ls1": vector(f"l{i}.ls1"), "ff": None}
            if L["type"] == "delta":
                out["mixer"] = GatedDelta(d, L["mixer"], mix, cfg.width, cfg.eps)
            else:
                out["mixer"] = Attention(d, L["mixer"], mix, cfg.width, cfg.eps, self.capacity, slots)
            if L.get("mlp"):
                out["ff"] = (DenseFF if L["mlp"]["kind"] == "dense" else MoeFF)(d, L["mlp"], Below(weights, f"l{i}.mlp."), cfg.width)
                out["norm2"], out["ls2"] = d.f32(W["norm2"]), d.f32(W["ls2"])
            return out

        own = {i: tensors(i, L) for i, L in enumerate(cfg.layers) if L.get("weights_of") is None}
        self._own = list(own.values())
        self.layers = []
        for i, L in enumerate(cfg.layers):
            shared = own[cfg.tensors_of(i)]
            self.layers.append({**shared, "state": shared["mixer"].new_state(self.pool)})
        self.ldh = up(cfg.width, 64)
        self.x = torch.zeros(self.step_rows, cfg.width, dtype=f32, device=d.dev)
        self.h = torch.zeros(self.step_rows, self.ldh, dtype=d.act, device=d.dev)
        self.y = torch.zeros(self.step_rows, up(cfg.width, 4), dtype=f32, device=d.dev)
        self.max_wanted = max(int(max_wanted), slots)
        self.picked = torch.zeros(self.max_wanted, self.ldh, dtype=d.act, device=d.dev)
        self.logits = torch.zeros(self.max_wanted, cfg.vocab, dtype=f32, device=d.dev)
        d.buffer("batch", 1, BATCH_WORDS(d.rows), torch.int32)
        torch.cuda.synchronize()   # torch filled the buffers on its own stream; the kernels use the context's

    @staticmethod
    def load(path: str, gpu, **kw) -> "SonalornModel":
        return SonalornModel(SonalornConfig.load(path), SafetensorsFile(os.path.join(path, "model.safetensors")), gpu, **kw)

    # ---- one step ------------------------------------------------------------------------------------------------
    def step_ops(self, batch: Batch) -> Iterator[str]:
        """Enqueues the layers for the rows of `batch`, yielding a label whenever the residual stream `x` is complete."""
        d, c = self.d, self.cfg
        ck, lib, gh = d.check, self.lib, self.gpu.handle
        rows, x, h, y = batch.rows, self.x, self.h, self.y
        ck(lib.pg_embed_norm(gh, C.byref(batch.c), self.embed.data_ptr(), self.pos.data_ptr(), c.width, self.embed_norm.data_ptr(), c.eps, x.data_ptr(),
                             h.data_ptr(), d.code, self.ldh))
        yield "embed"

        def add(norm, scale):
            def run(out, route=None):
                args = (out.stride(0), x.data_ptr(), norm.data_ptr(), scale.data_ptr(), rows, c.width, c.eps, h.data_ptr(), d.code, self.ldh)
                if route is None:
                    ck(lib.pg_norm_add(gh, out.data_ptr(), *args))
                else:
                    ck(lib.pg_routed_norm_add(gh, route, out.data_ptr(), *args))
            return run

        for i, L in enumerate(self.layers):
            L["mixer"].run(batch, h, L["state"], y)
            add(L["norm1"], L["ls1"])(y)
            yield f"l{i}.mixer"
            if L["ff"] is not None:
                L["ff"].run(batch, h, y, add(L["norm2"], L["ls2"]))
            yield f"l{i}"

    def head_rows(self, d_rows: int, n: int) -> None:
        """logits[:n] of the rows of the residual stream named by n int32 at the device address d_rows."""
        d, c = self.d, self.cfg
        d.check(self.lib.pg_norm_rows(self.gpu.handle, self.x.data_ptr(), d_rows, n, c.width, self.final_norm.data_ptr(), c.eps, self.picked.data_ptr(),
                                      d.code, self.ldh))
        self.head.run(self.picked, n, self.logits)

    def weight_bytes(self, tokens: int = 1) -> int:
        """bf16 weight bytes that a step of `tokens` tokens reads at most (every expert that can be chosen, once)."""
        total = self.head.bytes()
        for L in self.layers:
            total += L["mixer"].proj.bytes() + L["mixer"].out.bytes()
            f = L["ff"]
            if isinstance(f, DenseFF):
                total += f.gate_up.bytes() + f.down.bytes()
            elif f is not None:
                used = min(f.E, tokens * f.top)
                total += f.router.bytes() + (f.gate_up.bytes() + f.down.bytes()) * used // f.E
        return total

    def free(self) -> None:
        for L in self._own:
            L["mixer"].free()
            if L["ff"] is not None:
                L["ff"].free()
        self.head.free()
        self._own, self.layers = [], []
