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
from dataclasses import dataclass
from typing import Iterator, List

from .layers import Attention, Batch, DenseFF, GatedDelta, MoeFF
from .slot_model import Below, ResidualModel

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


class SonalornModel(ResidualModel):
    Config = SonalornConfig

    def build(self, weights) -> None:
        cfg, d = self.cfg, self.d
        self.pos, self.embed_norm = self.matrix("pos", cfg.max_positions), self.vector("embed.norm")

        def tensors(i, L):
            mix = Below(weights, f"l{i}.mix.")
            out = {"norm1": self.vector(f"l{i}.norm1"), "ls1": self.vector(f"l{i}.ls1"), "ff": None}
            if L["type"] == "delta":
                out["mixer"] = GatedDelta(d, L["mixer"], mix, cfg.width, cfg.eps)
            else:
                out["mixer"] = Attention(d, L["mixer"], mix, cfg.width, cfg.eps, self.capacity, self.slots)
            if L.get("mlp"):
                out["ff"] = (DenseFF if L["mlp"]["kind"] == "dense" else MoeFF)(d, L["mlp"], Below(weights, f"l{i}.mlp."), cfg.width)
                out["norm2"], out["ls2"] = self.vector(f"l{i}.norm2"), self.vector(f"l{i}.ls2")
            return out

        own = {i: tensors(i, L) for i, L in enumerate(cfg.layers) if L.get("weights_of") is None}
        self._own = list(own.values())
        for i in range(len(cfg.layers)):
            shared = own[cfg.tensors_of(i)]
            self.layers.append({**shared, "state": shared["mixer"].new_state(self.pool)})

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
