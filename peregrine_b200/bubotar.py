"""Bubotar: a decoder-only language model of latent attention, chunked attention and selective scan layers.

    x = embed[token]
    per layer:  x += norm1b(mixer(norm1(x)));  x += norm2b(ff(norm2(x)))        (norms before and after each sublayer)
    logits = logit_scale * head norm(x)

The configuration lists the layers: the type of mixer and its sizes, and a feed-forward or none.  A latent attention layer may
name an earlier one (`kv_from`) whose latents it reads from that layer's cache.  The mechanisms are in
peregrine_b200/layers.py.
"""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass
from typing import Iterator, List

from .layers import Attention, Batch, DenseFF, LatentAttention, SelectiveScan, halving_slopes
from .slot_model import Below, ResidualModel

ARCHITECTURE = "Bubotar"
MIXERS = ("latent_attention", "attention", "mamba1")


@dataclass
class BubotarConfig:
    vocab: int
    width: int
    eps: float
    logit_scale: float
    layers: List[dict]
    max_positions: int = 1 << 20     # rotations and biases have no end of their own

    @staticmethod
    def from_dict(c: dict) -> "BubotarConfig":
        cfg = BubotarConfig(vocab=int(c["vocab"]), width=int(c["width"]), eps=float(c["norm"]["eps"]), logit_scale=float(c["logit_scale"]),
                            layers=list(c["layers"]))
        for i, L in enumerate(cfg.layers):
            if L["type"] not in MIXERS:
                raise ValueError(f"layer {i}: unknown mixer type {L['type']!r}")
            if L.get("mlp") and L["mlp"]["kind"] != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward kind {L['mlp']['kind']!r}")
            j = L["mixer"].get("kv_from")
            if j is not None:
                if L["type"] != "latent_attention" or not 0 <= j < i or cfg.layers[j]["type"] != "latent_attention":
                    raise ValueError(f"layer {i}: kv_from {j} is not an earlier latent attention layer")
                a, b = L["mixer"], cfg.layers[j]["mixer"]
                if b.get("kv_from") is not None or any(a[k] != b[k] for k in ("kv_rank", "rot_dim", "rot")):
                    raise ValueError(f"layer {i}: layer {j} has no latents that fit")
        return cfg


class BubotarModel(ResidualModel):
    Config = BubotarConfig
    POSITIONS = 4096     # of a sequence, where nothing is said

    def __init__(self, cfg: BubotarConfig, weights, gpu, capacity: int = 0, **kw):
        super().__init__(cfg, weights, gpu, capacity=capacity or self.POSITIONS, **kw)

    def build(self, weights) -> None:
        cfg, d = self.cfg, self.d
        self.final_norm *= cfg.logit_scale
        for i, L in enumerate(cfg.layers):
            p, mix = L["mixer"], Below(weights, f"l{i}.mix.")
            out = {"norm1": self.vector(f"l{i}.norm1"), "norm1b": self.vector(f"l{i}.norm1b"), "ff": None}
            source = p.get("kv_from")
            if L["type"] == "latent_attention":
                out["mixer"] = LatentAttention(d, p, mix, cfg.width, cfg.eps, self.capacity, self.slots, own=source is None)
            elif L["type"] == "attention":
                out["mixer"] = Attention(d, p, mix, cfg.width, cfg.eps, self.capacity, self.slots, sink=False, norms=False,
                                         slopes=halving_slopes(int(p["heads"])), chunk=int(p["mask"]["size"]))
            else:
                out["mixer"] = SelectiveScan(d, p, mix, cfg.width)
            out["state"] = out["mixer"].new_state(self.pool) if source is None else self.layers[source]["state"]
            if L.get("mlp"):
                out["ff"] = DenseFF(d, L["mlp"], Below(weights, f"l{i}.mlp."), cfg.width)
                out["norm2"], out["norm2b"] = self.vector(f"l{i}.norm2"), self.vector(f"l{i}.norm2b")
            self.layers.append(out)
        self._own = list(self.layers)

    def step_ops(self, batch: Batch) -> Iterator[str]:
        """Enqueues the layers for the rows of `batch`, yielding a label whenever the residual stream `x` is complete."""
        d, c = self.d, self.cfg
        ck, lib, gh = d.check, self.lib, self.gpu.handle
        rows, x, h, y = batch.rows, self.x, self.h, self.y
        ck(lib.pg_embed_prenorm(gh, C.byref(batch.c), self.embed.data_ptr(), c.width, self.layers[0]["norm1"].data_ptr(), c.eps, x.data_ptr(), h.data_ptr(),
                                d.code, self.ldh))
        yield "embed"

        def add(norm, following):
            """The residual update of a sublayer; h is then the input of the next one, whose norm is `following`."""
            def run(out):
                ck(lib.pg_norm_add_prenorm(gh, out.data_ptr(), out.stride(0), x.data_ptr(), norm.data_ptr(), following.data_ptr() if following is not None else 0,
                                           rows, c.width, c.eps, h.data_ptr(), d.code, self.ldh))
            return run

        for i, L in enumerate(self.layers):
            following = self.layers[i + 1]["norm1"] if i + 1 < len(self.layers) else None
            L["mixer"].run(batch, h, L["state"], y)
            add(L["norm1b"], L["norm2"] if L["ff"] is not None else following)(y)
            yield f"l{i}.mixer"
            if L["ff"] is not None:
                L["ff"].run(batch, h, y, add(L["norm2b"], following))
            yield f"l{i}"
