"""What the engine asks of a model that keeps a slot per sequence (SlotModel), on top of the model's own `step_ops` (the layers
of one step) and `head_rows` (logits of rows of the residual stream); and what the models with an f32 residual stream have in
common (ResidualModel)."""
from __future__ import annotations

import json
import os
from typing import List, Sequence

import numpy as np

from .layers import BATCH_WORDS, Batch, Device, Linear, up
from .safetensors_file import SafetensorsFile
from .state import SlotPool


class SlotModel:
    """A subclass has: d (layers.Device), gpu, lib, pool (state.SlotPool), vocab, capacity, step_rows, max_wanted, logits
    [max_wanted, vocab] f32, step_ops(batch) and head_rows(device address of row numbers, n)."""

    def forward(self, batch: Batch) -> None:
        for _ in self.step_ops(batch):
            pass

    def run(self, entries, wanted: Sequence[int]) -> np.ndarray:
        """One step: entries = (slot, first position, tokens) per sequence.  Logits [len(wanted), vocab] of the wanted rows."""
        batch = Batch(self.d, entries, wanted)
        self.forward(batch)
        out = np.empty((len(wanted), self.vocab), np.float32)
        for i in range(0, len(wanted), self.max_wanted):
            n = min(self.max_wanted, len(wanted) - i)
            self.head_rows(batch.d_wanted + 4 * i, n)
            part = out[i:i + n]
            self.gpu.check(self.lib.pg_mem_download(self.gpu.handle, part.ctypes.data, self.logits.data_ptr(), part.nbytes))
        self.check_device()
        return out

    def run_greedy(self, entries, wanted: Sequence[int]) -> List[int]:
        """One step and the greedy choice behind each wanted row (at most one per sequence)."""
        batch = Batch(self.d, entries, wanted)
        self.forward(batch)
        n = len(wanted)
        out = np.empty(n, np.int32)
        if n:
            self.head_rows(batch.d_wanted, n)
            # the choice goes to the head of the batch's own arrays, which the step is done with
            self.d.check(self.lib.pg_argmax_rows(self.gpu.handle, self.logits.data_ptr(), n, self.vocab, batch.d_tokens, None, 0))
            self.gpu.check(self.lib.pg_mem_download(self.gpu.handle, out.ctypes.data, batch.d_tokens, out.nbytes))
        self.check_device()
        return out.tolist()

    def decoder(self, n: int) -> "Decoder":
        return Decoder(self, n)

    def check_device(self) -> None:
        status = self.gpu.device_status()
        if status:
            raise RuntimeError(f"a kernel reported status {status}")


class Below:
    """The tensors whose names start with a prefix, by the rest of their names."""

    def __init__(self, weights, prefix: str):
        self.weights, self.prefix = weights, prefix

    def __getitem__(self, name: str):
        return self.weights[self.prefix + name]


class ResidualModel(SlotModel):
    """weights: mapping name -> host array (bf16 bits as uint16, or f32, which is rounded to bf16 where a product reads it).
    slots / capacity: sequences alive at once and positions of each; step_rows: most tokens of one step; max_wanted: most
    rows of logits of one `head` call.

    A subclass names its configuration class (`Config`), builds `layers` -- dicts with at least mixer, ff (or None) and state
    -- in `build(weights)`, and enqueues them in `step_ops`."""

    Config = None

    def __init__(self, cfg, weights, gpu, dtype: str = "bfloat16", slots: int = 1, capacity: int = 0, step_rows: int = 2048, max_wanted: int = 64):
        self.cfg, self.gpu, self.lib, self.weights = cfg, gpu, gpu.lib, weights
        self.dtype, self.vocab, self.step_rows, self.slots = dtype, cfg.vocab, max(int(step_rows), slots + 1), int(slots)
        d = self.d = Device(gpu, dtype, self.step_rows)
        torch = self.torch = d.torch
        f32 = torch.float32
        self.capacity = min(int(capacity or cfg.max_positions), cfg.max_positions)
        self.pool = SlotPool(slots, self.capacity, d.dev)
        self.embed, self.head, self.final_norm = self.matrix("embed", cfg.vocab), Linear(d, self.matrix("head", cfg.vocab)), self.vector("final.norm")
        self.layers: List[dict] = []
        self._own: List[dict] = []     # what `free` frees: layers with tensors of their own
        self.build(weights)
        self.ldh = up(cfg.width, 64)
        self.x = torch.zeros(self.step_rows, cfg.width, dtype=f32, device=d.dev)
        self.h = torch.zeros(self.step_rows, self.ldh, dtype=d.act, device=d.dev)
        self.y = torch.zeros(self.step_rows, up(cfg.width, 4), dtype=f32, device=d.dev)
        self.max_wanted = max(int(max_wanted), slots)
        self.picked = torch.zeros(self.max_wanted, self.ldh, dtype=d.act, device=d.dev)
        self.logits = torch.zeros(self.max_wanted, cfg.vocab, dtype=f32, device=d.dev)
        d.buffer("batch", 1, BATCH_WORDS(d.rows), torch.int32)
        self.weights = None
        torch.cuda.synchronize()   # torch filled the buffers on its own stream; the kernels use the context's

    @classmethod
    def load(cls, path: str, gpu, **kw) -> "ResidualModel":
        with open(os.path.join(path, "config.json")) as f:
            cfg = cls.Config.from_dict(json.load(f))
        return cls(cfg, SafetensorsFile(os.path.join(path, "model.safetensors")), gpu, **kw)

    def build(self, weights) -> None:
        raise NotImplementedError

    def matrix(self, name: str, rows: int):
        t = self.d.bf16(self.weights[name]).contiguous()
        if tuple(t.shape) != (rows, self.cfg.width):
            raise ValueError(f"{name} is {list(t.shape)}, the configuration says [{rows}, {self.cfg.width}]")
        return t

    def vector(self, name: str):
        t = self.d.f32(self.weights[name])
        if tuple(t.shape) != (self.cfg.width,):
            raise ValueError(f"{name} is {list(t.shape)}, the configuration says [{self.cfg.width}]")
        return t

    def head_rows(self, d_rows: int, n: int) -> None:
        """logits[:n] of the rows of the residual stream named by n int32 at the device address d_rows."""
        d, c = self.d, self.cfg
        d.check(self.lib.pg_norm_rows(self.gpu.handle, self.x.data_ptr(), d_rows, n, c.width, self.final_norm.data_ptr(), c.eps, self.picked.data_ptr(),
                                      d.code, self.ldh))
        self.head.run(self.picked, n, self.logits)

    def weight_bytes(self, tokens: int = 1) -> int:
        """Weight bytes that a step of `tokens` tokens reads at most."""
        return self.head.bytes() + sum(L["mixer"].bytes() + (L["ff"].bytes(tokens) if L["ff"] is not None else 0) for L in self.layers)

    def free(self) -> None:
        for L in self._own:
            L["mixer"].free()
            if L["ff"] is not None:
                L["ff"].free()
        self.head.free()
        self._own, self.layers = [], []


class Decoder:
    """The greedy decode step of n sequences, recorded once as a graph and replayed: tokens, positions and slots are arrays
    on the device, and a step leaves the next tokens and positions in them."""

    def __init__(self, model: SlotModel, n: int):
        self.model, self.n = model, n
        self.batch = Batch(model.d, [(0, 0, [0])] * n, list(range(n)), fixed=True)
        self.graph = None

    def load(self, entries) -> None:
        """entries: (slot, position, token) per sequence."""
        n = self.n
        host = np.zeros(6 * n + 1, np.int32)
        host[:n] = [e[2] for e in entries]
        host[n:2 * n] = [e[1] for e in entries]
        host[2 * n:3 * n] = np.arange(n)
        host[3 * n:4 * n + 1] = np.arange(n + 1)
        host[4 * n + 1:5 * n + 1] = [e[0] for e in entries]
        host[5 * n + 1:] = np.arange(n)
        self.batch.write(host)

    def enqueue(self) -> None:
        m, b = self.model, self.batch
        m.forward(b)
        m.head_rows(b.d_wanted, self.n)
        m.d.check(m.lib.pg_argmax_rows(m.gpu.handle, m.logits.data_ptr(), self.n, m.vocab, b.d_tokens, b.d_pos, m.capacity))

    def run(self) -> None:
        if self.graph is None:
            with self.model.gpu.record() as g:
                self.enqueue()
            self.graph = g
        self.graph.launch()

    def tokens(self) -> List[int]:
        out = np.empty(self.n, np.int32)
        m = self.model
        m.gpu.check(m.lib.pg_mem_download(m.gpu.handle, out.ctypes.data, self.batch.d_tokens, out.nbytes))
        m.check_device()
        return out.tolist()

    def free(self) -> None:
        if self.graph is not None:
            self.graph.free()
            self.graph = None
