"""What the engine asks of a model that keeps a slot per sequence, on top of the model's own `step_ops` (the layers of one
step) and `head_rows` (logits of rows of the residual stream)."""
from __future__ import annotations

from typing import List, Sequence

import numpy as np

from .layers import Batch


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
