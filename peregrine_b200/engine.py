"""The serving loop of the models that keep a slot per sequence: requests, their slots, the steps that the scheduler
makes of them, and greedy generation.

A step runs the next tokens of one or more requests.  `Engine.step` takes exactly what it is given (a trace);
`Engine.generate` schedules: waiting prompts are run in portions of at most `portion` tokens as slots come free, and all
sequences whose prompt is done decode together.  Decoding is one recorded graph per number of sequences, replayed; the
greedy choice, the next tokens and the positions stay on the device.
"""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass, field
from typing import Dict, Hashable, List, Optional, Sequence, Tuple

import numpy as np

from .layers import Batch


class RequestError(ValueError):
    pass


@dataclass
class Live:
    """A request with a slot: `length` tokens are in its cache or state."""
    slot: int
    length: int = 0


@dataclass
class Generation:
    prompt: List[int]
    max_new: int
    stop: frozenset
    key: Hashable = None
    fed: int = 0
    out: List[int] = field(default_factory=list)

    @property
    def done(self) -> bool:
        return len(self.out) >= self.max_new or (bool(self.out) and self.out[-1] in self.stop)


class _Decode:
    """The recorded decode step of `n` sequences."""

    def __init__(self, model, n: int):
        self.model, self.n = model, n
        self.batch = Batch(model.d, [(0, 0, [0])] * n, list(range(n)), fixed=True)
        self.graph = None
        self.keys: Optional[Tuple] = None     # the sequences whose tokens and positions the device arrays hold

    def load(self, entries) -> None:
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
        """One step from what the device arrays hold."""
        m = self.model
        if self.graph is None:
            with m.gpu.record() as g:
                self.enqueue()
            self.graph = g
        self.graph.launch()

    def tokens(self) -> np.ndarray:
        out = np.empty(self.n, np.int32)
        m = self.model
        m.gpu.check(m.lib.pg_mem_download(m.gpu.handle, out.ctypes.data, self.batch.d_tokens, out.nbytes))
        return out


class Engine:
    def __init__(self, model, portion: int = 0):
        self.model = model
        self.portion = min(int(portion or model.step_rows), model.step_rows)
        self.live: Dict[Hashable, Live] = {}
        self._decode: Dict[int, _Decode] = {}

    # ---- requests ------------------------------------------------------------------------------------------------
    def _request(self, key) -> Live:
        r = self.live.get(key)
        if r is None:
            r = self.live[key] = Live(self.model.pool.take())
        return r

    def end(self, key) -> None:
        """The request is finished: its slot is given back."""
        r = self.live.pop(key, None)
        if r is not None:
            self.model.pool.give_back(r.slot)

    def _check_tokens(self, key, r: Live, tokens) -> None:
        if not len(tokens):
            raise RequestError(f"request {key!r}: no tokens")
        if min(tokens) < 0 or max(tokens) >= self.model.vocab:
            raise RequestError(f"request {key!r}: a token outside the vocabulary of {self.model.vocab}")
        if r.length + len(tokens) > self.model.capacity:
            raise RequestError(f"request {key!r}: {r.length + len(tokens)} positions, the cache has {self.model.capacity}")

    # ---- steps ---------------------------------------------------------------------------------------------------
    def step(self, entries: Sequence[Tuple[Hashable, Sequence[int], Sequence[int]]]) -> np.ndarray:
        """Runs the next tokens of each entry's request and returns the logits at the wanted places (indices into the
        entry's tokens), [wanted, vocab], in the order of the entries."""
        seen = set()
        for key, tokens, want in entries:
            if key in seen:
                raise RequestError(f"request {key!r} is in the step twice")
            seen.add(key)
            known = self.live.get(key)
            self._check_tokens(key, known or Live(-1), tokens)
            if any(not 0 <= w < len(tokens) for w in want):
                raise RequestError(f"request {key!r}: a wanted place outside its tokens")
        out, parts = [], []
        # rows of one step are limited: what does not fit follows in further steps
        todo = [[key, self._request(key), list(tokens), sorted(set(want)), 0] for key, tokens, want in entries]
        got: Dict[Tuple[Hashable, int], np.ndarray] = {}
        while todo:
            room, parts = self.portion, []
            for item in todo:
                n = min(room, len(item[2]) - item[4])
                if n > 0:
                    parts.append((item, item[4], n))
                    room -= n
            rows, wanted = [], []
            at = 0
            for item, lo, n in parts:
                for w in item[3]:
                    if lo <= w < lo + n:
                        wanted.append(at + w - lo)
                        rows.append((item[0], w))
                at += n
            self._run([(item[1].slot, item[1].length, item[2][lo:lo + n]) for item, lo, n in parts], wanted, rows, got)
            for item, lo, n in parts:
                item[1].length += n
                item[4] = lo + n
            todo = [item for item in todo if item[4] < len(item[2])]
        for key, _tokens, want in entries:
            out += [got[(key, w)] for w in want]
        return np.stack(out) if out else np.zeros((0, self.model.vocab), np.float32)

    def _run(self, entries, wanted, names, got) -> None:
        m = self.model
        batch = Batch(m.d, entries, wanted)
        m.forward(batch)
        for i in range(0, len(wanted), m.max_wanted):
            n = min(m.max_wanted, len(wanted) - i)
            m.head_rows(batch.d_wanted + 4 * i, n)
            for name, row in zip(names[i:i + n], m.read_logits(n)):
                got[name] = row.copy()
        self.check_device()

    def check_device(self) -> None:
        status = self.model.gpu.device_status()
        if status:
            raise RuntimeError(f"a kernel reported status {status}")

    # ---- generation ----------------------------------------------------------------------------------------------
    def generate(self, prompts: Sequence[Sequence[int]], max_new: int, stop: Sequence[int] = ()) -> List[List[int]]:
        """Greedy continuation of every prompt (token ids): at most max_new tokens each, up to and including a stop token."""
        m = self.model
        jobs = [Generation(list(p), int(max_new), frozenset(stop), key=("generate", id(self), i)) for i, p in enumerate(prompts)]
        for j in jobs:
            self._check_tokens(j.key, Live(-1), j.prompt)
            # the last new token is not run
            if len(j.prompt) + max_new - 1 > m.capacity:
                raise RequestError(f"a prompt of {len(j.prompt)} and {max_new} new tokens, the cache has {m.capacity} positions")
        waiting, running = ([j for j in jobs if max_new > 0]), []
        prefilling: List[Generation] = []
        try:
            while waiting or prefilling or running:
                while waiting and m.pool.free:
                    j = waiting.pop(0)
                    self._request(j.key)
                    prefilling.append(j)
                if prefilling:
                    self._prefill(prefilling)
                else:
                    self._decode_step(running)
                for j in [j for j in prefilling if j.fed == len(j.prompt)]:
                    prefilling.remove(j)
                    running.append(j)
                for j in [j for j in running if j.done]:
                    running.remove(j)
                    self.end(j.key)
        finally:
            for j in jobs:
                self.end(j.key)
        return [j.out for j in jobs]

    def _prefill(self, jobs: List[Generation]) -> None:
        """One step of prompt portions; prompts that end in it get their first token."""
        m = self.model
        room, parts, wanted, enders, at = self.portion, [], [], [], 0
        for j in jobs:
            n = min(room, len(j.prompt) - j.fed)
            if n <= 0:
                continue
            r = self.live[j.key]
            parts.append((r.slot, r.length, j.prompt[j.fed:j.fed + n]))
            r.length += n
            j.fed += n
            room -= n
            at += n
            if j.fed == len(j.prompt):
                wanted.append(at - 1)
                enders.append(j)
        batch = Batch(m.d, parts, wanted)
        m.forward(batch)
        if enders:
            n = len(enders)
            m.head_rows(batch.d_wanted, n)
            # the choice goes to the head of the batch's own arrays, which the step is done with
            m.d.check(m.lib.pg_argmax_rows(m.gpu.handle, m.logits.data_ptr(), n, m.vocab, batch.d_tokens, None, 0))
            out = np.empty(n, np.int32)
            m.gpu.check(m.lib.pg_mem_download(m.gpu.handle, out.ctypes.data, batch.d_tokens, out.nbytes))
            for j, t in zip(enders, out):
                j.out.append(int(t))
        self.check_device()

    def _decode_step(self, jobs: List[Generation]) -> None:
        n = len(jobs)
        d = self._decode.get(n)
        if d is None:
            d = self._decode[n] = _Decode(self.model, n)
        keys = tuple((j.key, len(j.out)) for j in jobs)
        if d.keys != keys:
            d.load([(self.live[j.key].slot, self.live[j.key].length, j.out[-1]) for j in jobs])
        d.run()
        for j, t in zip(jobs, d.tokens()):
            self.live[j.key].length += 1
            j.out.append(int(t))
        d.keys = tuple((j.key, len(j.out)) for j in jobs)
        self.check_device()


class LockstepEngine:
    """`generate` for the decoders that step a fixed batch at one common position (`LlamaInt8Decoder`): prompts of one
    length, run token by token through the recorded step."""

    def __init__(self, decoder):
        self.model = decoder

    def generate(self, prompts: Sequence[Sequence[int]], max_new: int, stop: Sequence[int] = ()) -> List[List[int]]:
        m = self.model
        B, n = m.cfg.batch, len(prompts[0])
        if len(prompts) > B or any(len(p) != n for p in prompts) or n == 0:
            raise RequestError(f"this model decodes up to {B} prompts of one length together")
        if n + max_new - 1 > m.cfg.capacity:
            raise RequestError(f"a prompt of {n} and {max_new} new tokens, the cache has {m.cfg.capacity} positions")
        rows = [list(p) for p in prompts] + [list(prompts[0])] * (B - len(prompts))
        if any(not 0 <= t < m.cfg.vocab for p in rows for t in p):
            raise RequestError(f"a token outside the vocabulary of {m.cfg.vocab}")
        out: List[List[int]] = [[] for _ in prompts]
        done = [max_new <= 0] * len(prompts)
        for i in range(n + max_new - 1):
            if all(done):
                break
            m.set_position(i)
            if i < n:
                m.set_tokens([p[i] for p in rows])
                m.embed()
            m.gpu.sync()
            if m.graph is None:
                m.record()
            m.graph.launch()
            m.gpu.sync()
            if i >= n - 1:
                for k, t in enumerate(m.tokens.cpu().tolist()[:len(prompts)]):
                    if not done[k]:
                        out[k].append(int(t))
                        done[k] = len(out[k]) >= max_new or int(t) in stop
        return out
