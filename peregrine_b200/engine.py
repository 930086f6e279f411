"""The serving loop of the models that keep a slot per sequence: requests, their slots, the steps that the scheduler
makes of them, and greedy generation.

A step runs the next tokens of one or more requests.  `Engine.step` takes exactly what it is given (a trace);
`Engine.generate` schedules: waiting prompts get slots as they come free; while a prompt is unfinished, a step carries the
next token of every running sequence and portions of prompts, at most `portion` tokens in all; otherwise all sequences
decode together, as one recorded graph per number of sequences, replayed, in which the greedy choice, the next tokens and
the positions stay on the device (peregrine_b200/slot_model.py).
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Dict, Hashable, List, Optional, Sequence, Tuple

import numpy as np

from .state import OutOfSlots


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


class Engine:
    def __init__(self, model, portion: int = 0):
        self.model = model
        # a step has room for the next tokens of all slots and some of a prompt
        self.portion = max(min(int(portion or model.step_rows), model.step_rows), min(model.pool.slots + 1, model.step_rows))
        self._runs = 0
        self.live: Dict[Hashable, Live] = {}
        self._decoders: Dict[int, object] = {}
        self._loaded: Dict[int, tuple] = {}     # the sequences whose next tokens a decoder's device arrays hold

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
        if len(seen - set(self.live)) > self.model.pool.free:
            raise OutOfSlots(f"{len(seen - set(self.live))} new requests, {self.model.pool.free} free slots")
        out = []
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
            got.update(zip(rows, self.model.run([(item[1].slot, item[1].length, item[2][lo:lo + n]) for item, lo, n in parts], wanted)))
            for item, lo, n in parts:
                item[1].length += n
                item[4] = lo + n
            todo = [item for item in todo if item[4] < len(item[2])]
        for key, _tokens, want in entries:
            out += [got[(key, w)] for w in want]
        return np.stack(out) if out else np.zeros((0, self.model.vocab), np.float32)

    # ---- generation ----------------------------------------------------------------------------------------------
    def generate(self, prompts: Sequence[Sequence[int]], max_new: int, stop: Sequence[int] = ()) -> List[List[int]]:
        """Greedy continuation of every prompt (token ids): at most max_new tokens each, up to and including a stop token."""
        m = self.model
        self._runs += 1
        jobs = [Generation(list(p), int(max_new), frozenset(stop), key=("generate", self._runs, i)) for i, p in enumerate(prompts)]
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
                    self._mixed_step(prefilling, running)
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

    def _mixed_step(self, prefilling: List[Generation], running: List[Generation]) -> None:
        """One step of the running sequences' next tokens and, in the room that is left, portions of prompts; prompts that
        end in it get their first token."""
        parts, wanted, enders, at = [], [], [], 0
        for j, tokens in [(j, j.out[-1:]) for j in running] + [(j, j.prompt[j.fed:]) for j in prefilling]:
            tokens = tokens[:self.portion - at]
            if not tokens:
                continue
            r = self.live[j.key]
            parts.append((r.slot, r.length, tokens))
            r.length += len(tokens)
            at += len(tokens)
            if j.fed < len(j.prompt):
                j.fed += len(tokens)
            if j.fed == len(j.prompt):
                wanted.append(at - 1)
                enders.append(j)
        for j, t in zip(enders, self.model.run_greedy(parts, wanted)):
            j.out.append(t)

    def _decode_step(self, jobs: List[Generation]) -> None:
        n = len(jobs)
        d = self._decoders.get(n)
        if d is None:
            d = self._decoders[n] = self.model.decoder(n)
        if self._loaded.get(n) != tuple((j.key, len(j.out)) for j in jobs):
            d.load([(self.live[j.key].slot, self.live[j.key].length, j.out[-1]) for j in jobs])
        d.run()
        for j, t in zip(jobs, d.tokens()):
            self.live[j.key].length += 1
            j.out.append(t)
        self._loaded[n] = tuple((j.key, len(j.out)) for j in jobs)

    def close(self) -> None:
        for d in self._decoders.values():
            d.free()
        self._decoders = {}


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
            if i == 0:
                m.set_position(0)          # every step advances it
            if i < n:
                m.set_tokens([p[i] for p in rows])     # (waits until torch's writes have landed)
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
