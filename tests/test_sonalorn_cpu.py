"""The Sonalorn oracle against itself and by hand, the host side of the framework around the model (configuration, container,
slots, scheduler, registry), and the boundary of libperegrine_b200_lm.  No GPU."""
import ctypes as C
import json
import math
import os
import re
import subprocess
import sys

import numpy as np
import pytest

from oracle import sonalorn_oracle as so
from peregrine_b200 import safetensors_file
from peregrine_b200.engine import Engine, LockstepEngine, RequestError
from peregrine_b200.sonalorn import SonalornConfig
from peregrine_b200.state import OutOfSlots, SlotPool
from tests import _sonalorn as t

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


# ---- the oracle --------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("make", [t.small_config, t.other_config])
def test_oracle_portions_equal_whole(make):
    cfg = make()
    m = so.Model(cfg, t.weights(cfg, 3))
    tokens = np.random.Generator(np.random.PCG64(5)).integers(0, cfg["vocab"], 41).tolist()
    whole = m.forward(tokens, m.start())
    for cuts in ([1] * 41, [2, 3, 5, 1, 1, 17, 12], [40, 1]):
        state, at, out = m.start(), 0, []
        for n in cuts:
            out.append(m.forward(tokens[at:at + n], state))
            at += n
        assert np.abs(np.concatenate(out) - whole).max() < 1e-9


def test_oracle_pieces_by_hand():
    # one token, one channel: S = beta k v, o = S q
    o, S = so.delta_recurrence(np.array([[[2.0]]]), np.array([[[3.0]]]), np.array([[[5.0]]]), np.array([[0.25]]), np.array([[0.5]]), np.zeros((1, 1, 1)))
    assert S[0, 0, 0] == 7.5 and o[0, 0, 0] == 15.0
    # a second token: decayed state 1.875, u = 0.5 (1 - 1.875 * 3), S = 1.875 + 3 u
    o, S = so.delta_recurrence(np.array([[[1.0]]]), np.array([[[3.0]]]), np.array([[[1.0]]]), np.array([[0.25]]), np.array([[0.5]]), S)
    assert abs(S[0, 0, 0] - (1.875 + 3 * 0.5 * (1 - 5.625))) < 1e-12 and o[0, 0, 0] == S[0, 0, 0]
    y, carry = so.short_conv(np.array([[1.0], [2.0]]), np.array([[10.0, 1.0, 0.5]]), np.array([[3.0], [4.0]]))
    assert np.allclose(y[:, 0], so.silu(np.array([30.0 + 4 + 0.5, 40.0 + 1 + 1]))) and carry[:, 0].tolist() == [1.0, 2.0]
    assert np.allclose(so.sink_softmax(np.array([0.0, math.log(2.0)])), [0.25, 0.5])
    assert np.allclose(so.query_temperature(np.array([0, 6, 7, 15]), 0.5, 8), 1 + 0.5 * np.log([1, 1, 2, 3]))
    # choice: the correction chooses but does not weigh; a negative choice score beats a group that is out
    z = np.log(np.array([0.4, 0.3, 0.2, 0.1]))
    idx, w = so.route(z, np.array([-1.0, 0.0, 0.0, 0.5]), 1, None)
    assert idx.tolist() == [3] and np.allclose(w, [0.1])
    idx, w = so.route(z, np.array([-1.0, -1.0, -2.0, -2.0]), 2, {"count": 2, "keep": 1})
    assert sorted(idx.tolist()) == [0, 1] and np.allclose(sorted(w), [0.3, 0.4])
    assert np.allclose(so.expert_ff(np.array([[1.0]]), {"gate": np.array([[9.0]]), "up": np.array([[-9.0]]), "down": np.array([[1.0]])}, 2.0),
                       2.0 * so.sigmoid(3.404) * (-1.0))


# ---- container and configuration -----------------------------------------------------------------------------------
def test_safetensors_round_trip_and_damage(tmp_path):
    p = str(tmp_path / "x.safetensors")
    a = {"w": t.to_bits(np.array([[1.0, -2.5], [3.0, 0.1]], np.float32)), "i": np.array([1, -2], np.int32), "f": np.array([0.5], np.float32)}
    safetensors_file.write(p, a, bf16=("w",))
    f = safetensors_file.SafetensorsFile(p)
    assert sorted(f) == ["f", "i", "w"] and f.dtype("w") == "BF16" and f.shape("w") == (2, 2) and "w" in f
    for k in a:
        assert np.array_equal(f[k], a[k])
    raw = open(p, "rb").read()
    open(p, "wb").write(raw[:-2])
    with pytest.raises(ValueError):
        safetensors_file.SafetensorsFile(p)
    open(p, "wb").write(b"\xff" * 8 + raw)
    with pytest.raises(ValueError):
        safetensors_file.SafetensorsFile(p)


def test_config():
    c = SonalornConfig.from_dict(t.small_config())
    assert (c.vocab, c.width, c.max_positions, c.eps, len(c.layers)) == (83, 96, 300, 1e-5, 4)
    d = t.small_config()
    d["layers"].append(dict(d["layers"][1], weights_of=2))
    assert [SonalornConfig.from_dict(d).tensors_of(i) for i in range(5)] == [0, 1, 1, 3, 1]
    for change in (lambda d: d["layers"][0].update(type="window"), lambda d: d["layers"][0]["mlp"].update(kind="none"),
                   lambda d: d["layers"][2].update(weights_of=2), lambda d: d["layers"][2].update(weights_of=0), lambda d: d["layers"][2].update(weights_of=9)):
        d = t.small_config()
        change(d)
        with pytest.raises(ValueError):
            SonalornConfig.from_dict(d)


def test_registry_names_what_it_knows(tmp_path):
    from peregrine_b200 import registry

    (tmp_path / "config.json").write_text(json.dumps({"architecture": "Unheard"}))
    with pytest.raises(ValueError, match="Sonalorn"):
        registry.load_engine(str(tmp_path))
    assert "llama" in registry.FILES


# ---- slots and scheduling, with a model that runs on the host --------------------------------------------------------
class HostModel:
    """Next token = (sum of the sequence's tokens so far + its length) mod vocab, from what each slot has been fed."""

    vocab, capacity, step_rows = 50, 64, 16

    def __init__(self, slots):
        self.pool = SlotPool(slots, self.capacity, "cpu")
        self.seen = [[] for _ in range(slots)]
        self.log = []

    def _feed(self, entries):
        self.log.append([(s, len(x)) for s, _p, x in entries])
        rows = []
        for slot, pos, tokens in entries:
            if pos == 0:
                self.seen[slot] = []
            assert len(self.seen[slot]) == pos
            for x in tokens:
                self.seen[slot].append(x)
                rows.append((sum(self.seen[slot]) + len(self.seen[slot])) % self.vocab)
        assert len(rows) <= self.step_rows
        return rows

    def run(self, entries, wanted):
        rows = self._feed(entries)
        return np.array([[float(v == rows[w]) for v in range(self.vocab)] for w in wanted], np.float32).reshape(len(wanted), self.vocab)

    def run_greedy(self, entries, wanted):
        rows = self._feed(entries)
        return [rows[w] for w in wanted]

    def decoder(self, n):
        model = self

        class D:
            def load(self, entries):
                self.e = [list(e) for e in entries]

            def run(self):
                nxt = model._feed([(s, p, [x]) for s, p, x in self.e])
                self.e = [[s, p + 1, x] for (s, p, _), x in zip(self.e, nxt)]

            def tokens(self):
                return [e[2] for e in self.e]

            def free(self):
                pass
        return D()


def _continue(prompt, n, vocab=50, stop=()):
    seq, out = list(prompt), []
    while len(out) < n and not (out and out[-1] in stop):
        out.append((sum(seq) + len(seq)) % vocab)
        seq.append(out[-1])
    return out


@pytest.mark.parametrize("slots,portion", [(1, 0), (2, 5), (3, 16), (7, 3)])
def test_engine_generates_what_each_prompt_alone_gives(slots, portion):
    g = np.random.Generator(np.random.PCG64(9))
    prompts = [g.integers(0, 50, n).tolist() for n in (1, 23, 4, 16, 17, 2, 9)]
    for n, stop in ((1, ()), (6, ()), (12, (7, 20, 33))):
        m = HostModel(slots)
        e = Engine(m, portion=portion)
        for _ in range(2):      # slots, decoders and what they hold are used again
            assert e.generate(prompts, n, stop) == [_continue(p, n, stop=stop) for p in prompts]
        assert m.pool.free == slots and not e.live


def test_engine_mixes_prompts_and_decoding():
    m = HostModel(2)
    Engine(m, portion=8).generate([[1, 2], list(range(20))], 6)
    assert [(0, 2), (1, 6)] in m.log and [(0, 1), (1, 7)] in m.log and [(0, 1), (1, 1)] in m.log


def test_engine_steps_and_errors():
    m = HostModel(2)
    e = Engine(m)
    a = list(range(30))
    out = e.step([("a", a, [29, 0, 16, 0])])          # more rows than one step has
    assert out.argmax(1).tolist() == [_continue(a[:k], 1)[0] for k in (30, 1, 17, 1)]
    assert e.step([("b", [5], [])]).shape == (0, 50)
    out = e.step([("b", [6, 7], [1]), ("a", [3], [0])])
    assert out.argmax(1).tolist() == [_continue([5, 6, 7], 1)[0], _continue(a + [3], 1)[0]]
    with pytest.raises(OutOfSlots):
        e.step([("c", [1], [])])
    e.end("b")
    assert e.step([("c", [9], [0])]).argmax(1).tolist() == _continue([9], 1)     # in b's slot
    for entries in ([("a", [], [])], [("a", [50], [])], [("a", [1], [1])], [("a", [1] * 40, [])], [("a", [1], []), ("a", [2], [])]):
        with pytest.raises(RequestError):
            e.step(entries)
    with pytest.raises(RequestError):
        e.generate([[1] * 60], 6)
    assert e.live["a"].length == 31


def test_lockstep_engine_checks_its_prompts():
    class Cfg:
        batch, capacity, vocab = 2, 8, 10

    class Decoder:
        cfg = Cfg()

    e = LockstepEngine(Decoder())
    for prompts, n in (([[1], [1, 2]], 2), ([[1], [1], [1]], 2), ([[1, 2, 3]], 7), ([[11]], 2)):
        with pytest.raises(RequestError):
            e.generate(prompts, n)


# ---- the boundary --------------------------------------------------------------------------------------------------
def test_lm_library_exports_its_header_and_the_shared_part():
    from peregrine_b200 import _lib
    from peregrine_b200.build import ensure_built

    ensure_built("lm")
    text = open(os.path.join(ROOT, "include", "peregrine_b200_lm.h")).read()
    text = re.sub(r"/\*.*?\*/", "", text, flags=re.S)
    declared = sorted(set(re.findall(r"PG_API\s+[\w\s\*]+?\b(pg_\w+)\s*\(", text)))
    assert declared == sorted(_lib.LM_SIGNATURES)
    out = subprocess.run(["nm", "-D", "--defined-only", _lib.LIB_LM_PATH], capture_output=True, text=True, check=True).stdout
    exported = sorted({line.split()[-1] for line in out.splitlines() if line.split() and line.split()[-1].startswith("pg_")})
    assert exported == sorted(declared + _lib.CORE)
    lib = _lib.load("lm")
    assert lib.pg_ctx_sync(None) == _lib.PG_ERR_INVALID and b"null context" in lib.pg_last_error()
    h = C.c_void_p()
    assert lib.pg_linear_wrap(None, None, 1, 64, 1, C.byref(h)) == _lib.PG_ERR_INVALID


def test_command_line_help_and_bad_model(tmp_path):
    run = lambda *a: subprocess.run([sys.executable, "-m", "peregrine_b200", *a], cwd=ROOT, capture_output=True, text=True)
    assert "generate" in run("--help").stdout
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "Unheard"}))
    r = run("generate", "--model", str(tmp_path), "--prompt", "1,2")
    assert r.returncode != 0 and "Unheard" in r.stderr
