"""The Bubotar oracle against itself and by hand, the model's configuration, and its place in the registry.  No GPU."""
import json
import math

import numpy as np
import pytest

from oracle import bubotar_oracle as bo
from peregrine_b200.bubotar import BubotarConfig
from peregrine_b200.layers import halving_slopes
from tests import _bubotar as t


@pytest.mark.parametrize("make", t.CONFIGS)
def test_oracle_portions_equal_whole(make):
    cfg = make()
    m = bo.Model(cfg, t.weights(cfg, 3))
    tokens = np.random.Generator(np.random.PCG64(5)).integers(0, cfg["vocab"], 53).tolist()
    whole = m.forward(tokens, m.start())
    for cuts in ([1] * 53, [2, 3, 5, 1, 1, 17, 24], [52, 1]):
        state, at, out = m.start(), 0, []
        for n in cuts:
            out.append(m.forward(tokens[at:at + n], state))
            at += n
        assert np.abs(np.concatenate(out) - whole).max() < 1e-9


def test_oracle_rotation_and_scores_by_hand():
    x = np.array([[1.0, 2.0, 3.0, 4.0]])
    y = bo.rotate_pairs(x, np.array([2]), 100.0)[0]
    a, b = 2.0, 2.0 * 100.0 ** -0.5
    want = [math.cos(a) - 2 * math.sin(a), 2 * math.cos(a) + math.sin(a), 3 * math.cos(b) - 4 * math.sin(b), 4 * math.cos(b) + 3 * math.sin(b)]
    assert np.allclose(y, want)
    # a rotation depends on the distance only
    q, k = np.random.Generator(np.random.PCG64(1)).standard_normal((2, 1, 8))
    dots = [bo.rotate_pairs(q, np.array([p]), 50.0)[0] @ bo.rotate_pairs(k, np.array([p - 3]), 50.0)[0] for p in (3, 10, 999)]
    assert np.allclose(dots, dots[0])
    assert np.allclose(bo.slopes(4), [2.0 ** -2, 2.0 ** -4, 2.0 ** -6, 2.0 ** -8]) and np.allclose(bo.slopes(6), halving_slopes(6))
    i, j = np.arange(7)[:, None], np.arange(7)[None, :]
    seen = bo.chunk_visible(i, j, 3)
    assert seen.sum(1).tolist() == [1, 2, 3, 1, 2, 3, 1] and seen[4, 3] and not seen[3, 2] and not seen[3, 4]
    # equal scores, so the weights come from the distance alone: one head has the slope 2^-8
    q, k, v = np.zeros((3, 1, 1)), np.zeros((3, 1, 1)), np.array([1.0, 0.0, 0.0]).reshape(3, 1, 1)
    s = 2.0 ** -8
    e = [math.exp(-2 * s), math.exp(-s), 1.0]
    assert np.allclose(bo.attention(q, k, v, 0, 1.0, 8)[2, 0, 0], e[0] / sum(e))


def test_oracle_scan_and_feed_forward_by_hand():
    # one channel, one state: S = dt x B, then decayed
    y, S = bo.selective_scan(np.array([[2.0], [3.0]]), np.array([[0.5], [1.0]]), np.array([[4.0], [1.0]]), np.array([[10.0], [1.0]]), np.array([[-1.0]]),
                             np.array([0.25]), np.zeros((1, 1)))
    assert np.allclose(y[:, 0], [40.5, 4.0 * math.exp(-1.0) + 3.0 + 0.75]) and np.allclose(S, 4.0 * math.exp(-1.0) + 3.0)
    y, carry = bo.short_conv(np.array([[1.0], [2.0]]), np.array([[10.0, 1.0, 0.5]]), np.array([0.125]), np.array([[3.0], [4.0]]))
    assert np.allclose(y[:, 0], bo.silu(np.array([30.0 + 4 + 0.5, 40.0 + 1 + 1]) + 0.125)) and carry[:, 0].tolist() == [1.0, 2.0]
    one = lambda v: np.array([[v]])
    for g, u in ((9.0, -9.0), (-9.0, 9.0), (0.5, 0.25)):
        gg, uu = min(g, 2.0), max(-2.0, min(2.0, u))
        got = bo.dense_ff(one(1.0), {"gate": one(g), "up": one(u), "down": one(1.0)}, 2.0)
        assert np.allclose(got, gg / (1 + math.exp(-1.702 * gg)) * (uu + 1.0))


def test_config():
    c = BubotarConfig.from_dict(t.small_config())
    assert (c.vocab, c.width, c.eps, c.logit_scale, len(c.layers)) == (83, 96, 2e-4, 1.5, 5)
    for change in (lambda d: d["layers"][0].update(type="window"), lambda d: d["layers"][0]["mlp"].update(kind="moe"),
                   lambda d: d["layers"][3]["mixer"].update(kv_from=3), lambda d: d["layers"][3]["mixer"].update(kv_from=1),
                   lambda d: d["layers"][3]["mixer"].update(kv_rank=39), lambda d: d["layers"][3]["mixer"].update(rot={"base": 501.0, "dims": 6}),
                   lambda d: d["layers"].append(dict(d["layers"][3], mixer=dict(d["layers"][3]["mixer"], kv_from=3)))):
        d = json.loads(json.dumps(t.small_config()))
        change(d)
        with pytest.raises(ValueError):
            BubotarConfig.from_dict(d)


def test_registry_knows_the_design(tmp_path):
    from peregrine_b200 import registry

    assert "Bubotar" in registry.FOLDERS
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "Unheard"}))
    with pytest.raises(ValueError, match="Bubotar"):
        registry.load_engine(str(tmp_path))
