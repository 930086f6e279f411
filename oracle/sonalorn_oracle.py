"""Plain, slow restatement of the Sonalorn layers: numpy, one function per mechanism, 64-bit by default.

Nothing here is shared with the package.  Arrays are [tokens, channels]; linear weights are [out, in].  Recurrences and
attention take and return what they carry from one portion of a sequence to the next, so that a test can cut a
sequence anywhere.
"""
from __future__ import annotations

import math
from typing import Dict, Optional

import numpy as np

F = np.float64


# ---- elementwise pieces ------------------------------------------------------------------------------------------
def rms_norm(x, w, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * w


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def embed(tokens, pos0, table, pos_table, norm_w, eps):
    t = np.asarray(tokens)
    return rms_norm(table[t] + pos_table[pos0:pos0 + len(t)], norm_w, eps)


# ---- gated delta rule --------------------------------------------------------------------------------------------
def short_conv(x, taps_w, carried):
    """x [T, C]; taps_w [C, taps], last column for the current token; carried [taps - 1, C] (oldest first).
    Returns (silu of the convolution, the inputs to carry on)."""
    taps = taps_w.shape[1]
    full = np.concatenate([carried, x], axis=0)
    y = np.zeros_like(x)
    for t in range(len(x)):
        for j in range(taps):
            y[t] += taps_w[:, j] * full[t + j]
    return silu(y), full[len(full) - (taps - 1):]


def unit(x):
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + 1e-6)


def decay(a, a_log, dt_bias):
    return np.exp(-np.exp(a_log) * softplus(a + dt_bias))


def delta_recurrence(q, k, v, g, beta, state):
    """q, k [T, G, dim]; v [T, H, vdim]; g, beta [T, H]; state [H, dim, vdim]."""
    T, H = v.shape[0], v.shape[1]
    rep = H // q.shape[1]
    S = state.copy()
    o = np.zeros(v.shape, v.dtype)
    for t in range(T):
        for h in range(H):
            kk, qq = k[t, h // rep], q[t, h // rep]
            S[h] = g[t, h] * S[h]
            u = beta[t, h] * (v[t, h] - S[h].T @ kk)
            S[h] = S[h] + np.outer(kk, u)
            o[t, h] = S[h].T @ qq
    return o, S


def delta_mixer(h, W, p, eps, carried):
    """W: the tensors below the layer's `mix.`; carried: dict with q, k, v (convolution inputs) and S."""
    T = len(h)
    G, H, D, V = p["kv_heads"], p["heads"], p["dim"], p["vdim"]
    nxt = {}
    q, nxt["q"] = short_conv(h @ W["q"].T, W["q.conv"], carried["q"])
    k, nxt["k"] = short_conv(h @ W["k"].T, W["k.conv"], carried["k"])
    v, nxt["v"] = short_conv(h @ W["v"].T, W["v.conv"], carried["v"])
    q = unit(q.reshape(T, G, D)) * D ** -0.5
    k = unit(k.reshape(T, G, D))
    beta = sigmoid(h @ W["b"].T)
    g = decay(h @ W["a"].T, W["A_log"], W["dt_bias"])
    o, nxt["S"] = delta_recurrence(q, k, v.reshape(T, H, V), g, beta, carried["S"])
    o = rms_norm(o, W["norm"], eps) * silu(h @ W["g"].T).reshape(T, H, V)
    return o.reshape(T, H * V) @ W["o"].T, nxt


def delta_start(p, dtype=F):
    G, H, D, V, n = p["kv_heads"], p["heads"], p["dim"], p["vdim"], p["conv"] - 1
    return {"q": np.zeros((n, G * D), dtype), "k": np.zeros((n, G * D), dtype), "v": np.zeros((n, H * V), dtype), "S": np.zeros((H, D, V), dtype)}


# ---- attention ---------------------------------------------------------------------------------------------------
def query_temperature(pos, coef, every):
    return 1.0 + coef * np.log(np.floor((pos + 1) / every) + 1.0)


def sink_softmax(s):
    """exp(s_j) / (1 + sum exp(s_j)) along the last axis; -inf entries get nothing."""
    m = np.maximum(np.max(s, axis=-1, keepdims=True), 0.0)
    e = np.exp(s - m)
    return e / (np.exp(-m) + np.sum(e, axis=-1, keepdims=True))


def attention(q, k, v, pos0, scale):
    """q [T, H, dim] at positions pos0 ..; k [P, G, dim], v [P, G, vdim] of positions 0 .. P - 1 = pos0 + T - 1."""
    T, H = q.shape[:2]
    rep = H // k.shape[1]
    out = np.zeros((T, H, v.shape[2]), q.dtype)
    for h in range(H):
        s = (q[:, h] @ k[:, h // rep].T) * scale
        i, j = np.arange(T)[:, None] + pos0, np.arange(len(k))[None, :]
        out[:, h] = sink_softmax(np.where(j <= i, s, -np.inf)) @ v[:, h // rep]
    return out


def attention_mixer(h, W, p, eps, carried, pos0):
    T = len(h)
    H, G, D, V = p["heads"], p["kv_heads"], p["dim"], p["vdim"]
    q = rms_norm((h @ W["q"].T).reshape(T, H, D), W["q.norm"], eps)
    k = rms_norm((h @ W["k"].T).reshape(T, G, D), W["k.norm"], eps)
    v = (h @ W["v"].T).reshape(T, G, V)
    if p.get("q_temp"):
        q = q * query_temperature(np.arange(pos0, pos0 + T), p["q_temp"]["coef"], p["q_temp"]["every"])[:, None, None]
    k = np.concatenate([carried["k"], k])
    v = np.concatenate([carried["v"], v])
    o = attention(q, k, v, pos0, p["scale"])
    return o.reshape(T, H * V) @ W["o"].T, {"k": k, "v": v}


def attention_start(p, dtype=F):
    return {"k": np.zeros((0, p["kv_heads"], p["dim"]), dtype), "v": np.zeros((0, p["kv_heads"], p["vdim"]), dtype)}


# ---- feed-forward ------------------------------------------------------------------------------------------------
def dense_ff(h, W):
    return (gelu_tanh(h @ W["gate"].T) * (h @ W["up"].T)) @ W["down"].T


def expert_ff(h, W, limit):
    g = np.minimum(h @ W["gate"].T, limit)
    u = np.clip(h @ W["up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ W["down"].T


def route(z, correction, top, groups: Optional[dict]):
    """One token's router logits [experts + identity] -> (chosen indices, weights)."""
    e = np.exp(z - np.max(z))
    s = e / np.sum(e)
    c = s + correction
    if groups:
        n = len(z) // groups["count"]
        best = np.array([np.max(c[i * n:(i + 1) * n]) for i in range(groups["count"])])
        keep = np.argsort(-best, kind="stable")[:groups["keep"]]
        ok = np.zeros(len(z), bool)
        for i in keep:
            ok[i * n:(i + 1) * n] = True
        c = np.where(ok, c, -np.inf)
    chosen = np.argsort(-c, kind="stable")[:top]
    return chosen, s[chosen]


def moe_ff(h, W, mlp):
    r = mlp["router"]
    z = h @ W["router"].T
    y = np.zeros_like(h)
    for t in range(len(h)):
        idx, w = route(z[t], W["correction"], r["top"], r.get("groups"))
        for e, we in zip(idx, w):
            if e < r["experts"]:
                y[t] += we * expert_ff(h[t:t + 1], {n: W[f"e{e}.{n}"] for n in ("gate", "up", "down")}, mlp["expert"]["limit"])[0]
            else:
                y[t] += we * h[t]
    return y


# ---- the model ---------------------------------------------------------------------------------------------------
def below(weights: Dict[str, np.ndarray], prefix: str) -> Dict[str, np.ndarray]:
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


class Model:
    """config: the parsed configuration; weights: name -> array."""

    def __init__(self, config, weights, dtype=F):
        self.c, self.dtype = config, dtype
        self.w = {k: np.asarray(v, dtype) for k, v in weights.items()}

    def start(self):
        return {"pos": 0, "layers": [(delta_start if L["type"] == "delta" else attention_start)(L["mixer"], self.dtype) for L in self.c["layers"]]}

    def forward(self, tokens, carried, taps: Optional[list] = None):
        """Logits [T, vocab] of `tokens`, which follow what `carried` has seen; `carried` is advanced."""
        c, w, pos0 = self.c, self.w, carried["pos"]
        eps = c["norm"]["eps"]
        x = embed(tokens, pos0, w["embed"], w["pos"], w["embed.norm"], eps)
        for i, L in enumerate(c["layers"]):
            P = f"l{L.get('weights_of', i)}."
            M = below(w, P + "mix.")
            if L["type"] == "delta":
                y, carried["layers"][i] = delta_mixer(x, M, L["mixer"], eps, carried["layers"][i])
            else:
                y, carried["layers"][i] = attention_mixer(x, M, L["mixer"], eps, carried["layers"][i], pos0)
            x = x + rms_norm(y, w[P + "norm1"], eps) * w[P + "ls1"]
            if L.get("mlp"):
                M = below(w, P + "mlp.")
                y = dense_ff(x, M) if L["mlp"]["kind"] == "dense" else moe_ff(x, M, L["mlp"])
                x = x + rms_norm(y, w[P + "norm2"], eps) * w[P + "ls2"]
            if taps is not None:
                taps.append(x.copy())
        carried["pos"] = pos0 + len(tokens)
        return rms_norm(x, w["final.norm"], eps) @ w["head"].T
