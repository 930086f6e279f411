"""Plain, slow restatement of the Bubotar layers: numpy, one function per mechanism, 64-bit by default.

Nothing here is shared with the package.  Arrays are [tokens, channels]; linear weights are [out, in].  Mixers take and
return what they carry from one portion of a sequence to the next, so that a test can cut a sequence anywhere.
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


def rotate_pairs(x, pos, base):
    """x [T, ..., dims] at positions pos [T]: (x[2i], x[2i+1]) turned by the angle pos * base^(-2i / dims)."""
    dims = x.shape[-1]
    out = np.empty_like(x)
    for i in range(dims // 2):
        a = pos * float(base) ** (-2.0 * i / dims)
        c, s = np.cos(a), np.sin(a)
        shape = (len(pos),) + (1,) * (x.ndim - 2)
        c, s = c.reshape(shape), s.reshape(shape)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i], out[..., 2 * i + 1] = u * c - v * s, v * c + u * s
    return out


def softmax(s):
    """Along the last axis; -inf entries get nothing."""
    e = np.exp(s - np.max(s, axis=-1, keepdims=True))
    return e / np.sum(e, axis=-1, keepdims=True)


# ---- latent attention --------------------------------------------------------------------------------------------
def latent_keys(h, W, p, eps, pos):
    """The latents [T, kv_rank] and the rotated key parts [T, rot_dim] that a layer with its own projection caches."""
    both = h @ W["dkv"].T
    c = rms_norm(both[:, :p["kv_rank"]], W["dkv.norm"], eps)
    return c, rotate_pairs(both[:, p["kv_rank"]:], pos, p["rot"]["base"])


def latent_heads(h, W, p, c, kr, pos):
    """Heads [T, H, vdim] of queries at positions pos over the latents c and key parts kr of positions 0 .. len(c) - 1."""
    T, H, D, R, V = len(h), p["heads"], p["dim"], p["rot_dim"], p["vdim"]
    q = (h @ W["q"].T).reshape(T, H, D + R)
    qn, qr = q[..., :D], rotate_pairs(q[..., D:], pos, p["rot"]["base"])
    k = (c @ W["uk"].T).reshape(len(c), H, D)
    v = (c @ W["uv"].T).reshape(len(c), H, V)
    seen = np.arange(len(c))[None, :] <= pos[:, None]
    out = np.zeros((T, H, V), h.dtype)
    for i in range(H):
        s = (qn[:, i] @ k[:, i].T + qr[:, i] @ kr.T) * p["scale"]
        out[:, i] = softmax(np.where(seen, s, -np.inf)) @ v[:, i]
    return out


def latent_mixer(h, W, p, eps, carried, pos0, source: Optional[dict] = None):
    """carried: the latents and key parts so far, of a layer of its own; `source`: the (already advanced) carried dict of
    the layer whose latents this one uses."""
    T = len(h)
    pos = np.arange(pos0, pos0 + T)
    if source is None:
        c, kr = latent_keys(h, W, p, eps, pos)
        carried = {"c": np.concatenate([carried["c"], c]), "kr": np.concatenate([carried["kr"], kr])}
        source = carried
    o = latent_heads(h, W, p, source["c"], source["kr"], pos).reshape(T, -1)
    return (o * sigmoid(h @ W["g"].T)) @ W["o"].T, carried


def latent_start(p, dtype=F):
    return {"c": np.zeros((0, p["kv_rank"]), dtype), "kr": np.zeros((0, p["rot_dim"]), dtype)}


# ---- chunked attention with a distance bias ------------------------------------------------------------------------
def slopes(heads):
    return np.array([2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)])


def chunk_visible(i, j, size):
    """Whether position i sees position j."""
    return (j <= i) & (i // size == j // size)


def attention(q, k, v, pos0, scale, size):
    """q [T, H, dim] at positions pos0 ..; k [P, G, dim], v [P, G, vdim] of positions 0 .. P - 1 = pos0 + T - 1."""
    T, H = q.shape[:2]
    rep = H // k.shape[1]
    m = slopes(H)
    out = np.zeros((T, H, v.shape[2]), q.dtype)
    i, j = np.arange(T)[:, None] + pos0, np.arange(len(k))[None, :]
    for h in range(H):
        s = (q[:, h] @ k[:, h // rep].T) * scale - m[h] * (i - j)
        out[:, h] = softmax(np.where(chunk_visible(i, j, size), s, -np.inf)) @ v[:, h // rep]
    return out


def attention_mixer(h, W, p, carried, pos0):
    T = len(h)
    H, G, D, V = p["heads"], p["kv_heads"], p["dim"], p["vdim"]
    q = (h @ W["q"].T).reshape(T, H, D)
    k = np.concatenate([carried["k"], (h @ W["k"].T).reshape(T, G, D)])
    v = np.concatenate([carried["v"], (h @ W["v"].T).reshape(T, G, V)])
    o = attention(q, k, v, pos0, p["scale"], p["mask"]["size"])
    return o.reshape(T, H * V) @ W["o"].T, {"k": k, "v": v}


def attention_start(p, dtype=F):
    return {"k": np.zeros((0, p["kv_heads"], p["dim"]), dtype), "v": np.zeros((0, p["kv_heads"], p["vdim"]), dtype)}


# ---- selective scan ------------------------------------------------------------------------------------------------
def short_conv(x, taps_w, bias, carried):
    """x [T, C]; taps_w [C, taps], last column for the current token; carried [taps - 1, C] (oldest first).
    Returns (silu of the convolution, the inputs to carry on)."""
    taps = taps_w.shape[1]
    full = np.concatenate([carried, x], axis=0)
    y = np.zeros_like(x)
    for t in range(len(x)):
        for j in range(taps):
            y[t] += taps_w[:, j] * full[t + j]
    return silu(y + bias), full[len(full) - (taps - 1):]


def selective_scan(x, dt, B, C, A, D, state):
    """x, dt [T, channels]; B, C [T, states]; A, state [channels, states]."""
    S = state.copy()
    y = np.zeros_like(x)
    for t in range(len(x)):
        S = np.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t][None, :]
        y[t] = S @ C[t] + D * x[t]
    return y, S


def mamba_mixer(h, W, p, carried):
    inner, R, N = p["inner"], p["dt_rank"], p["state"]
    xz = h @ W["in"].T
    x, conv = short_conv(xz[:, :inner], W["conv"], W["conv.b"], carried["conv"])
    low = x @ W["x"].T
    dt = softplus(low[:, :R] @ W["dt"].T + W["dt.b"])
    y, S = selective_scan(x, dt, low[:, R:R + N], low[:, R + N:], -np.exp(W["A_log"]), W["D"], carried["S"])
    return (y * silu(xz[:, inner:])) @ W["o"].T, {"conv": conv, "S": S}


def mamba_start(p, dtype=F):
    return {"conv": np.zeros((p["conv"] - 1, p["inner"]), dtype), "S": np.zeros((p["inner"], p["state"]), dtype)}


# ---- feed-forward ------------------------------------------------------------------------------------------------
def dense_ff(h, W, limit):
    g = np.minimum(h @ W["gate"].T, limit)
    u = np.clip(h @ W["up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ W["down"].T


# ---- the model ---------------------------------------------------------------------------------------------------
def below(weights: Dict[str, np.ndarray], prefix: str) -> Dict[str, np.ndarray]:
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


START = {"latent_attention": latent_start, "attention": attention_start, "mamba1": mamba_start}


class Model:
    """config: the parsed configuration; weights: name -> array."""

    def __init__(self, config, weights, dtype=F):
        self.c, self.dtype = config, dtype
        self.w = {k: np.asarray(v, dtype) for k, v in weights.items()}

    def start(self):
        return {"pos": 0, "layers": [START[L["type"]](L["mixer"], self.dtype) for L in self.c["layers"]]}

    def forward(self, tokens, carried, taps: Optional[list] = None):
        """Logits [T, vocab] of `tokens`, which follow what `carried` has seen; `carried` is advanced.  taps: the residual
        stream after every layer is appended to it."""
        c, w, pos0 = self.c, self.w, carried["pos"]
        eps = c["norm"]["eps"]
        x = w["embed"][np.asarray(tokens)]
        state = carried["layers"]
        for i, L in enumerate(c["layers"]):
            P, p = f"l{i}.", L["mixer"]
            M = below(w, P + "mix.")
            h = rms_norm(x, w[P + "norm1"], eps)
            if L["type"] == "latent_attention":
                src = p.get("kv_from")
                y, state[i] = latent_mixer(h, M, p, eps, state[i], pos0, None if src is None else state[src])
            elif L["type"] == "attention":
                y, state[i] = attention_mixer(h, M, p, state[i], pos0)
            else:
                y, state[i] = mamba_mixer(h, M, p, state[i])
            x = x + rms_norm(y, w[P + "norm1b"], eps)
            if L.get("mlp"):
                y = dense_ff(rms_norm(x, w[P + "norm2"], eps), below(w, P + "mlp."), L["mlp"]["limit"])
                x = x + rms_norm(y, w[P + "norm2b"], eps)
            if taps is not None:
                taps.append(x.copy())
        carried["pos"] = pos0 + len(tokens)
        return rms_norm(x, w["final.norm"], eps) @ w["head"].T * c["logit_scale"]
