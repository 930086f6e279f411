"""Small Sonalorn configurations and random weights for the tests.  Weights are bf16 values: `bits` is what a file holds,
`values` the same numbers as f32 for the oracle."""
import json
import os

import numpy as np


def to_bits(a):
    """f32 -> bf16 bit patterns, round to nearest even."""
    u = np.ascontiguousarray(a, np.float32).view(np.uint32)
    return ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16)


def from_bits(b):
    return (b.astype(np.uint32) << 16).view(np.float32)


def bf16_values(a):
    return from_bits(to_bits(a))


def delta(heads, kv_heads, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def attention(heads, kv_heads, dim, vdim, scale, temp=None):
    p = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if temp:
        p["q_temp"] = {"coef": temp[0], "every": temp[1]}
    return p


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, limit, experts, identity, top, groups=None):
    r = {"experts": experts, "identity": identity, "top": top}
    if groups:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": r}


def layer(kind, mixer, mlp, weights_of=None):
    L = {"type": kind, "mixer": mixer, "mlp": mlp}
    if weights_of is not None:
        L["weights_of"] = weights_of
    return L


def config(vocab, width, layers, eps=1e-5, max_positions=512):
    return {"architecture": "Sonalorn", "vocab": vocab, "width": width, "max_positions": max_positions, "norm": {"eps": eps}, "layers": layers}


def mixer_weights(g, kind, p, width):
    n = lambda *s: g.standard_normal(s).astype(np.float32)
    G, H, D, V = p["kv_heads"], p["heads"], p["dim"], p["vdim"]
    s = width ** -0.5
    if kind == "attention":
        return {"q": n(H * D, width) * s, "k": n(G * D, width) * s, "v": n(G * V, width) * s, "o": n(width, H * V) * (H * V) ** -0.5,
                "q.norm": 1 + 0.3 * n(D), "k.norm": 1 + 0.3 * n(D)}
    return {"q": n(G * D, width) * s, "k": n(G * D, width) * s, "v": n(H * V, width) * s, "g": n(H * V, width) * s, "b": n(H, width) * s,
            "a": n(H, width) * s, "o": n(width, H * V) * (H * V) ** -0.5, "q.conv": n(G * D, p["conv"]) * 0.6, "k.conv": n(G * D, p["conv"]) * 0.6,
            "v.conv": n(H * V, p["conv"]) * 0.6, "A_log": n(H) * 0.7 - 1.5, "dt_bias": n(H) * 0.5 - 1.0, "norm": 1 + 0.3 * n(V)}


def mlp_weights(g, mlp, width):
    n = lambda *s: g.standard_normal(s).astype(np.float32)
    s = width ** -0.5

    def three(F, prefix=""):
        return {prefix + "gate": n(F, width) * s, prefix + "up": n(F, width) * s, prefix + "down": n(width, F) * F ** -0.5}

    if mlp["kind"] == "dense":
        return three(mlp["ff"])
    r = mlp["router"]
    out = {"router": n(r["experts"] + r["identity"], width) * s * 2, "correction": n(r["experts"] + r["identity"]) * 0.1}
    for e in range(r["experts"]):
        out.update(three(mlp["expert"]["ff"], f"e{e}."))
    return out


def weights(cfg, seed=0):
    """name -> f32 array of bf16 values"""
    g = np.random.Generator(np.random.PCG64(seed))
    n = lambda *s: g.standard_normal(s).astype(np.float32)
    N = cfg["width"]
    W = {"embed": n(cfg["vocab"], N), "pos": n(cfg["max_positions"], N) * 0.5, "embed.norm": 1 + 0.2 * n(N), "final.norm": 1 + 0.2 * n(N),
         "head": n(cfg["vocab"], N) * N ** -0.5}
    for i, L in enumerate(cfg["layers"]):
        if L.get("weights_of") is not None:
            continue
        P = f"l{i}."
        W.update({P + "mix." + k: v for k, v in mixer_weights(g, L["type"], L["mixer"], N).items()})
        W[P + "norm1"], W[P + "ls1"] = 1 + 0.2 * n(N), 0.5 + 0.2 * n(N)
        if L["mlp"]:
            W.update({P + "mlp." + k: v for k, v in mlp_weights(g, L["mlp"], N).items()})
            W[P + "norm2"], W[P + "ls2"] = 1 + 0.2 * n(N), 0.5 + 0.2 * n(N)
    return {k: bf16_values(v) for k, v in W.items()}


def save(path, cfg, W):
    from peregrine_b200 import safetensors_file

    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    safetensors_file.write(os.path.join(path, "model.safetensors"), {k: to_bits(v) for k, v in W.items()}, bf16=True)


# widths, head counts and constants differ between the two, and several are odd on purpose
def small_config():
    m = moe(24, 0.8, 6, 3, 2, (3, 2))
    return config(83, 96, [layer("attention", attention(6, 2, 20, 12, 0.3, (0.7, 16)), dense(40)),
                           layer("delta", delta(6, 3, 24, 10, 4), m),
                           layer("delta", delta(6, 3, 24, 10, 4), m, 1),
                           layer("attention", attention(4, 4, 16, 28, 0.25), m)], max_positions=300)


def other_config():
    return config(61, 70, [layer("delta", delta(2, 1, 17, 33, 2), None),
                           layer("attention", attention(5, 1, 36, 36, 0.2, (1.3, 7)), moe(17, 2.5, 5, 0, 3)),
                           layer("attention", attention(5, 1, 36, 36, 0.2, (1.3, 7)), moe(17, 2.5, 5, 0, 3), 1),
                           layer("delta", delta(3, 3, 40, 8, 1), dense(90))], eps=3e-4, max_positions=200)
