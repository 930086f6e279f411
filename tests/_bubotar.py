"""Small Bubotar configurations and random weights for the tests.  Weights are bf16 values, as a file holds them."""
import numpy as np

from tests._sonalorn import bf16_values, save, to_bits  # noqa: F401  (used through this module)


def latent(heads, dim, rot_dim, vdim, kv_rank, scale, base=10000.0, kv_from=None):
    p = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale, "rot": {"base": base, "dims": rot_dim}}
    if kv_from is not None:
        p["kv_from"] = kv_from
    return p


def attention(heads, kv_heads, dim, vdim, scale, size):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": size}}


def mamba(inner, state, dt_rank, conv):
    return {"inner": inner, "state": state, "dt_rank": dt_rank, "conv": conv}


def dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def layer(kind, mixer, mlp):
    return {"type": kind, "mixer": mixer, "mlp": mlp}


def config(vocab, width, layers, eps=1e-5, logit_scale=1.0):
    return {"architecture": "Bubotar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_scale": logit_scale, "layers": layers}


def mixer_weights(g, kind, p, width):
    n = lambda *s: g.standard_normal(s).astype(np.float32)
    s = width ** -0.5
    if kind == "mamba1":
        I, N, R = p["inner"], p["state"], p["dt_rank"]
        return {"in": n(2 * I, width) * s, "conv": n(I, p["conv"]) * p["conv"] ** -0.5, "conv.b": n(I) * 0.3, "x": n(R + 2 * N, I) * I ** -0.5 * 1.5,
                "dt": n(I, R) * R ** -0.5, "dt.b": n(I) - 1.0, "A_log": n(I, N) * 0.7, "D": 1 + 0.3 * n(I), "o": n(width, I) * I ** -0.5}
    H, D, V = p["heads"], p["dim"], p["vdim"]
    if kind == "attention":
        G = p["kv_heads"]
        return {"q": n(H * D, width) * s * 2, "k": n(G * D, width) * s, "v": n(G * V, width) * s, "o": n(width, H * V) * (H * V) ** -0.5}
    R, K = p["rot_dim"], p["kv_rank"]
    out = {"q": n(H * (D + R), width) * s * 2, "uk": n(H * D, K) * K ** -0.5, "uv": n(H * V, K) * K ** -0.5, "g": n(H * V, width) * s,
           "o": n(width, H * V) * (H * V) ** -0.5}
    if p.get("kv_from") is None:
        out.update({"dkv": n(K + R, width) * s, "dkv.norm": 1 + 0.2 * n(K)})
    return out


def mlp_weights(g, mlp, width):
    n = lambda *s: g.standard_normal(s).astype(np.float32)
    F = mlp["ff"]
    return {"gate": n(F, width) * width ** -0.5 * 1.5, "up": n(F, width) * width ** -0.5 * 1.5, "down": n(width, F) * F ** -0.5}


def weights(cfg, seed=0):
    """name -> f32 array of bf16 values"""
    g = np.random.Generator(np.random.PCG64(seed))
    n = lambda *s: g.standard_normal(s).astype(np.float32)
    N = cfg["width"]
    W = {"embed": n(cfg["vocab"], N), "final.norm": 1 + 0.2 * n(N), "head": n(cfg["vocab"], N) * N ** -0.5}
    for i, L in enumerate(cfg["layers"]):
        P = f"l{i}."
        W.update({P + "mix." + k: v for k, v in mixer_weights(g, L["type"], L["mixer"], N).items()})
        W[P + "norm1"], W[P + "norm1b"] = 1 + 0.2 * n(N), 0.6 + 0.2 * n(N)
        if L["mlp"]:
            W.update({P + "mlp." + k: v for k, v in mlp_weights(g, L["mlp"], N).items()})
            W[P + "norm2"], W[P + "norm2b"] = 1 + 0.2 * n(N), 0.6 + 0.2 * n(N)
    return {k: bf16_values(v) for k, v in W.items()}


# widths, head counts and constants differ between the models, and several are odd on purpose; in the last, prompts run on the
# tcgen05 attention kernel and the widths are whole multiples
def small_config():
    lat = (6, 20, 6, 12, 40)
    return config(83, 96, [layer("latent_attention", latent(*lat, 0.25, 500.0), dense(40, 0.9)),
                           layer("mamba1", mamba(72, 5, 7, 3), None),
                           layer("attention", attention(6, 2, 20, 12, 0.3, 11), dense(24, 1.7)),
                           layer("latent_attention", latent(4, 33, 6, 17, 40, 0.2, 500.0, 0), None),
                           layer("mamba1", mamba(40, 18, 3, 4), dense(50, 0.6))], eps=2e-4, logit_scale=1.5)


def other_config():
    return config(61, 70, [layer("attention", attention(5, 5, 9, 36, 0.4, 40), None),
                           layer("latent_attention", latent(17, 8, 2, 5, 70, 0.35), dense(33, 2.5)),
                           layer("latent_attention", latent(3, 16, 2, 40, 70, 0.3, kv_from=1), dense(90, 1.1)),
                           layer("mamba1", mamba(130, 33, 66, 2), dense(17, 3.0)),
                           layer("mamba1", mamba(17, 1, 1, 1), None)], eps=1e-6, logit_scale=0.4)


def even_config():
    return config(120, 128, [layer("mamba1", mamba(192, 16, 8, 4), None),
                             layer("latent_attention", latent(4, 64, 32, 64, 128, 0.1, 3000.0), dense(72, 1.4)),
                             layer("attention", attention(4, 2, 64, 128, 0.12, 48), dense(136, 2.0)),
                             layer("latent_attention", latent(2, 128, 32, 96, 128, 0.08, 3000.0, 1), None)], logit_scale=3.0)


CONFIGS = [small_config, other_config, even_config]
