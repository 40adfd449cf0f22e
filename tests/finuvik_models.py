"""Small Finuvik models for the tests: configurations and random weights."""
import numpy as np


def layer(left=(6, 2, 24, 40), right=(3, 16, 24), ff=72, scale=0.21, temp=(0.4, 16), scales=(0.9, 1.1), weights_of=None):
    """left = (heads, kv_heads, dim, vdim), right = (heads, dim, vdim); ff None: no feed-forward."""
    e = {"type": "parallel",
         "mixer": {"left": {"heads": left[0], "kv_heads": left[1], "dim": left[2], "vdim": left[3], "scale": scale,
                            "q_temp": {"coef": temp[0], "every": temp[1]}},
                   "left_scale": scales[0], "right_scale": scales[1],
                   "right": {"heads": right[0], "dim": right[1], "vdim": right[2]}},
         "mlp": None if ff is None else {"kind": "dense", "ff": ff}}
    if weights_of is not None:
        e["weights_of"] = weights_of
    return e


def config(layers, vocab=203, width=88, max_positions=320, eps=1e-5):
    return {"architecture": "Finuvik", "vocab": vocab, "width": width, "max_positions": max_positions, "norm": {"eps": eps},
            "layers": layers}


def weights(cfg, seed=0):
    """Random weights, already rounded to bfloat16; every mechanism has a visible share of the result."""
    from oracle.finuvik_ref import round_bf16
    rng = np.random.default_rng(seed)
    W = cfg["width"]
    lin = lambda o, i, g=1.0: g * rng.standard_normal((o, i)) / np.sqrt(i)
    w = {"embed": rng.standard_normal((cfg["vocab"], W)), "pos": 0.5 * rng.standard_normal((cfg["max_positions"], W))}
    for n, l in enumerate(cfg["layers"]):
        if l.get("weights_of") is not None:
            continue
        a, b = l["mixer"]["left"], l["mixer"]["right"]
        p = f"l{n}."
        w[p + "norm1"], w[p + "norm2"] = 0.3 * rng.standard_normal(W), 0.3 * rng.standard_normal(W)
        m = p + "mix.left."
        w[m + "q"] = lin(a["heads"] * a["dim"], W, 1.5)
        w[m + "k"] = lin(a["kv_heads"] * a["dim"], W, 1.5)
        w[m + "v"] = lin(a["kv_heads"] * a["vdim"], W)
        w[m + "r1"] = rng.uniform(0.0, 1.5, a["heads"])
        w[m + "r2"] = rng.uniform(0.02, 0.6, a["heads"])
        w[m + "o"] = lin(W, a["heads"] * a["vdim"], 1.3)
        m = p + "mix.right."
        n_k = b["heads"] * b["dim"]
        w[m + "q"], w[m + "f"], w[m + "v"] = lin(n_k, W), lin(n_k, W, 2.0), lin(b["heads"] * b["vdim"], W)
        w[m + "f.b"] = rng.uniform(-1.0, 7.0, n_k)
        w[m + "lower"] = rng.uniform(0.0, 0.9, n_k) * (rng.uniform(size=n_k) > 0.2)
        w[m + "norm"] = 1.0 + 0.3 * rng.standard_normal(b["vdim"])
        w[m + "o"] = lin(W, b["heads"] * b["vdim"])
        if l["mlp"]:
            ff = l["mlp"]["ff"]
            w[p + "mlp.gate"], w[p + "mlp.up"], w[p + "mlp.down"] = lin(ff, W), lin(ff, W), lin(W, ff)
    w["final.norm"] = 0.3 * rng.standard_normal(W)
    w["head"] = lin(cfg["vocab"], W)
    return {n: round_bf16(a) for n, a in w.items()}


# two layers of unequal sizes, none of them padded evenly; the third run shares the weights of the first, one has no
# feed-forward
ODD = config([layer(), layer(left=(5, 5, 8, 56), right=(2, 40, 72), ff=None, scale=0.3, temp=(0.0, 1), scales=(0.5, 1.0)),
              layer(weights_of=0)])
# aligned sizes, one key/value head, sizes that meet the kernels' tile sizes exactly
EVEN = config([layer(left=(8, 1, 64, 64), right=(2, 64, 32), ff=128, scale=0.125, temp=(0.25, 32), scales=(1.0, 1.0)),
               layer(left=(4, 2, 128, 128), right=(1, 128, 96), ff=192, scale=0.09, temp=(0.5, 100), scales=(1.3, 0.6))],
              vocab=256, width=192, max_positions=512)
