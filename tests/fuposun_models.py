"""Small Fuposun models for the tests: configurations and random weights."""
import numpy as np


def attention(heads=3, dim=24, vdim=40, q_rank=56, kv_rank=72, window=9, scale=0.4):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale,
                                                  "mask": {"size": window}}}


def gla(heads=2, dim=24, vdim=40, tau=4.0):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}}


def dense(ff=72):
    return {"kind": "dense", "ff": ff}


def moe(experts=7, top=2, ff=40, limit=1.1, shared=56, shared_limit=0.8):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff, "limit": limit},
            "shared": {"ff": shared, "limit": shared_limit}}


def config(layers, vocab=211, width=88, eps=1e-5, mult=0.4, cap=9.0):
    """layers: (mixer, feed-forward or None)"""
    return {"architecture": "Fuposun", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult, "logit_softcap": cap,
            "layers": [dict(m, mlp=f) for m, f in layers]}


def weights(cfg, seed=0, gate_rank=8):
    """Random weights, already rounded to bfloat16; every mechanism has a visible share of the result."""
    from oracle.finuvik_ref import round_bf16
    rng = np.random.default_rng(seed)
    W = cfg["width"]
    lin = lambda o, i, g=1.0: g * rng.standard_normal((o, i)) / np.sqrt(i)
    vec = lambda n: 1.0 + 0.3 * rng.standard_normal(n)
    w = {"embed": rng.standard_normal((cfg["vocab"], W)) * rng.uniform(0.2, 3.0, (cfg["vocab"], 1)), "embed.norm": vec(W)}
    for n, l in enumerate(cfg["layers"]):
        m, f, p = l["mixer"], l["mlp"], f"l{n}."
        H, hk, hv = m["heads"], m["heads"] * m["dim"], m["heads"] * m["vdim"]
        w[p + "norm1"] = vec(W)
        x = p + "mix."
        if l["type"] == "gla":
            w[x + "q"], w[x + "k"], w[x + "v"], w[x + "g"] = lin(hk, W, 1.5), lin(hk, W), lin(hv, W), lin(hv, W)
            w[x + "a1"], w[x + "a2"], w[x + "a2.b"] = lin(gate_rank + n, W), lin(hk, gate_rank + n, 2.0), rng.uniform(-1, 6, hk)
            w[x + "norm"] = vec(m["vdim"])
        else:
            w[x + "dq"], w[x + "dq.norm"], w[x + "uq"] = lin(m["q_rank"], W), vec(m["q_rank"]), lin(hk, m["q_rank"], 1.5)
            w[x + "dkv"], w[x + "dkv.norm"] = lin(m["kv_rank"], W), vec(m["kv_rank"])
            w[x + "uk"], w[x + "uv"], w[x + "g"] = lin(hk, m["kv_rank"], 1.5), lin(hv, m["kv_rank"]), lin(H, W, 1.5)
        w[x + "o"] = lin(W, hv, 2.0)
        if f is None:
            continue
        w[p + "norm2"] = vec(W)
        if f["kind"] == "dense":
            w[p + "mlp.gate"], w[p + "mlp.up"], w[p + "mlp.down"] = lin(f["ff"], W), lin(f["ff"], W), lin(W, f["ff"], 2.0)
            continue
        w[p + "mlp.router"] = lin(f["router"]["experts"], W, 2.0)
        for name, ff in [(f"e{e}", f["expert"]["ff"]) for e in range(f["router"]["experts"])] + [("shared", f["shared"]["ff"])]:
            w[f"{p}mlp.{name}.gate"], w[f"{p}mlp.{name}.up"] = lin(ff, W, 1.5), lin(ff, W, 1.5)
            w[f"{p}mlp.{name}.down"] = lin(W, ff, 1.5)
    w["final.norm"], w["head"] = vec(W), lin(cfg["vocab"], W, 3.0)
    return {n: round_bf16(a) for n, a in w.items()}


# none of the sizes padded evenly, every kind of layer and feed-forward, windows of one and of a few tokens
ODD = config([(attention(), moe()), (gla(), None), (attention(heads=1, dim=56, vdim=16, q_rank=24, kv_rank=40, window=1, scale=0.2), dense()),
              (gla(heads=1, dim=40, vdim=72, tau=9.5), moe(experts=3, top=3, shared_limit=3.0)),
              (attention(heads=5, dim=8, vdim=24, q_rank=88, kv_rank=24, window=70, scale=0.9), None)])
# aligned sizes that meet the kernels' tiles exactly; a window longer than most prompts
EVEN = config([(gla(heads=2, dim=64, vdim=64, tau=1.0), dense(128)),
               (attention(heads=16, dim=64, vdim=64, q_rank=128, kv_rank=256, window=64, scale=0.3), moe(experts=16, top=4, ff=64, shared=128)),
               (attention(heads=2, dim=128, vdim=128, q_rank=64, kv_rank=128, window=250, scale=0.2), moe(experts=8, top=1, ff=128, limit=7.0, shared=64))],
              vocab=256, width=128, mult=0.5, cap=30.0)
# everything that can be one is one
ONES = config([(gla(heads=1, dim=1, vdim=1, tau=1.0), dense(1)), (attention(1, 1, 1, 1, 1, 1, 1.0), moe(1, 1, 1, 1.0, 1, 1.0)),
               (gla(heads=3, dim=5, vdim=7, tau=1.0), moe(2, 1, 3, 0.5, 1, 2.0))], vocab=9, width=8, eps=1e-3, mult=1.0, cap=1.0)
