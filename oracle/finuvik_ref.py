"""Plain float64 statement of the Finuvik decoder, one function per mechanism, for tests.

Everything here works on one sequence at a time with numpy loops and no caching tricks; it shares no code with the
CUDA engine.  `weights` is a dict tensor-name -> array ([out, in] projections), `config` the parsed config.json.
"""
from __future__ import annotations

import json
import os
import struct

import numpy as np


# ---- files -------------------------------------------------------------------------------------------------
def bf16_to_f32(u16):
    return (u16.astype(np.uint32) << 16).view(np.float32)


def f32_to_bf16_bits(x):
    """Round to nearest even; finite inputs."""
    u = np.ascontiguousarray(x, np.float32).view(np.uint32).astype(np.uint64)
    return ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16)


def round_bf16(x):
    return bf16_to_f32(f32_to_bf16_bits(x)).reshape(np.shape(x))


def read_safetensors(path):
    with open(path, "rb") as f:
        n = struct.unpack("<Q", f.read(8))[0]
        head = json.loads(f.read(n))
        data = f.read()
    out = {}
    for name, t in head.items():
        if name == "__metadata__":
            continue
        b, e = t["data_offsets"]
        kind = {"BF16": np.uint16, "F32": np.float32, "I32": np.int32}[t["dtype"]]
        a = np.frombuffer(data[b:e], kind)
        out[name] = (bf16_to_f32(a) if t["dtype"] == "BF16" else a).reshape(t["shape"])
    return out


def save_model(folder, config, weights):
    """config.json and model.safetensors (bfloat16) of a test model."""
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(config, f)
    head, blobs, off = {}, [], 0
    for name, a in weights.items():
        raw = f32_to_bf16_bits(a).tobytes()
        head[name] = {"dtype": "BF16", "shape": list(np.shape(a)), "data_offsets": [off, off + len(raw)]}
        blobs.append(raw)
        off += len(raw)
    h = json.dumps(head).encode()
    with open(os.path.join(folder, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(h)) + h + b"".join(blobs))


# ---- mechanisms --------------------------------------------------------------------------------------------
def zero_centred_rms_norm(x, w, eps):
    """Rows of x scaled to unit root mean square, times (1 + w)."""
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps) * (1.0 + w)


def plain_rms_norm(x, w, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps) * w


def query_temperature(pos, coef, every):
    """Factor on the queries of a position: grows with the logarithm of the number of completed blocks."""
    return 1.0 + coef * np.log(np.floor((pos + 1) / every) + 1.0)


def distance_penalty(dist, r1, r2):
    """What a head takes off the score of a key `dist` positions back."""
    return r1 * np.log(1.0 + r2 * dist)


def biased_attention(q, k, v, pos_q, scale, r1, r2, coef, every):
    """q [T, H, d] at positions pos_q over k [S, G, d], v [S, G, e] at positions 0..S-1 -> [T, H, e]."""
    T, H, _ = q.shape
    group = H // k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    for t in range(T):
        p = int(pos_q[t])
        for h in range(H):
            g = h // group
            s = k[:p + 1, g] @ (q[t, h] * query_temperature(p, coef, every)) * scale
            s = s - distance_penalty(p - np.arange(p + 1), r1[h], r2[h])
            w = np.exp(s - s.max())
            out[t, h] = (w / w.sum()) @ v[:p + 1, g]
    return out


def sigmoid(x):
    return np.where(x >= 0, 1.0 / (1.0 + np.exp(-np.abs(x))), np.exp(-np.abs(x)) / (1.0 + np.exp(-np.abs(x))))


def forget_gate(z, lower):
    """z: projection plus bias; a sigmoid squeezed into [lower, 1]."""
    return lower + (1.0 - lower) * sigmoid(z)


def gated_recurrence(q, f, v, state):
    """q, f [T, H, d], v [T, H, e], state [H, d, e] (changed in place) -> [T, H, e].

    The state decays per channel by f and takes (1 - f) of the value; the query reads it after the update."""
    out = np.zeros(v.shape)
    for t in range(q.shape[0]):
        for h in range(q.shape[1]):
            state[h] = f[t, h][:, None] * state[h] + (1.0 - f[t, h])[:, None] * v[t, h][None, :]
            out[t, h] = q[t, h] @ state[h]
    return out


def relu_glu(h, gate, up, down):
    return (np.maximum(h @ gate.T, 0.0) * (h @ up.T)) @ down.T


# ---- the model ---------------------------------------------------------------------------------------------
class FinuvikRef:
    """One sequence: keys, values and recurrent states are kept per layer run, so that feeding tokens in any
    portions continues where the last call stopped."""

    def __init__(self, config, weights):
        self.c = config
        self.w = {n: np.asarray(a, np.float64) for n, a in weights.items()}
        self.reset()

    def reset(self):
        self.pos = 0
        self.mem = [dict() for _ in self.c["layers"]]

    def _mixer(self, i, pre, m, h, pos):
        w, mem = self.w, self.mem[i]
        T = h.shape[0]
        a = m["left"]
        p = pre + ".mix.left."
        q = (h @ w[p + "q"].T).reshape(T, a["heads"], a["dim"])
        k = (h @ w[p + "k"].T).reshape(T, a["kv_heads"], a["dim"])
        v = (h @ w[p + "v"].T).reshape(T, a["kv_heads"], a["vdim"])
        mem["k"] = k = np.concatenate([mem["k"], k]) if "k" in mem else k
        mem["v"] = v = np.concatenate([mem["v"], v]) if "v" in mem else v
        left = biased_attention(q, k, v, pos, a["scale"], w[p + "r1"], w[p + "r2"], a["q_temp"]["coef"], a["q_temp"]["every"])
        left = left.reshape(T, -1) @ w[p + "o"].T
        b = m["right"]
        p = pre + ".mix.right."
        q = h @ w[p + "q"].T
        q = (q * sigmoid(q)).reshape(T, b["heads"], b["dim"])
        f = forget_gate(h @ w[p + "f"].T + w[p + "f.b"], w[p + "lower"]).reshape(T, b["heads"], b["dim"])
        v = (h @ w[p + "v"].T).reshape(T, b["heads"], b["vdim"])
        state = mem.setdefault("s", np.zeros((b["heads"], b["dim"], b["vdim"])))
        o = gated_recurrence(q, f, v, state)
        o = plain_rms_norm(o, w[p + "norm"], self.c["norm"]["eps"])
        right = o.reshape(T, -1) @ w[p + "o"].T
        return m["left_scale"] * left + m["right_scale"] * right

    def forward(self, tokens, want_layers=False):
        """Logits of every given token ([T, vocab]); with want_layers also the stream behind every layer."""
        w, eps = self.w, self.c["norm"]["eps"]
        tokens = np.asarray(tokens)
        pos = self.pos + np.arange(len(tokens))
        self.pos += len(tokens)
        x = w["embed"][tokens] + w["pos"][pos]
        seen = []
        for i, layer in enumerate(self.c["layers"]):
            pre = "l%d" % layer.get("weights_of", i)
            y = self._mixer(i, pre, layer["mixer"], zero_centred_rms_norm(x, w[pre + ".norm1"], eps), pos)
            if layer.get("mlp"):
                h = zero_centred_rms_norm(x, w[pre + ".norm2"], eps)
                y = y + relu_glu(h, w[pre + ".mlp.gate"], w[pre + ".mlp.up"], w[pre + ".mlp.down"])
            x = x + y
            seen.append(x)
        logits = zero_centred_rms_norm(x, w["final.norm"], eps) @ w["head"].T
        return (logits, np.stack(seen)) if want_layers else logits
