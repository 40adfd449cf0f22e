"""Plain float64 statement of the Fuposun decoder, one function per mechanism, for tests.

One sequence at a time, numpy loops, no absorbed projections, no ring buffers and no sorting of tokens by expert: latents
are kept from the first token on and keys and values are formed from them anew.  It shares no code with the CUDA engine.
`weights` is a dict tensor-name -> array ([out, in] projections), `config` the parsed config.json.
"""
from __future__ import annotations

import numpy as np

from oracle.finuvik_ref import plain_rms_norm, sigmoid


def silu(x):
    return x * sigmoid(x)


# ---- attention over latents --------------------------------------------------------------------------------
def visible(i, j, size):
    """A query at position i sees the key at position j: itself and the size - 1 positions before it."""
    return 0 <= i - j < size


def latent_attention(q, c, uk, uv, pos_q, pos_c, scale, size):
    """q [T, H, d] at positions pos_q over the latents c [S, r] at positions pos_c; uk [H * d, r] and uv [H * e, r] turn a
    latent into the keys and values of all heads -> [T, H, e]."""
    T, H, d = q.shape
    k = (c @ uk.T).reshape(len(c), H, d)
    v = (c @ uv.T).reshape(len(c), H, -1)
    out = np.zeros((T, H, v.shape[2]))
    for t in range(T):
        seen = [n for n in range(len(c)) if visible(pos_q[t], pos_c[n], size)]
        for h in range(H):
            s = k[seen, h] @ q[t, h] * scale
            w = np.exp(s - s.max())
            out[t, h] = (w / w.sum()) @ v[seen, h]
    return out


# ---- gated linear attention --------------------------------------------------------------------------------
def channel_decay(z, tau):
    """sigmoid(z) ** (1 / tau)"""
    return np.exp(-np.logaddexp(0.0, -z) / tau)


def gated_linear_attention(q, k, v, alpha, state):
    """q, k, alpha [T, H, d], v [T, H, e], state [H, d, e] (changed in place) -> [T, H, e].

    The rows of the state (key channels) decay by alpha, then the outer product of key and value comes on top; the query
    reads the new state."""
    out = np.zeros(v.shape)
    for t in range(q.shape[0]):
        for h in range(q.shape[1]):
            state[h] = alpha[t, h][:, None] * state[h] + np.outer(k[t, h], v[t, h])
            out[t, h] = state[h].T @ q[t, h]
    return out


# ---- feed-forward ------------------------------------------------------------------------------------------
def swiglu(h, gate, up, down):
    return (silu(h @ gate.T) * (h @ up.T)) @ down.T


def clamped_glu(g, u, limit):
    """Gate bounded from above, up value from both sides and moved up by one."""
    g = np.minimum(g, limit)
    u = np.clip(u, -limit, limit)
    return g * sigmoid(1.702 * g) * (u + 1.0)


def expert(x, gate, up, down, limit):
    return clamped_glu(x @ gate.T, x @ up.T, limit) @ down.T


def route(h, router, top):
    """Chosen experts [T, top], best first (the lower number on a tie), and their weights: the scores as they are."""
    s = sigmoid(h @ router.T)
    chosen = np.argsort(-s, axis=1, kind="stable")[:, :top]
    return chosen, np.take_along_axis(s, chosen, 1)


def mixture(h, router, top, experts, limit):
    """experts: list of (gate, up, down).  The weight of an expert multiplies what goes into it."""
    chosen, weight = route(h, router, top)
    y = np.zeros((h.shape[0], experts[0][2].shape[0]))
    for t in range(h.shape[0]):
        for e, w in zip(chosen[t], weight[t]):
            y[t] += expert((w * h[t])[None], *experts[e], limit)[0]
    return y


# ---- the model ---------------------------------------------------------------------------------------------
class FuposunRef:
    """One sequence: latents and recurrent states are kept per layer, so that feeding tokens in any portions continues
    where the last call stopped."""

    def __init__(self, config, weights):
        self.c = config
        self.w = {n: np.asarray(a, np.float64) for n, a in weights.items()}
        self.reset()

    def reset(self):
        self.margins = []  # per forward call and token: how close the closest choice of experts was, in logits
        self.pos = 0
        self.mem = [dict() for _ in self.c["layers"]]

    def _latent_attention(self, p, m, mem, h, pos):
        w, eps = self.w, self.c["norm"]["eps"]
        T, H = len(h), m["heads"]
        q = plain_rms_norm(h @ w[p + "dq"].T, w[p + "dq.norm"], eps) @ w[p + "uq"].T
        c = plain_rms_norm(h @ w[p + "dkv"].T, w[p + "dkv.norm"], eps)
        mem["c"] = c = np.concatenate([mem["c"], c]) if "c" in mem else c
        o = latent_attention(q.reshape(T, H, m["dim"]), c, w[p + "uk"], w[p + "uv"], pos, np.arange(len(c)), m["scale"], m["mask"]["size"])
        o = o * sigmoid(h @ w[p + "g"].T)[:, :, None]
        return o.reshape(T, -1) @ w[p + "o"].T

    def _gla(self, p, m, mem, h):
        w, eps = self.w, self.c["norm"]["eps"]
        T, H, d, e = len(h), m["heads"], m["dim"], m["vdim"]
        q = (h @ w[p + "q"].T).reshape(T, H, d) * d ** -0.5
        k = (h @ w[p + "k"].T).reshape(T, H, d)
        v = (h @ w[p + "v"].T).reshape(T, H, e)
        z = (h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "a2.b"]
        state = mem.setdefault("s", np.zeros((H, d, e)))
        o = gated_linear_attention(q, k, v, channel_decay(z, m["tau"]).reshape(T, H, d), state)
        o = plain_rms_norm(o, w[p + "norm"], eps).reshape(T, -1)
        return (o * silu(h @ w[p + "g"].T)) @ w[p + "o"].T

    def _feed_forward(self, p, m, h):
        w = self.w
        parts = lambda name: (w[p + name + "gate"], w[p + name + "up"], w[p + name + "down"])
        if m["kind"] == "dense":
            return swiglu(h, *parts(""))
        r = m["router"]
        if r["top"] < r["experts"]:
            z = -np.sort(-(h @ w[p + "router"].T), 1)
            self.margins[-1] = np.minimum(self.margins[-1], z[:, r["top"] - 1] - z[:, r["top"]])
        y = mixture(h, w[p + "router"], r["top"], [parts(f"e{n}.") for n in range(r["experts"])], m["expert"]["limit"])
        return y + expert(h, *parts("shared."), m["shared"]["limit"])

    def forward(self, tokens, want_layers=False):
        """Logits of every given token ([T, vocab]); with want_layers also the stream behind every layer."""
        w, eps, mult = self.w, self.c["norm"]["eps"], self.c["residual_mult"]
        tokens = np.asarray(tokens)
        pos = self.pos + np.arange(len(tokens))
        self.pos += len(tokens)
        self.margins.append(np.full(len(tokens), np.inf))
        x = plain_rms_norm(w["embed"][tokens], w["embed.norm"], eps)
        seen = []
        for i, layer in enumerate(self.c["layers"]):
            p = f"l{i}."
            h = plain_rms_norm(x, w[p + "norm1"], eps)
            if layer["type"] == "gla":
                y = self._gla(p + "mix.", layer["mixer"], self.mem[i], h)
            else:
                y = self._latent_attention(p + "mix.", layer["mixer"], self.mem[i], h, pos)
            x = x + mult * y
            if layer.get("mlp"):
                x = x + mult * self._feed_forward(p + "mlp.", layer["mlp"], plain_rms_norm(x, w[p + "norm2"], eps))
            seen.append(x)
        cap = self.c["logit_softcap"]
        logits = cap * np.tanh(plain_rms_norm(x, w["final.norm"], eps) @ w["head"].T / cap)
        return (logits, np.stack(seen)) if want_layers else logits
