"""Plain, slow numpy implementation of the Numuzen design: one function per mechanism, float64 throughout, loops where
loops are clearest.  It shares no code with the package; tests compare the library's kernels and the whole model with it.

Weights come as a dict of float arrays under the checkpoint's tensor names, the configuration as the parsed config.json.
"""
import math

import numpy as np


def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    x = np.asarray(x, np.float64)
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def norm(x, w, eps):
    """The layers' norm: its weight is stored as the distance from one."""
    return rms(x, eps) * (1.0 + w)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-np.asarray(z, np.float64)))


def frequencies(rot):
    """(frequency of every rotated pair, factor on cosine and sine)."""
    dims, base, sc = rot["dims"], rot["base"], rot.get("scaling")
    f = np.array([base ** (-2.0 * i / dims) for i in range(dims // 2)])
    if not sc:
        return f, 1.0
    where = lambda turns: dims * math.log(sc["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
    lo = max(math.floor(where(sc["fast"])), 0)
    hi = min(math.ceil(where(sc["slow"])), dims - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / sc["factor"] * ramp + fi * (1 - ramp))
    return np.array(out), 0.1 * math.log(sc["factor"]) + 1.0


def rotate(x, pos, rot):
    """x [heads, dim] at one position: dimension i of a head turns with dimension i + dims/2, the rest stays."""
    f, mult = frequencies(rot)
    n = rot["dims"] // 2
    c, s = np.cos(pos * f) * mult, np.sin(pos * f) * mult
    u, v = x[:, :n].copy(), x[:, n:2 * n].copy()
    out = np.array(x, np.float64)
    out[:, :n], out[:, n:2 * n] = u * c - v * s, v * c + u * s
    return out


def visible(i, j, size):
    """Whether the query at position i sees the key at position j."""
    return 0 <= i - j < size


def one_query(q, keys, values, i, scale, softcap, size, sink=0.0):
    """One query vector at position i over keys and values at positions 0 .. i: scores capped unless softcap is 0, and a sink
    of the given score (None: none) in the denominator."""
    js = [j for j in range(max(0, i - size + 1), i + 1) if visible(i, j, size)]
    s = keys[js] @ q * scale
    if softcap:
        s = softcap * np.tanh(s / softcap)
    m = s.max() if sink is None else max(s.max(), sink)
    w = np.exp(s - m)
    return (w / (w.sum() + (0.0 if sink is None else np.exp(sink - m)))) @ values[js]


def attention(q, keys, values, start, scale, softcap, size, sink=0.0):
    """q [n, H, dim] of positions start ..; keys [total, G, dim], values [total, G, vdim] of all positions.  [n, H, vdim]."""
    n, H = q.shape[:2]
    G = keys.shape[1]
    return np.array([[one_query(q[r, h], keys[:, h // (H // G)], values[:, h // (H // G)], start + r, scale, softcap, size, sink)
                      for h in range(H)] for r in range(n)])


def gla(q, k, v, alpha, S):
    """Gated linear attention of one head: q, k, alpha [n, dim], v [n, vdim], state S [dim, vdim].  Returns (o, S)."""
    out = np.zeros((len(q), v.shape[1]))
    for t in range(len(q)):
        S = alpha[t][:, None] * S + np.outer(k[t], v[t])
        out[t] = S.T @ q[t]
    return out, S


def decay(z, tau):
    """sigmoid(z) ** (1 / tau)"""
    return sigmoid(z) ** (1.0 / tau)


def clamped_glu(gate, up, limit):
    g = np.minimum(gate, limit)
    u = np.clip(up, -limit, limit)
    return g * sigmoid(1.702 * g) * (u + 1.0)


def choose(z, top):
    """(experts, weights) of one token from its router logits: the largest sigmoid scores, used as they are."""
    s = sigmoid(z)
    e = sorted(range(len(s)), key=lambda i: (-s[i], i))[:top]
    return e, [s[i] for i in e]


class Numuzen:
    """A sequence's state: {layer: (keys, values)} of attention layers, {layer: [H, dim, vdim]} of recurrent ones."""

    def __init__(self, config, weights):
        self.c, self.w = config, {k: np.asarray(v, np.float64) for k, v in weights.items()}
        self.eps = config["norm"]["eps"]

    def new_state(self):
        return {"n": 0, "kv": {}, "S": {}}

    def attention_layer(self, i, h, state):
        m, p = self.c["layers"][i]["mixer"], f"l{i}.mix."
        H, G, D = m["heads"], m["kv_heads"], m["dim"]
        start, n = state["n"], len(h)
        q, k = h @ self.w[p + "q"].T, h @ self.w[p + "k"].T
        v = k.reshape(n, G, D)
        q = (rms(q, self.eps) * self.w[p + "q.norm"]).reshape(n, H, D)
        k = (rms(k, self.eps) * self.w[p + "k.norm"]).reshape(n, G, D)
        q = np.array([rotate(q[r], start + r, m["rot"]) for r in range(n)])
        k = np.array([rotate(k[r], start + r, m["rot"]) for r in range(n)])
        if i in state["kv"]:
            k, v = np.concatenate([state["kv"][i][0], k]), np.concatenate([state["kv"][i][1], v])
        state["kv"][i] = (k, v)
        o = attention(q, k, v, start, m["scale"], m["softcap"], m["mask"]["size"]).reshape(n, H * D)
        return (o * sigmoid(h @ self.w[p + "g"].T)) @ self.w[p + "o"].T

    def gla_layer(self, i, h, state):
        m, p = self.c["layers"][i]["mixer"], f"l{i}.mix."
        H, D, V, n = m["heads"], m["dim"], m["vdim"], len(h)
        q = (h @ self.w[p + "q"].T * D ** -0.5).reshape(n, H, D)
        k = (h @ self.w[p + "k"].T).reshape(n, H, D)
        v = (h @ self.w[p + "v"].T).reshape(n, H, V)
        z = (h @ self.w[p + "a1"].T) @ self.w[p + "a2"].T + self.w[p + "a2.b"]
        a = decay(z, m["tau"]).reshape(n, H, D)
        S = state["S"].get(i, np.zeros((H, D, V)))
        o, S2 = np.zeros((n, H, V)), S.copy()
        for hd in range(H):
            o[:, hd], S2[hd] = gla(q[:, hd], k[:, hd], v[:, hd], a[:, hd], S[hd])
        state["S"][i] = S2
        o = (rms(o, self.eps) * self.w[p + "norm"]).reshape(n, H * V)
        g = h @ self.w[p + "g"].T
        return (o * g * sigmoid(g)) @ self.w[p + "o"].T

    def experts(self, i, h):
        mlp, p = self.c["layers"][i]["mlp"], f"l{i}.mlp."
        out = np.zeros_like(h)
        for r, x in enumerate(h):
            for e, s in zip(*choose(self.w[p + "router"] @ x, mlp["router"]["top"])):
                y = s * x
                out[r] += self.w[p + f"e{e}.down"] @ clamped_glu(self.w[p + f"e{e}.gate"] @ y, self.w[p + f"e{e}.up"] @ y, mlp["expert"]["limit"])
        return out

    def forward(self, tokens, state, trace=None):
        """Logits [n, vocab] of the next tokens of one sequence; `trace` (a list) receives the stream after every layer."""
        x = self.w["embed"][list(tokens)]
        for i, layer in enumerate(self.c["layers"]):
            w = lambda name: self.w[f"l{i}.{name}"]
            mixer = self.attention_layer if layer["type"] == "attention" else self.gla_layer
            x = x + norm(mixer(i, norm(x, w("norm1"), self.eps), state), w("norm1b"), self.eps)
            if layer.get("mlp"):
                x = x + norm(self.experts(i, norm(x, w("norm2"), self.eps)), w("norm2b"), self.eps)
            if trace is not None:
                trace.append(x.copy())
        state["n"] += len(tokens)
        return norm(x, self.w["final.norm"], self.eps) @ self.w["embed"].T
