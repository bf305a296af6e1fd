"""Plain, slow numpy implementation of the Tofazen design: one function per mechanism, float64 throughout, loops where
loops are clearest.  It shares no code with the package; tests compare the library's kernels and the whole model with it.

Weights come as a dict of float arrays under the checkpoint's tensor names, the configuration as the parsed config.json.
"""
import math

import numpy as np


def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    x = np.asarray(x, np.float64)
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def embed(tokens, start, table, pos_table):
    """Token row plus the learned row of the token's absolute position."""
    return np.stack([table[t] + pos_table[start + i] for i, t in enumerate(tokens)]).astype(np.float64)


def visible(i, j, size, keep_first):
    """Whether the query at position i sees the key at position j."""
    if j > i:
        return False
    return i - j < size or j < keep_first


def one_map(q, keys, values, i, scale, size, keep_first):
    """Softmax attention of one query vector at position i over keys [n, dim] at positions 0..n-1 (n = i + 1)."""
    js = [j for j in range(i + 1) if visible(i, j, size, keep_first)]
    s = np.array([float(np.dot(q, keys[j])) * scale for j in js])
    w = np.exp(s - s.max())
    w /= w.sum()
    return sum(wj * values[j] for wj, j in zip(w, js))


def lam(lq1, lk1, lq2, lk2, diff):
    return math.exp(float(np.dot(lq1, lk1))) - math.exp(float(np.dot(lq2, lk2))) + diff


def combine_maps(a1, a2, lam_value, diff, eps):
    """Difference of the two maps' outputs, unit root mean square per head, scaled by 1 - diff."""
    return rms(a1 - lam_value * a2, eps) * (1.0 - diff)


def diff_attention(q, keys, values, start, scale, size, keep_first, lam_value, diff, eps):
    """q [n, H, 2, dim] of positions start .. start+n-1; keys [total, G, 2, dim], values [total, G, vdim] of ALL
    positions 0 .. start+n-1.  Returns [n, H, vdim]."""
    n, H = q.shape[:2]
    G = keys.shape[1]
    out = np.zeros((n, H, values.shape[2]))
    for r in range(n):
        for h in range(H):
            g = h // (H // G)
            a = [one_map(q[r, h, m], keys[:, g, m], values[:, g], start + r, scale, size, keep_first) for m in (0, 1)]
            out[r, h] = combine_maps(a[0], a[1], lam_value, diff, eps)
    return out


def clamped_glu(gate, up, limit):
    """g = min(gate, limit), u = clamp(up, -limit, limit);  g * sigmoid(1.702 g) * (u + 1)."""
    g = np.minimum(gate, limit)
    u = np.clip(up, -limit, limit)
    return g / (1.0 + np.exp(-1.702 * g)) * (u + 1.0)


class Tofazen:
    """A sequence's state is {layer: (keys, values)} of every layer that projects its own."""

    def __init__(self, config, weights):
        self.c, self.w = config, {k: np.asarray(v, np.float64) for k, v in weights.items()}

    def new_state(self):
        return {"n": 0, "kv": {}}

    def attention(self, i, h, state):
        m = self.c["layers"][i]["mixer"]
        H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        p = f"l{i}.mix."
        start, n = state["n"], h.shape[0]
        q = (h @ self.w[p + "q"].T).reshape(n, H, 2, D)
        src = m.get("kv_from")
        if src is None:
            k = (h @ self.w[p + "k"].T).reshape(n, G, 2, D)
            v = (h @ self.w[p + "v"].T).reshape(n, G, V)
            if i in state["kv"]:
                k, v = np.concatenate([state["kv"][i][0], k]), np.concatenate([state["kv"][i][1], v])
            state["kv"][i] = (k, v)
        else:
            k, v = state["kv"][src]
        lv = lam(*(self.w[p + x] for x in ("lq1", "lk1", "lq2", "lk2")), m["diff"])
        mask = m["mask"]
        o = diff_attention(q, k, v, start, m["scale"], mask["size"], mask["keep_first"], lv, m["diff"], self.c["norm"]["eps"])
        return o.reshape(n, H * V) @ self.w[p + "o"].T

    def feed_forward(self, i, h):
        mlp = self.c["layers"][i]["mlp"]
        if mlp is None:
            return 0.0
        p = f"l{i}.mlp."
        return clamped_glu(h @ self.w[p + "gate"].T, h @ self.w[p + "up"].T, mlp["limit"]) @ self.w[p + "down"].T

    def forward(self, tokens, state, trace=None):
        """Logits [n, vocab] of the next tokens of one sequence; `trace` (a list) receives the stream after every layer."""
        eps = self.c["norm"]["eps"]
        x = embed(tokens, state["n"], self.w["embed"], self.w["pos"])
        for i in range(len(self.c["layers"])):
            h = rms(x, eps) * self.w[f"l{i}.norm1"]
            x = x + self.c["residual_mult"] * (self.attention(i, h, state) + self.feed_forward(i, h))
            if trace is not None:
                trace.append(x.copy())
        state["n"] += len(tokens)
        return (rms(x, eps) * self.w["final.norm"]) @ self.w["head"].T
