"""Plain, slow numpy implementation of the Sakinex design: one function per mechanism, float64 throughout, loops where
loops are clearest.  It shares no code with the package; tests compare the library's kernels and the whole model with it.

Weights come as a dict of float arrays under the checkpoint's tensor names, the configuration as the parsed config.json.
"""
import math

import numpy as np


def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    x = np.asarray(x, np.float64)
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-np.asarray(z, np.float64)))


def silu(z):
    return z * sigmoid(z)


def conv(rows, w, before):
    """Causal convolution of every channel: rows [n, channels], w [channels, taps], `before` the taps - 1 rows ahead of them.
    Returns (convolved rows, the last taps - 1 rows)."""
    taps = w.shape[1]
    seen = np.concatenate([before, rows])
    out = np.array([sum(w[:, j] * seen[t + j] for j in range(taps)) for t in range(len(rows))])
    return out, seen[len(seen) - (taps - 1):]


def frequencies(rot):
    """(frequency of every pair, factor on cosine and sine), stretched by turns over the original context if there is a scaling."""
    dims, base, sc = rot["dims"], rot["base"], rot.get("scaling")
    f = np.array([base ** (-2.0 * i / dims) for i in range(dims // 2)])
    if not sc:
        return f, 1.0
    where = lambda turns: dims * math.log(sc["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
    lo, hi = max(math.floor(where(sc["fast"])), 0), min(math.ceil(where(sc["slow"])), dims - 1)
    ramp = np.array([min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0) for i in range(dims // 2)])
    return f / sc["factor"] * ramp + f * (1 - ramp), 0.1 * math.log(sc["factor"]) + 1.0


def rotate(x, pos, freq, mult):
    """x [..., dim] at one position: dimension i turns with dimension i + len(freq), the rest stays."""
    out, n = np.array(x, np.float64), len(freq)
    c, s = np.cos(pos * freq) * mult, np.sin(pos * freq) * mult
    u, v = np.array(x[..., :n]), np.array(x[..., n:2 * n])
    out[..., :n], out[..., n:2 * n] = u * c - v * s, v * c + u * s
    return out


def seen_tokens(i, size):
    """Positions that the query at position i sees one by one."""
    return [j for j in range(i + 1) if i - j < size]


def seen_blocks(i, size, pool):
    """Blocks that its window has moved past."""
    return [b for b in range(i // pool + 1) if b * pool + pool - 1 <= i - size]


def pooled(rows, b, pool):
    return rows[b * pool:(b + 1) * pool].mean(0)


def one_query(q, keys, values, i, scale, size, pool):
    """One query vector at position i over keys [.., dim] and values [.., vdim] of positions 0 .. i."""
    js, bs = seen_tokens(i, size), seen_blocks(i, size, pool)
    k = np.concatenate([keys[js], np.array([pooled(keys, b, pool) for b in bs]).reshape(-1, keys.shape[1])])
    v = np.concatenate([values[js], np.array([pooled(values, b, pool) for b in bs]).reshape(-1, values.shape[1])])
    s = k @ q * scale
    p = np.exp(s - s.max())
    return (p / p.sum()) @ v


def attention(q, keys, values, start, scale, size, pool):
    """q [n, H, dim] of positions start ..; keys [total, G, dim], values [total, G, vdim] of all positions.  [n, H, vdim]."""
    n, H = q.shape[:2]
    G = keys.shape[1]
    return np.array([[one_query(q[r, h], keys[:, h // (H // G)], values[:, h // (H // G)], start + r, scale, size, pool) for h in range(H)]
                     for r in range(n)])


def min_gru(z, u, S):
    """Rows of gate logits and candidate inputs, state S.  Returns (the states after every row, the last one)."""
    out = []
    for zt, ut in zip(z, u):
        g = sigmoid(zt)
        S = (1 - g) * S + g * np.where(ut >= 0, ut + 0.5, sigmoid(ut))
        out.append(S)
    return np.array(out), S


def gated(gate, up):
    return silu(gate) * up


def choose(z, top):
    """(experts, weights) of one token from its router logits: the largest ones, weighed by a softmax over themselves."""
    e = sorted(range(len(z)), key=lambda i: (-z[i], i))[:top]
    p = np.exp(z[e] - z[e].max())
    return e, p / p.sum()


class Sakinex:
    """A sequence's state: its length and, by layer run, what every convolution, cache and recurrence holds."""

    def __init__(self, config, weights):
        self.c, self.w = config, {k: np.asarray(v, np.float64) for k, v in weights.items()}
        self.eps = config["norm"]["eps"]
        n, loop = len(config["layers"]), config.get("loop") or {"start": 0, "stop": 0, "times": 1}
        a, b = loop["start"], loop["stop"]
        # (layer, whether the embedding output is added ahead of it)
        self.runs = [(i, False) for i in range(a)]
        for t in range(loop["times"]):
            self.runs += [(i, t > 0 and i == a) for i in range(a, b)]
        self.runs += [(i, False) for i in range(b, n)]

    def new_state(self):
        return {"n": 0}

    def short(self, state, key, rows, w):
        out, state[key] = conv(rows, w, state.get(key, np.zeros((w.shape[1] - 1, rows.shape[1]))))
        return out

    def left(self, run, m, w, h, state):
        H, G, D, V, start, n = m["heads"], m["kv_heads"], m["dim"], m["vdim"], state["n"], len(h)
        q, k, v = (h @ w(x).T for x in "qkv")
        if m.get("conv"):
            q, k, v = (self.short(state, (run, x), r, w(x + ".conv")) for x, r in zip("qkv", (q, k, v)))
        q, k, v = q.reshape(n, H, D), k.reshape(n, G, D), v.reshape(n, G, V)
        if m.get("rot"):
            f, mult = frequencies(m["rot"])
            q = np.array([rotate(q[r], start + r, f, mult) for r in range(n)])
            k = np.array([rotate(k[r], start + r, f, mult) for r in range(n)])
        q, k = rms(q, self.eps), rms(k, self.eps)
        if (run, "kv") in state:
            k, v = np.concatenate([state[run, "kv"][0], k]), np.concatenate([state[run, "kv"][1], v])
        state[run, "kv"] = (k, v)
        o = attention(q, k, v, start, m["scale"], m["mask"]["size"], m["mask"]["pool"])
        return o.reshape(n, H * V) @ w("o").T

    def right(self, run, m, w, h, state):
        S, state[run, "S"] = min_gru(h @ w("z").T + w("z.b"), h @ w("x").T + w("x.b"), state.get((run, "S"), np.zeros(m["width"])))
        return (S * silu(h @ w("g").T)) @ w("o").T

    def mixer(self, run, m, w, h, state):
        left = self.left(run, m["left"], lambda n: w("left." + n), h, state)
        right = self.right(run, m["right"], lambda n: w("right." + n), h, state)
        return m["left_scale"] * left + m["right_scale"] * right

    def experts(self, mlp, w, h):
        out = np.zeros_like(h)
        for r, x in enumerate(h):
            for e, p in zip(*choose(w("router") @ x + w("router.b"), mlp["router"]["top"])):
                out[r] += p * (w(f"e{e}.down") @ gated(w(f"e{e}.gate") @ x, w(f"e{e}.up") @ x))
            if mlp.get("shared"):
                out[r] += sigmoid(w("shared.sg").reshape(-1) @ x) * (w("shared.down") @ gated(w("shared.gate") @ x, w("shared.up") @ x))
        return out

    def forward(self, tokens, state, trace=None):
        """Logits [n, vocab] of the next tokens of one sequence; `trace` (a list) receives the residual stream after every layer run."""
        embedded = self.w["embed"][list(tokens)]
        x, mult = embedded.copy(), self.c["residual_mult"]
        for run, (i, again) in enumerate(self.runs):
            layer = self.c["layers"][i]
            if again:
                x = x + embedded
            w = lambda name: self.w[f"l{i}.{name}"]
            subs = [lambda h: self.mixer(run, layer["mixer"], lambda n: w("mix." + n), h, state)]
            if layer.get("mlp"):
                subs.append(lambda h: self.experts(layer["mlp"], lambda n: w("mlp." + n), h))
            for s, sub in enumerate(subs, 1):
                h = rms(x, self.eps) * w(f"norm{s}")
                h = h + self.short(state, (run, "canon", s), h, w(f"canon{s}"))
                x = x + mult * sub(h)
            if trace is not None:
                trace.append(x.copy())
        state["n"] += len(tokens)
        return (rms(x, self.eps) * self.w["final.norm"]) @ self.w["head"].T
