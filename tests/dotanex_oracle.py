"""Plain, slow numpy implementation of the Dotanex design: one function per mechanism, float64 throughout, loops where
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


def plain_frequencies(dims, base):
    return np.array([base ** (-2.0 * i / dims) for i in range(dims // 2)])


def banded_frequencies(rot):
    """Stretched by wavelength: short waves stay, long ones are divided by the factor, the band between is blended."""
    sc, out = rot.get("scaling"), []
    for f in plain_frequencies(rot["dims"], rot["base"]):
        if sc:
            wave = 2 * math.pi / f
            if wave > sc["original"] / sc["low"]:
                f = f / sc["factor"]
            elif wave >= sc["original"] / sc["high"]:
                s = (sc["original"] / wave - sc["low"]) / (sc["high"] - sc["low"])
                f = (1 - s) * f / sc["factor"] + s * f
        out.append(f)
    return np.array(out), 1.0


def yarn_frequencies(rot):
    """Stretched by turns over the original context; the second value multiplies cosine and sine."""
    sc, f = rot.get("scaling"), plain_frequencies(rot["dims"], rot["base"])
    if not sc:
        return f, 1.0
    dims = rot["dims"]
    where = lambda turns: dims * math.log(sc["original"] / (2 * math.pi * turns)) / (2 * math.log(rot["base"]))
    lo, hi = max(math.floor(where(sc["fast"])), 0), min(math.ceil(where(sc["slow"])), dims - 1)
    ramp = np.array([min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0) for i in range(dims // 2)])
    return f / sc["factor"] * ramp + f * (1 - ramp), 0.1 * math.log(sc["factor"]) + 1.0


def turn(u, v, pos, freq, mult):
    c, s = np.cos(pos * freq) * mult, np.sin(pos * freq) * mult
    return u * c - v * s, v * c + u * s


def rotate_halves(x, pos, freq, mult=1.0):
    """x [..., dim] at one position: dimension i turns with dimension i + len(freq), the rest stays."""
    out, n = np.array(x, np.float64), len(freq)
    out[..., :n], out[..., n:2 * n] = turn(out[..., :n].copy(), out[..., n:2 * n].copy(), pos, freq, mult)
    return out


def rotate_neighbours(x, pos, freq, mult=1.0):
    """x [..., dim] at one position: dimension 2i turns with dimension 2i + 1, the rest stays."""
    out, n = np.array(x, np.float64), len(freq)
    out[..., 0:2 * n:2], out[..., 1:2 * n:2] = turn(out[..., 0:2 * n:2].copy(), out[..., 1:2 * n:2].copy(), pos, freq, mult)
    return out


def visible(i, j, size):
    """Whether the query at position i sees the key at position j (size None: every earlier key)."""
    return 0 <= i - j and (size is None or i - j < size)


def one_query(q, keys, values, i, scale, size, sink):
    """One query vector at position i over keys and values at positions 0 .. i; a sink (None: none) is one more term of the
    denominator."""
    js = [j for j in range(max(0, i - size + 1) if size else 0, i + 1) if visible(i, j, size)]
    s = keys[js] @ q * scale
    m = s.max() if sink is None else max(s.max(), sink)
    w = np.exp(s - m)
    return (w / (w.sum() + (0.0 if sink is None else np.exp(sink - m)))) @ values[js]


def attention(q, keys, values, start, scale, size=None, sinks=None):
    """q [n, H, dim] of positions start ..; keys [total, G, dim], values [total, G, vdim] of all positions.  [n, H, vdim]."""
    n, H = q.shape[:2]
    G = keys.shape[1]
    return np.array([[one_query(q[r, h], keys[:, h // (H // G)], values[:, h // (H // G)], start + r, scale, size, None if sinks is None else sinks[h])
                      for h in range(H)] for r in range(n)])


def lightning(q, k, v, decay, S):
    """Linear attention of one head with one decay: q, k [n, dim], v [n, vdim], state S [dim, vdim].  Returns (o, S)."""
    out = np.zeros((len(q), v.shape[1]))
    for t in range(len(q)):
        S = decay * S + np.outer(k[t], v[t])
        out[t] = S.T @ q[t]
    return out, S


def gated(gate, up):
    return silu(gate) * up


def clamped_gated(gate, up, limit):
    g = np.minimum(gate, limit)
    u = np.clip(up, -limit, limit)
    return g * sigmoid(1.702 * g) * (u + 1.0)


def choose(z, correction, top):
    """(experts, weights) of one token from its router logits: softmax scores, chosen with the correction and weighed without."""
    s = np.exp(z - z.max())
    s = s / s.sum()
    e = sorted(range(len(s)), key=lambda i: (-(s[i] + correction[i]), i))[:top]
    return e, s[e] / (s[e].sum() + 1e-20)


def read_streams(xs, w_in):
    """xs [streams, n, width] -> the sublayer's input before its norm."""
    return np.tensordot(w_in, xs, 1)


def write_streams(xs, mix, w_out, y):
    """New stream t: the old streams weighed by column t of `mix`, plus the sublayer's output by w_out[t]."""
    return np.array([sum(mix[s, t] * xs[s] for s in range(len(xs))) + w_out[t] * y for t in range(len(xs))])


class Dotanex:
    """A sequence's state: {layer: (keys, values)} or {layer: (latents, rotated parts)} of attention layers, {layer: [H, dim, vdim]}
    of recurrent ones."""

    def __init__(self, config, weights):
        self.c, self.w = config, {k: np.asarray(v, np.float64) for k, v in weights.items()}
        self.eps = config["norm"]["eps"]

    def new_state(self):
        return {"n": 0, "kv": {}, "S": {}}

    def keep(self, i, state, a, b):
        if i in state["kv"]:
            a, b = np.concatenate([state["kv"][i][0], a]), np.concatenate([state["kv"][i][1], b])
        state["kv"][i] = (a, b)
        return a, b

    def attention_layer(self, i, m, w, h, state):
        H, G, D, start, n = m["heads"], m["kv_heads"], m["dim"], state["n"], len(h)
        q, k = (h @ w("q").T).reshape(n, H, D), (h @ w("k").T).reshape(n, G, D)
        v = k
        q, k = rms(q, self.eps) * w("q.norm"), rms(k, self.eps) * w("k.norm")
        f, mult = banded_frequencies(m["rot"])
        q = np.array([rotate_halves(q[r], start + r, f, mult) for r in range(n)])
        k = np.array([rotate_halves(k[r], start + r, f, mult) for r in range(n)])
        k, v = self.keep(i, state, k, v)
        return attention(q, k, v, start, m["scale"], m["mask"]["size"], w("sink")).reshape(n, H * D) @ w("o").T

    def latent_layer(self, i, m, w, h, state):
        H, D, R, V, C, start, n = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], state["n"], len(h)
        q = ((rms(h @ w("dq").T, self.eps) * w("dq.norm")) @ w("uq").T).reshape(n, H, D + R)
        low = h @ w("dkv").T
        c, r = rms(low[:, :C], self.eps) * w("dkv.norm"), low[:, C:]
        f, mult = yarn_frequencies(m["rot"])
        q[:, :, D:] = [rotate_neighbours(q[t, :, D:], start + t, f, mult) for t in range(n)]
        r = np.array([rotate_neighbours(r[t], start + t, f, mult) for t in range(n)])
        c, r = self.keep(i, state, c, r)
        k = np.concatenate([(c @ w("uk").T).reshape(-1, H, D), np.repeat(r[:, None], H, 1)], 2)
        v = (c @ w("uv").T).reshape(-1, H, V)
        o = attention(q, k, v, start, m["scale"]).reshape(n, H * V)
        return (o * sigmoid(h @ w("g").T)) @ w("o").T

    def lightning_layer(self, i, m, w, h, state):
        H, D, V, n = m["heads"], m["dim"], m["vdim"], len(h)
        q, k, v = (silu(h @ w(x).T).reshape(n, H, -1) for x in "qkv")
        S = state["S"].get(i, np.zeros((H, D, V)))
        o, S2 = np.zeros((n, H, V)), S.copy()
        for hd in range(H):
            o[:, hd], S2[hd] = lightning(q[:, hd], k[:, hd], v[:, hd], m["decay"][hd], S[hd])
        state["S"][i] = S2
        return (rms(o.reshape(n, H * V), self.eps) * w("norm") * sigmoid(h @ w("g").T)) @ w("o").T

    def experts(self, mlp, w, h):
        rt, limit = mlp["router"], mlp["expert"]["limit"]
        out = np.zeros_like(h)
        for r, x in enumerate(h):
            for e, s in zip(*choose(w("router") @ x, w("correction"), rt["top"])):
                if e >= rt["experts"]:
                    y = x
                else:
                    y = w(f"e{e}.down") @ clamped_gated(w(f"e{e}.gate") @ x, w(f"e{e}.up") @ x, limit)
                out[r] += s * y
        return out + clamped_gated(h @ w("shared.gate").T, h @ w("shared.up").T, mlp["shared"]["limit"]) @ w("shared.down").T

    def feed_forward(self, mlp, w, h):
        if mlp["kind"] == "dense":
            return gated(h @ w("gate").T, h @ w("up").T) @ w("down").T
        return self.experts(mlp, w, h)

    def forward(self, tokens, state, trace=None):
        """Logits [n, vocab] of the next tokens of one sequence; `trace` (a list) receives the summed streams after every layer."""
        xs = np.array([self.w["embed"][list(tokens)]] * self.c["streams"])
        for i, layer in enumerate(self.c["layers"]):
            src = layer.get("weights_of", i)
            w = lambda name: self.w[f"l{src}.{name}"]
            mixer = {"attention": self.attention_layer, "latent_attention": self.latent_layer, "lightning": self.lightning_layer}[layer["type"]]
            subs = [lambda h: mixer(i, layer["mixer"], lambda n: w("mix." + n), h, state)]
            if layer.get("mlp"):
                subs.append(lambda h: self.feed_forward(layer["mlp"], lambda n: w("mlp." + n), h))
            for q, sub in enumerate(subs, 1):
                h = rms(read_streams(xs, w(f"hc{q}.in")), self.eps) * w(f"norm{q}")
                xs = write_streams(xs, w(f"hc{q}.mix"), w(f"hc{q}.out"), sub(h))
            if trace is not None:
                trace.append(xs.sum(0))
        state["n"] += len(tokens)
        return (rms(xs.sum(0), self.eps) * self.w["final.norm"]) @ self.w["head"].T
