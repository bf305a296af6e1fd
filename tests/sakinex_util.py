"""Small random Sakinex models, as a configuration and a dict of tensors, for the library and for the numpy implementation."""
import numpy as np

import sakinex_oracle as X
from tofazen_util import row_errors, save, views  # noqa: F401
from util import bf16_round


def moe(experts, top, ff, shared=None):
    out = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}
    if shared:
        out["shared"] = {"ff": shared}
    return out


def layer(heads, kv_heads, dim, vdim, window, pool, state, mlp=None, conv=3, rot=None, base=10000.0, scaling=(4.0, 64, 16.0, 1.0), scale=None, left=0.7, right=1.2):
    sc = None if scaling is None else dict(zip(("factor", "original", "fast", "slow"), scaling))
    rot = dim // 2 * 2 if rot is None else rot
    return {"type": "parallel", "mlp": mlp, "mixer": {
        "left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "mask": {"size": window, "pool": pool},
                 "rot": {"base": base, "dims": rot, "scaling": sc}, "scale": 1.5 * dim ** -0.5 if scale is None else scale},
        "right": {"width": state}, "left_scale": left, "right_scale": right}}


def config(layers, width=72, vocab=101, taps=3, loop=None, mult=0.6, eps=1e-5):
    out = {"architecture": "Sakinex", "canon": {"taps": taps}, "layers": layers, "norm": {"eps": eps}, "residual_mult": mult, "vocab": vocab, "width": width}
    if loop:
        out["loop"] = dict(zip(("start", "stop", "times"), loop))
    return out


# Sizes that differ from layer to layer, odd ones, groups of 1 to 12 heads, one and many taps, no convolution on the heads, no
# rotation, windows below, at and above the 64-key tiles and smaller than a block, blocks of 1 and more tokens than a window, layers
# without a feed-forward or a shared expert, all experts chosen or one of them, loops over the first, the last, one or all layers.
CONFIGS = {
    "mixed": config([layer(6, 2, 20, 24, 17, 4, 50, moe(5, 2, 24, 40)), layer(3, 3, 24, 8, 64, 16, 36, moe(4, 4, 37)), layer(4, 1, 16, 40, 5, 8, 64, None, conv=4, rot=8),
                     layer(6, 2, 20, 24, 33, 3, 24, moe(6, 1, 16, 24), conv=2, scaling=None)], loop=(1, 3, 3)),
    "odd": config([layer(1, 1, 7, 9, 70, 5, 13, moe(3, 3, 11, 13), conv=1, rot=4), layer(5, 1, 33, 51, 9, 2, 37, moe(2, 1, 50), conv=6, rot=10, scale=0.3),
                   layer(4, 4, 9, 5, 1, 1, 1, None, conv=0, rot=0)], width=101, vocab=67, taps=5, loop=(0, 2, 2), eps=1e-3, mult=1.0),
    "aligned": config([layer(12, 1, 16, 16, 40, 8, 128, moe(8, 2, 48, 64), rot=16), layer(4, 2, 64, 32, 100, 20, 96, moe(8, 6, 32, 48), conv=4, rot=32),
                       layer(4, 2, 32, 128, 64, 64, 32, moe(4, 2, 64), conv=2)], width=192, vocab=300, taps=4, loop=(2, 3, 2), mult=0.4),
    "large_heads": config([layer(2, 1, 136, 40, 40, 4, 64, moe(3, 1, 32, 24), rot=64), layer(2, 2, 264, 24, 50, 10, 40), layer(4, 2, 128, 256, 30, 6, 520)],
                          width=128, vocab=64, taps=2, loop=(0, 3, 2), mult=0.5),
}


def weights(cfg, seed):
    """Random tensors by name, rounded to bf16.  The routers read channels of the stream of their own: only the embedding writes them,
    in well separated products with the routers' orthonormal rows, and nothing of the neighbours is mixed into them, so the order of a
    layer's logits is never a close call in any number format.  A router's bias keeps one expert from ever being chosen."""
    rng = np.random.default_rng(seed)
    d, vocab, taps = cfg["width"], cfg["vocab"], cfg["canon"]["taps"]

    def mat(r, c, gain=1.0):
        return rng.standard_normal((r, c)) * gain / np.sqrt(c)

    def vec(n, around=0.0, std=0.2):
        return around + std * rng.standard_normal(n)

    def taps_of(channels, n):
        return np.concatenate([rng.standard_normal((channels, n - 1)) * 0.4, vec((channels, 1), 0.8)], 1) if n else None

    counts = [(e.get("mlp") or {"router": {"experts": 0}})["router"]["experts"] for e in cfg["layers"]]
    kept = sum(counts)
    assert kept + 8 <= d
    w = {"embed": rng.standard_normal((vocab, d)), "final.norm": vec(d, 1), "head": mat(vocab, d)}
    rows = np.linalg.qr(rng.standard_normal((max(kept, 1), max(kept, 1))))[0]
    if kept:
        w["embed"][:, :kept] = np.concatenate([np.array([rng.permutation(n) - (n - 1) / 2.0 for _ in range(vocab)]).reshape(vocab, n) * 3.0 for n in counts if n], 1) @ rows

    def away(a):
        a[:kept] = 0
        return a

    at = 0
    for i, (e, n) in enumerate(zip(cfg["layers"], counts)):
        left, state, mlp, p = e["mixer"]["left"], e["mixer"]["right"]["width"], e.get("mlp"), f"l{i}."
        H, G, D, V = left["heads"], left["kv_heads"], left["dim"], left["vdim"]
        for s in (1, 2)[:2 if mlp else 1]:
            w[p + f"norm{s}"], w[p + f"canon{s}"] = vec(d, 1, 0.1), rng.standard_normal((d, taps)) * 0.3
            if s == 2:
                w[p + "norm2"][:kept] = 1
                w[p + "canon2"][:kept] = 0
                w[p + "canon2"][:kept, -1] = 0.25
        q = p + "mix.left."
        w[q + "q"], w[q + "k"], w[q + "v"], w[q + "o"] = mat(H * D, d), mat(G * D, d), mat(G * V, d), away(mat(d, H * V, 1.5))
        if left.get("conv"):
            for x, c in (("q", H * D), ("k", G * D), ("v", G * V)):
                w[q + x + ".conv"] = taps_of(c, left["conv"])
        q = p + "mix.right."
        w[q + "z"], w[q + "z.b"], w[q + "x"], w[q + "x.b"] = mat(state, d, 1.3), vec(state, -1, 0.8), mat(state, d), vec(state, 0, 0.5)
        w[q + "g"], w[q + "o"] = mat(state, d, 1.5), away(mat(d, state, 1.5))
        q = p + "mlp."
        if mlp:
            r = np.zeros((n, d))
            r[:, :kept] = rows[at:at + n]
            at += n
            w[q + "router"], w[q + "router.b"] = r, vec(n, 0, 0.05)
            if mlp["router"]["top"] < n:
                w[q + "router.b"][rng.integers(n)] = -40.0
            for x, ff in [(f"e{x}", mlp["expert"]["ff"]) for x in range(n)] + ([("shared", mlp["shared"]["ff"])] if mlp.get("shared") else []):
                w[q + f"{x}.gate"], w[q + f"{x}.up"], w[q + f"{x}.down"] = mat(ff, d, 1.5), mat(ff, d, 1.5), away(mat(d, ff, 1.5))
            if mlp.get("shared"):
                w[q + "shared.sg"] = mat(1, d, 1.5)
    return {k: bf16_round(v.astype(np.float32))[1] for k, v in w.items()}


def reference(cfg, w, tokens):
    """Logits [n, vocab] of a whole prompt."""
    m = X.Sakinex(cfg, w)
    return m.forward(tokens, m.new_state())


TOL = {"f32": 2e-5, "bf16": 4e-2}
