"""Small random Numuzen models, as a configuration and a dict of tensors, for the library and for the numpy implementation."""
import numpy as np

import numuzen_oracle as N
from tofazen_util import row_errors, save, views  # noqa: F401
from util import bf16_round


def moe(experts, top, ff, limit=1.3):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff, "limit": limit}}


def attn(heads, kv_heads, dim, window, mlp=None, rot=8, base=10000.0, scaling=(4.0, 64, 16.0, 1.0), softcap=20.0, scale=None):
    sc = None if scaling is None else dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"type": "attention", "mlp": mlp, "mixer": {
        "heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": dim ** -0.5 if scale is None else scale, "softcap": softcap,
        "mask": {"size": window}, "rot": {"base": base, "dims": rot, "scaling": sc}}}


def gla(heads, dim, vdim, mlp=None, tau=12.0):
    return {"type": "gla", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}}


def config(layers, width=72, vocab=101, eps=1e-5):
    return {"architecture": "Numuzen", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}


# Sizes that differ from layer to layer, odd ones, groups of 1 to 12 heads, layers without a feed-forward, windows below, at
# and above the 64-key tiles, all experts of a layer chosen or one of them, and sizes that take the tensor-core recurrence.
CONFIGS = {
    "mixed": config([attn(6, 2, 20, 17, moe(5, 2, 24)), gla(3, 20, 40, moe(4, 1, 37)), attn(3, 3, 24, 64), gla(2, 24, 16, None, tau=1.0),
                     attn(6, 2, 20, 33, moe(6, 3, 16), rot=20, scaling=None, softcap=7.0)]),
    "odd": config([gla(1, 7, 9, moe(3, 3, 11)), attn(5, 1, 33, 70, moe(2, 1, 50), rot=10, scale=0.3), gla(5, 33, 51, moe(7, 2, 8), tau=3.0)], width=100, vocab=67,
                  eps=1e-3),
    "aligned": config([gla(2, 64, 128, moe(8, 2, 48)), attn(12, 1, 16, 1, moe(1, 1, 40), rot=16), gla(4, 32, 64, moe(8, 4, 32), tau=5.0),
                       attn(4, 2, 64, 130, moe(4, 2, 64), rot=32)], width=192, vocab=300),
    "large_heads": config([attn(2, 1, 136, 40, moe(3, 1, 32), rot=64), attn(2, 2, 264, 50), gla(1, 160, 264, moe(3, 2, 24)), gla(2, 128, 256)], width=128,
                          vocab=64),
}
RANKS = {"mixed": 5, "odd": 3, "aligned": 16, "large_heads": 24}
SHARPNESS = 1.5


def weights(cfg, seed, rank=6):
    """Random tensors by name, rounded to bf16.  The routers' rows are orthonormal over all layers, and every token's embedding
    has well separated products with each of them: expert choices are never close calls, in any number format.  The final norm's gains have both signs, or else the tied embeddings
    would make every token predict itself."""
    rng = np.random.default_rng(seed)
    d, vocab = cfg["width"], cfg["vocab"]

    def mat(r, c, gain=1.0):
        return rng.standard_normal((r, c)) * gain / np.sqrt(c)

    def vec(n, around, std=0.2):
        return around + std * rng.standard_normal(n)

    w = {"embed": rng.standard_normal((vocab, d)), "final.norm": vec(d, -1, 1.0)}
    counts = [e["mlp"]["router"]["experts"] if e.get("mlp") else 0 for e in cfg["layers"]]
    rows = np.linalg.qr(rng.standard_normal((d, sum(counts))))[0].T
    target = np.concatenate([np.array([rng.permutation(n) - (n - 1) / 2.0 for _ in range(vocab)]).reshape(vocab, n) * 3.0 for n in counts], axis=1)
    w["embed"] += (target - w["embed"] @ rows.T) @ rows
    at = 0
    for i, (e, n) in enumerate(zip(cfg["layers"], counts)):
        m, p = e["mixer"], f"l{i}."
        H, D, V = m["heads"], m["dim"], m["vdim"]
        w[p + "norm1"], w[p + "norm1b"] = vec(d, 0), vec(d, -0.75, 0.1)
        w[p + "mix.q"], w[p + "mix.g"], w[p + "mix.o"] = mat(H * D, d, SHARPNESS), mat(H * V, d, 1.5), mat(d, H * V)
        if e["type"] == "attention":
            w[p + "mix.k"] = mat(m["kv_heads"] * D, d, SHARPNESS)
            w[p + "mix.q.norm"], w[p + "mix.k.norm"] = vec(H * D, 1.5), vec(m["kv_heads"] * D, 1.5)
        else:
            w[p + "mix.k"], w[p + "mix.v"] = mat(H * D, d), mat(H * V, d)
            w[p + "mix.a1"], w[p + "mix.a2"], w[p + "mix.a2.b"] = mat(rank, d, 2.0), mat(H * D, rank, 2.0), vec(H * D, 1.0, 2.0)
            w[p + "mix.norm"] = vec(V, 1)
        if n:
            ff = e["mlp"]["expert"]["ff"]
            w[p + "norm2"], w[p + "norm2b"] = vec(d, 0, 0.05), vec(d, -0.75, 0.1)
            w[p + "mlp.router"] = rows[at:at + n]
            at += n
            for x in range(n):
                w[p + f"mlp.e{x}.gate"], w[p + f"mlp.e{x}.up"], w[p + f"mlp.e{x}.down"] = mat(ff, d, 1.5), mat(ff, d, 1.5), mat(d, ff)
    return {k: bf16_round(v.astype(np.float32))[1] for k, v in w.items()}


def reference(cfg, w, tokens):
    """Logits [n, vocab] of a whole prompt."""
    m = N.Numuzen(cfg, w)
    return m.forward(tokens, m.new_state())


TOL = {"f32": 2e-5, "bf16": 4e-2}
