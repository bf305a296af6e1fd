"""Small random Dotanex models, as a configuration and a dict of tensors, for the library and for the numpy implementation."""
import numpy as np

import dotanex_oracle as X
from tofazen_util import row_errors, save, views  # noqa: F401
from util import bf16_round


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, identity, top, ff, shared, limit=1.3, shared_limit=0.9):
    return {"kind": "moe", "router": {"experts": experts, "identity": identity, "top": top}, "expert": {"ff": ff, "limit": limit},
            "shared": {"ff": shared, "limit": shared_limit}}


def attn(heads, kv_heads, dim, window, mlp=None, rot=8, base=10000.0, scaling=(4.0, 1.0, 3.0, 64), scale=None):
    sc = None if scaling is None else dict(zip(("factor", "low", "high", "original"), scaling))
    return {"type": "attention", "mlp": mlp, "mixer": {
        "heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": dim ** -0.5 if scale is None else scale, "mask": {"size": window},
        "rot": {"base": base, "dims": rot, "scaling": sc}}}


def latent(heads, dim, rot, vdim, q_rank, kv_rank, mlp=None, base=10000.0, scaling=(4.0, 64, 16.0, 1.0), scale=None):
    sc = None if scaling is None else dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"type": "latent_attention", "mlp": mlp, "mixer": {
        "heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": (dim + rot) ** -0.5 if scale is None else scale,
        "rot": {"base": base, "dims": rot, "scaling": sc}}}


def lightning(heads, dim, vdim, mlp=None, decay=None):
    return {"type": "lightning", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "vdim": vdim,
                                                        "decay": [1.0 - 0.6 ** (h + 1) for h in range(heads)] if decay is None else decay}}


def again(layers, j):
    """Layer j's entry with layer j's weights."""
    return {**layers[j], "weights_of": j}


def config(layers, width=72, vocab=101, streams=2, eps=1e-5):
    return {"architecture": "Dotanex", "layers": layers, "norm": {"eps": eps}, "streams": streams, "vocab": vocab, "width": width}


# Sizes that differ from layer to layer, odd ones, one stream and more than four, groups of 1 to 12 heads, more than 16 latent
# heads, latents below and above what the absorbed form takes, layers without a feed-forward, shared weights, windows below, at and
# above the 64-key tiles, all experts of a layer chosen or one of them, no identity experts, decays of 1 and 0, and sizes that take
# the tensor-core recurrence.
_mixed = [attn(6, 2, 20, 17, moe(5, 3, 2, 24, 40)), latent(3, 12, 8, 20, 24, 28, dense(50)), lightning(3, 20, 40, moe(4, 1, 1, 37, 16)),
          latent(5, 16, 6, 10, 20, 48, moe(6, 2, 4, 16, 30), scaling=None), attn(3, 3, 24, 64, None)]
_mixed += [again(_mixed, 1), lightning(2, 24, 16, None, decay=[1.0, 0.0]), again(_mixed, 0), attn(6, 2, 20, 33, dense(24), rot=20, scaling=None), again(_mixed, 2)]
CONFIGS = {
    "mixed": config(_mixed, streams=3),
    "odd": config([lightning(1, 7, 9, moe(3, 2, 3, 11, 13)), attn(5, 1, 33, 70, moe(2, 0, 1, 50, 8), rot=10, scale=0.3), latent(5, 7, 6, 9, 11, 13, moe(3, 1, 2, 9, 21)),
                   lightning(5, 33, 51, dense(37))], width=100, vocab=67, streams=1, eps=1e-3),
    "aligned": config([lightning(2, 64, 128, moe(8, 4, 2, 48, 64)), attn(12, 1, 16, 1, dense(96), rot=16), latent(17, 32, 16, 48, 64, 160, moe(6, 6, 4, 64, 32)),
                       lightning(4, 32, 64, moe(8, 2, 6, 32, 48)), attn(4, 2, 64, 130, moe(4, 1, 2, 64, 64), rot=32)], width=192, vocab=300, streams=4),
    "large_heads": config([attn(2, 1, 136, 40, moe(3, 1, 1, 32, 24), rot=64), latent(2, 128, 64, 128, 96, 320, dense(48)), attn(2, 2, 264, 50),
                           lightning(1, 160, 264, moe(3, 3, 2, 24, 16)), latent(3, 24, 16, 32, 40, 530), lightning(2, 128, 256)], width=128, vocab=64, streams=5),
}
SHARPNESS = 1.5


def weights(cfg, seed):
    """Random tensors by name, rounded to bf16.  The routers' rows are orthonormal over all layers, every token's embedding has
    well separated products with each of them, and nothing else that enters the streams has any: the order of a layer's logits is
    never a close call, in any number format.  One expert of a layer is always chosen for its correction and one never is."""
    rng = np.random.default_rng(seed)
    d, vocab, S = cfg["width"], cfg["vocab"], cfg["streams"]

    def mat(r, c, gain=1.0):
        return rng.standard_normal((r, c)) * gain / np.sqrt(c)

    def vec(n, around, std=0.2):
        return around + std * rng.standard_normal(n)

    w = {"embed": rng.standard_normal((vocab, d)), "final.norm": vec(d, 1), "head": mat(vocab, d)}
    counts = [0 if (e.get("mlp") or {}).get("kind") != "moe" or "weights_of" in e else e["mlp"]["router"]["experts"] + e["mlp"]["router"]["identity"]
              for e in cfg["layers"]]
    rows = np.linalg.qr(rng.standard_normal((d, max(1, sum(counts)))))[0].T
    if sum(counts):
        target = np.concatenate([np.array([rng.permutation(n) - (n - 1) / 2.0 for _ in range(vocab)]).reshape(vocab, n) * 3.0 for n in counts if n], axis=1)
        w["embed"] += (target - w["embed"] @ rows.T) @ rows
    away = (lambda a: a - rows.T @ (rows @ a)) if sum(counts) else lambda a: a
    at = 0
    for i, (e, n) in enumerate(zip(cfg["layers"], counts)):
        if "weights_of" in e:
            continue
        m, mlp, p = e["mixer"], e.get("mlp"), f"l{i}."
        H, D, V = m["heads"], m["dim"], m["vdim"]
        for q in (1, 2)[:2 if mlp else 1]:
            w[p + f"norm{q}"] = vec(d, 1, 0.05)
            w[p + f"hc{q}.in"], w[p + f"hc{q}.out"] = vec(S, 1.0 / S, 0.15 / S), vec(S, 0.5, 0.25)
            w[p + f"hc{q}.mix"] = 0.8 * np.eye(S) + rng.uniform(0, 0.4 / S, (S, S))
        p += "mix."
        w[p + "o"] = away(mat(d, H * V))
        if e["type"] == "attention":
            w[p + "q"], w[p + "k"] = mat(H * D, d, SHARPNESS), mat(m["kv_heads"] * D, d, SHARPNESS)
            w[p + "q.norm"], w[p + "k.norm"], w[p + "sink"] = vec(D, 1.5), vec(D, 1.5), vec(H, 1.0, 1.5)
        elif e["type"] == "latent_attention":
            R, C, Q = m["rot_dim"], m["kv_rank"], m["q_rank"]
            w[p + "dq"], w[p + "dq.norm"], w[p + "uq"] = mat(Q, d), vec(Q, 1), mat(H * (D + R), Q, SHARPNESS)
            w[p + "dkv"], w[p + "dkv.norm"], w[p + "uk"], w[p + "uv"] = mat(C + R, d, 1.2), vec(C, 1), mat(H * D, C, SHARPNESS), mat(H * V, C)
            w[p + "g"] = mat(H * V, d, 1.5)
        else:
            w[p + "q"], w[p + "k"], w[p + "v"], w[p + "g"], w[p + "norm"] = mat(H * D, d), mat(H * D, d), mat(H * V, d), mat(H * V, d, 1.5), vec(H * V, 1)
        p = f"l{i}.mlp."
        if mlp and mlp["kind"] == "dense":
            w[p + "gate"], w[p + "up"], w[p + "down"] = mat(mlp["ff"], d, 1.5), mat(mlp["ff"], d, 1.5), away(mat(d, mlp["ff"]))
        elif mlp:
            w[p + "router"] = rows[at:at + n]
            at += n
            w[p + "correction"] = np.zeros(n)
            if mlp["router"]["top"] > 1:
                w[p + "correction"][rng.integers(n - 1)] = 2.0
            if mlp["router"]["top"] < n - 1:
                w[p + "correction"][n - 1] = -2.0
            for x, ff in [(f"e{x}", mlp["expert"]["ff"]) for x in range(mlp["router"]["experts"])] + [("shared", mlp["shared"]["ff"])]:
                w[p + f"{x}.gate"], w[p + f"{x}.up"], w[p + f"{x}.down"] = mat(ff, d, 1.5), mat(ff, d, 1.5), away(mat(d, ff))
    return {k: bf16_round(v.astype(np.float32))[1] for k, v in w.items()}


def reference(cfg, w, tokens):
    """Logits [n, vocab] of a whole prompt."""
    m = X.Dotanex(cfg, w)
    return m.forward(tokens, m.new_state())


TOL = {"f32": 2e-5, "bf16": 4e-2}
