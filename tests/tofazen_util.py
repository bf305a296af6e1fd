"""Small random Tofazen models, as a configuration and a dict of tensors, for the library and for the numpy implementation."""
import numpy as np

import tofazen_oracle as T
from util import bf16_round


def layer(heads, kv_heads, dim, vdim, window, keep_first, ff=None, limit=1.5, diff=0.4, scale=None, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "diff": diff, "scale": dim ** -0.5 if scale is None else scale,
         "mask": {"size": window, "keep_first": keep_first}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": None if ff is None else {"kind": "dense", "ff": ff, "limit": limit}}


def config(layers, width=72, vocab=101, max_positions=400, eps=1e-5, residual_mult=0.9):
    return {"architecture": "Tofazen", "layers": layers, "max_positions": max_positions, "norm": {"eps": eps}, "residual_mult": residual_mult,
            "vocab": vocab, "width": width}


# Sizes that differ from layer to layer, odd ones, groups of 1 to 12 heads, layers without a feed-forward, shared keys
# under another mask, windows below, at and above the 64-key tiles, kept tokens below and above them.
CONFIGS = {
    "mixed": config([layer(6, 2, 20, 40, 17, 3, ff=88), layer(6, 2, 20, 40, 33, 0, ff=50, kv_from=0, diff=0.1),
                     layer(3, 3, 24, 16, 5, 1, ff=None), layer(6, 2, 20, 40, 9, 6, ff=None, kv_from=0, scale=0.4)]),
    "odd": config([layer(8, 1, 33, 51, 70, 70, ff=37, limit=0.8), layer(4, 4, 7, 9, 64, 2, ff=24)], width=100, vocab=67, residual_mult=1.0, eps=1e-3),
    "wide_group": config([layer(12, 1, 16, 24, 1, 0, ff=40), layer(12, 1, 16, 24, 130, 5, ff=160)], width=200, vocab=300, residual_mult=1.6),
    "large_heads": config([layer(2, 1, 136, 200, 40, 2, ff=64), layer(2, 2, 72, 264, 50, 1, ff=64)], width=128, vocab=64),
}


def weights(cfg, seed, sharp=1.0):
    """Random tensors by name, rounded to bf16.  `sharp` scales the queries: larger values concentrate the attention."""
    rng = np.random.default_rng(seed)
    d = cfg["width"]

    def mat(r, c, gain=1.0):
        return rng.standard_normal((r, c)) * gain / np.sqrt(c)

    w = {"embed": rng.standard_normal((cfg["vocab"], d)), "pos": rng.standard_normal((cfg["max_positions"], d)) * 0.7,
         "final.norm": 1 + 0.2 * rng.standard_normal(d), "head": mat(cfg["vocab"], d)}
    for i, e in enumerate(cfg["layers"]):
        m, p = e["mixer"], f"l{i}."
        w[p + "norm1"] = 1 + 0.2 * rng.standard_normal(d)
        w[p + "mix.q"] = mat(m["heads"] * 2 * m["dim"], d, 1.7 * sharp)
        if "kv_from" not in m:
            w[p + "mix.k"] = mat(m["kv_heads"] * 2 * m["dim"], d, 1.7)
            w[p + "mix.v"] = mat(m["kv_heads"] * m["vdim"], d)
        for n in ("lq1", "lk1", "lq2", "lk2"):
            w[p + "mix." + n] = rng.standard_normal(m["dim"]) * 0.5 / np.sqrt(m["dim"]) ** 0.5
        w[p + "mix.o"] = mat(d, m["heads"] * m["vdim"])
        if e["mlp"]:
            ff = e["mlp"]["ff"]
            w[p + "mlp.gate"], w[p + "mlp.up"], w[p + "mlp.down"] = mat(ff, d, 1.5), mat(ff, d, 1.5), mat(d, ff)
    return {k: bf16_round(v.astype(np.float32))[1] for k, v in w.items()}


def views(w):
    from tang_b200 import TensorView

    return {k: TensorView("BF16", v.shape, bf16_round(v)[0].reshape(-1)) for k, v in w.items()}


def save(folder, cfg, w):
    import json

    from tang_b200 import write_safetensors

    (folder / "config.json").write_text(json.dumps(cfg))
    write_safetensors(folder / "model.safetensors", {k: ("BF16", v.shape, bf16_round(v)[0].reshape(-1)) for k, v in w.items()})


def reference(cfg, w, tokens):
    """Logits [n, vocab] of a whole prompt."""
    m = T.Tofazen(cfg, w)
    return m.forward(tokens, m.new_state())


def row_errors(got, want):
    """Root mean square difference of every row over the rms of all of `want`."""
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    return np.sqrt(np.mean((got - want) ** 2, axis=-1)) / np.sqrt(np.mean(want * want))


TOL = {"f32": 2e-5, "bf16": 2.5e-2}
