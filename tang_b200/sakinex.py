"""Sakinex (``tq_sakinex_*`` in include/tangq.h): configuration, weight loading and the model.

A small decoder whose mixers run attention and a minGRU on the same input.  The attention convolves its queries, keys and values
over the last few tokens, rotates them (YaRN), norms queries and keys per head behind the rotation, and sees a sliding window and
averages over blocks of older tokens.  Every sublayer's input passes a short convolution; the
feed-forwards are routed experts with a gated shared one; a stretch of layers may run several times with the same weights, each
pass with caches and states of its own.  No counterpart in the reference.
"""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass

from . import _lib
from .checkpoint import TensorView
from .device import QuantComputeDevice
from .stepmodel import NO_WINDOW, ConfigError, StepModel, host_array, need

# tq_sakinex_tensor
(EMBED, FINAL_NORM, HEAD, NORM1, NORM2, CANON1, CANON2, Q, K, V, Q_CONV, K_CONV, V_CONV, LEFT_O, Z, Z_BIAS, X, X_BIAS, G, RIGHT_O, ROUTER, ROUTER_BIAS, GATE, UP,
 DOWN, SHARED_GATE, SHARED_UP, SHARED_DOWN, SHARED_SWITCH) = range(29)


class _CConfig(C.Structure):
    _fields_ = [(n, C.c_uint32) for n in ("n_layers", "width", "vocab", "taps", "max_seq", "max_slots")] + [("dtype", C.c_int), ("eps", C.c_float), (
        "residual_mult", C.c_float)]


class _CLayer(C.Structure):
    _fields_ = [("weights_of", C.c_int32), ("add_embedding", C.c_int32)] + [(n, C.c_uint32) for n in (
        "heads", "kv_heads", "dim", "vdim", "window", "pool", "taps", "rot_dims", "state_width", "experts", "top", "ff", "shared_ff")] + [
            (n, C.c_float) for n in ("scale", "left_scale", "right_scale")] + [(n, C.c_double) for n in (
                "rot_base", "rot_factor", "rot_original", "rot_fast", "rot_slow")]


@dataclass(frozen=True)
class Rotation:
    dims: int = 0
    base: float = 0.0
    factor: float = 0.0       # 0: no scaling
    original: float = 0.0
    fast: float = 0.0
    slow: float = 0.0


@dataclass(frozen=True)
class Experts:
    experts: int = 0          # 0: no feed-forward
    top: int = 0
    ff: int = 0
    shared_ff: int = 0        # 0: no shared expert


@dataclass(frozen=True)
class SakinexLayer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    state_width: int          # of the recurrence
    window: int = NO_WINDOW
    pool: int = 0             # tokens of a pooled block; 0: none
    taps: int = 0             # of the convolutions on queries, keys and values; 0: none
    rot: Rotation = Rotation()
    left_scale: float = 1.0
    right_scale: float = 1.0
    mlp: Experts = Experts()


@dataclass(frozen=True)
class Run:
    """One run of a layer."""
    layer: int
    weights_of: int           # the first run of the layer, -1: this one
    add_embedding: bool       # whether the embedding output joins the stream ahead of it


def _up(n: int, to: int) -> int:
    return (n + to - 1) // to * to


@dataclass
class SakinexConfig:
    vocab: int
    width: int
    eps: float
    residual_mult: float
    taps: int                 # of the convolution on a sublayer's input
    layers: list
    loop: tuple = (0, 0, 1)   # layers start .. stop - 1 run `times` times

    @classmethod
    def from_dict(cls, c: dict) -> "SakinexConfig":
        """From the parsed config.json."""
        try:
            loop = c.get("loop") or {"start": 0, "stop": 0, "times": 1}
            cfg = cls(int(c["vocab"]), int(c["width"]), float(c["norm"]["eps"]), float(c["residual_mult"]), int(c["canon"]["taps"]),
                      [_layer(i, e) for i, e in enumerate(c["layers"])], (int(loop["start"]), int(loop["stop"]), int(loop["times"])))
        except (KeyError, TypeError) as e:
            raise ConfigError(f"config.json lacks {e}") from None
        start, stop, times = cfg.loop
        if not 0 <= start <= stop <= len(cfg.layers) or times < 1:
            raise ConfigError(f"loop over layers {start} .. {stop}, {times} times")
        if cfg.taps < 1:
            raise ConfigError(f"a convolution of {cfg.taps} taps")
        return cfg

    def runs(self) -> list[Run]:
        """What runs, in order."""
        start, stop, times = self.loop
        out = [Run(i, -1, False) for i in range(stop if times else start)]
        for _ in range(1, times):
            out += [Run(i, i, i == start) for i in range(start, stop)]
        return out + [Run(i, -1, False) for i in range(stop, len(self.layers))]

    def cache_bytes_per_token(self, dtype: int) -> int:
        rows = 0
        for r in self.runs():
            l = self.layers[r.layer]
            rows += l.kv_heads * (_up(l.dim, 8) + _up(l.vdim, 8)) * (1 + (1 / l.pool if l.pool else 0))
        return int(rows * (4 if dtype == _lib.F32 else 2)) + 1

    def state_bytes(self, dtype: int) -> int:
        es, total = 4 if dtype == _lib.F32 else 2, 0
        for r in self.runs():
            l = self.layers[r.layer]
            heads = _up(l.heads * l.dim, 16) + _up(l.kv_heads * l.dim, 16) + _up(l.kv_heads * l.vdim, 16)
            total += 4 * _up(l.state_width, 2) + es * (max(l.taps - 1, 0) * heads + (self.taps - 1) * self.width * (2 if l.mlp.experts else 1))
        return total

    def bytes_per_slot(self, dtype: int, max_seq: int) -> int:
        """Device memory that one more concurrent sequence takes."""
        return max_seq * self.cache_bytes_per_token(dtype) + self.state_bytes(dtype)


def _rotation(i: int, rot: dict | None) -> Rotation:
    if not rot:
        return Rotation()
    sc = rot.get("scaling") or {}
    r = Rotation(int(rot["dims"]), float(rot["base"]), **{k: float(sc[k]) for k in ("factor", "original", "fast", "slow") if sc})
    if sc and not r.factor > 0:
        raise ConfigError(f"layer {i}: rotation stretched by {r.factor}")
    return r


def _experts(i: int, mlp: dict | None) -> Experts:
    if mlp is None:
        return Experts()
    if mlp["kind"] != "moe":
        raise ConfigError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
    shared = mlp.get("shared")
    return Experts(int(mlp["router"]["experts"]), int(mlp["router"]["top"]), int(mlp["expert"]["ff"]), int(shared["ff"]) if shared else 0)


def _layer(i: int, e: dict) -> SakinexLayer:
    if e["type"] != "parallel":
        raise ConfigError(f"layer {i}: unknown mixer {e['type']!r}")
    m = e["mixer"]
    left, mask = m["left"], m["left"].get("mask") or {}
    return SakinexLayer(int(left["heads"]), int(left["kv_heads"]), int(left["dim"]), int(left["vdim"]), float(left["scale"]), int(m["right"]["width"]),
                        int(mask.get("size", NO_WINDOW)), int(mask.get("pool") or 0), int(left.get("conv") or 0), _rotation(i, left.get("rot")),
                        float(m["left_scale"]), float(m["right_scale"]), _experts(i, e.get("mlp")))


_CONV = (("q.conv", Q_CONV), ("k.conv", K_CONV), ("v.conv", V_CONV))
_MIXER = [(f"left.{n}", t) for n, t in (("q", Q), ("k", K), ("v", V), ("o", LEFT_O))] + [
    (f"right.{n}", t) for n, t in (("z", Z), ("z.b", Z_BIAS), ("x", X), ("x.b", X_BIAS), ("g", G), ("o", RIGHT_O))]
_FF = (("gate", GATE), ("up", UP), ("down", DOWN))
_SHARED = (("gate", SHARED_GATE), ("up", SHARED_UP), ("down", SHARED_DOWN), ("sg", SHARED_SWITCH))


def tensor_names(cfg: SakinexConfig):
    """(name, tensor, run, expert) of every tensor of the checkpoint; a layer's tensors belong to its first run."""
    yield from (("embed", EMBED, 0, 0), ("final.norm", FINAL_NORM, 0, 0), ("head", HEAD, 0, 0))
    for run, r in enumerate(cfg.runs()):
        if r.weights_of >= 0:
            continue
        l = cfg.layers[r.layer]
        names = [("norm1", NORM1), ("canon1", CANON1)] + [(f"mix.{n}", t) for n, t in _MIXER]
        if l.taps:
            names += [(f"mix.left.{n}", t) for n, t in _CONV]
        if l.mlp.experts:
            names += [("norm2", NORM2), ("canon2", CANON2), ("mlp.router", ROUTER), ("mlp.router.b", ROUTER_BIAS)]
            if l.mlp.shared_ff:
                names += [(f"mlp.shared.{n}", t) for n, t in _SHARED]
        for n, t in names:
            yield f"l{r.layer}.{n}", t, run, 0
        for e in range(l.mlp.experts):
            for n, t in _FF:
                yield f"l{r.layer}.mlp.e{e}.{n}", t, run, e


class SakinexModel(StepModel):
    """Weights, caches, states and the step.  `dtype` BF16: bf16 weights, activations and caches with an f32 stream and states;
    F32: all f32.  ``trace`` receives the stream after every run of a layer."""

    abi = "tq_sakinex"

    def __init__(self, dev: QuantComputeDevice, cfg: SakinexConfig, dtype: int = _lib.BF16, max_slots: int = 64, max_seq: int | None = None):
        from .registry import DEFAULT_MAX_SEQ

        self.dev, self.cfg, self.dtype, self.max_slots = dev, cfg, dtype, max_slots
        self.max_seq = max_seq or DEFAULT_MAX_SEQ
        runs = cfg.runs()
        cc = _CConfig(len(runs), cfg.width, cfg.vocab, cfg.taps, self.max_seq, max_slots, dtype, cfg.eps, cfg.residual_mult)
        cl = (_CLayer * len(runs))()
        for c, r in zip(cl, runs):
            l = cfg.layers[r.layer]
            c.weights_of, c.add_embedding = r.weights_of, r.add_embedding
            for n in ("heads", "kv_heads", "dim", "vdim", "window", "pool", "taps", "state_width", "scale", "left_scale", "right_scale"):
                setattr(c, n, getattr(l, n))
            for n in ("experts", "top", "ff", "shared_ff"):
                setattr(c, n, getattr(l.mlp, n))
            for n in ("dims", "base", "factor", "original", "fast", "slow"):
                setattr(c, f"rot_{n}", getattr(l.rot, n))
        h = C.c_void_p()
        dev._check(dev._L.tq_sakinex_create(dev._ctx, C.byref(cc), cl, C.byref(h)))
        self.handle = h.value

    @classmethod
    def from_tensors(cls, dev: QuantComputeDevice, config: dict, tensors: dict, dtype: int = _lib.BF16, max_slots: int = 64,
                     max_seq: int | None = None) -> "SakinexModel":
        """From a parsed config.json and the tensors of the checkpoint (``read_safetensors``)."""
        cfg = SakinexConfig.from_dict(config)
        model = cls(dev, cfg, dtype, max_slots, max_seq)
        try:
            for name, tensor, run, expert in tensor_names(cfg):
                model.put(tensor, run, need(tensors, name), expert)
        except Exception:
            model.destroy()
            raise
        return model

    def put(self, tensor: int, run: int, view: TensorView, expert: int = 0) -> None:
        a, dt, rows, cols = host_array(view)
        self.put_pointer(tensor, run, a.ctypes.data, dt, rows, cols, expert)

    def put_pointer(self, tensor: int, run: int, ptr: int, dtype: int, rows: int, cols: int, expert: int = 0) -> None:
        """`ptr`: host or device address of the row-major [rows, cols] tensor."""
        self._call("put", tensor, run, expert, C.c_void_p(ptr), dtype, rows, cols)
