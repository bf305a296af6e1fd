"""Tofazen (``tq_tofazen_*`` in include/tangq.h): configuration, weight loading and the model.

A small decoder with learned absolute positions, parallel layers (one norm feeds attention and feed-forward),
differential attention under a sliding window that keeps the first tokens, layers that read an earlier layer's keys and
values, and a clamped gated feed-forward.  No counterpart in the reference.
"""
from __future__ import annotations

import ctypes as C
import math
from dataclasses import dataclass

import numpy as np

from . import _lib
from .checkpoint import TensorView
from .device import QuantComputeDevice
from .stepmodel import NO_WINDOW, ConfigError, StepModel, host_array, need

# tq_tofazen_tensor
EMBED, POS, FINAL_NORM, HEAD, NORM, Q, K, V, O, GATE, UP, DOWN = range(12)


class _CConfig(C.Structure):
    _fields_ = [(n, C.c_uint32) for n in ("n_layers", "width", "vocab", "max_positions", "max_seq", "max_slots")] + [
        ("dtype", C.c_int), ("eps", C.c_float), ("residual_mult", C.c_float)]


class _CLayer(C.Structure):
    _fields_ = [(n, C.c_uint32) for n in ("heads", "kv_heads", "dim", "vdim", "ff")] + [("kv_from", C.c_int)] + [
        (n, C.c_uint32) for n in ("window", "keep_first")] + [(n, C.c_float) for n in ("scale", "lam", "out_scale", "limit")]


@dataclass
class TofazenLayer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    diff: float
    window: int
    keep_first: int
    kv_from: int | None = None
    ff: int = 0               # 0: no feed-forward
    limit: float = 0.0


@dataclass
class TofazenConfig:
    vocab: int
    width: int
    max_positions: int
    eps: float
    residual_mult: float
    layers: list

    @classmethod
    def from_dict(cls, c: dict) -> "TofazenConfig":
        """From the parsed config.json."""
        try:
            layers = []
            for i, e in enumerate(c["layers"]):
                if e["type"] != "attention":
                    raise ConfigError(f"layer {i}: unknown mixer {e['type']!r}")
                m, mask, mlp = e["mixer"], e["mixer"].get("mask") or {}, e.get("mlp")
                if mlp is not None and mlp["kind"] != "dense":
                    raise ConfigError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
                src = m.get("kv_from")
                layers.append(TofazenLayer(
                    int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"]), float(m["diff"]),
                    int(mask.get("size", NO_WINDOW)), int(mask.get("keep_first", 0)), None if src is None else int(src),
                    0 if mlp is None else int(mlp["ff"]), 0.0 if mlp is None else float(mlp["limit"])))
            return cls(int(c["vocab"]), int(c["width"]), int(c["max_positions"]), float(c["norm"]["eps"]), float(c["residual_mult"]), layers)
        except (KeyError, TypeError) as e:
            raise ConfigError(f"config.json lacks {e}") from None

    def cache_bytes_per_token(self, dtype: int) -> int:
        up8 = lambda n: (n + 7) // 8 * 8
        n = sum(l.kv_heads * (2 * up8(l.dim) + up8(l.vdim)) for l in self.layers if l.kv_from is None)
        return n * (4 if dtype == _lib.F32 else 2)

    def bytes_per_slot(self, dtype: int, max_seq: int) -> int:
        """Device memory that one more concurrent sequence takes."""
        return max_seq * self.cache_bytes_per_token(dtype)


def tensor_names(cfg: TofazenConfig):
    """(name, tensor, layer) of every tensor that goes to the device as it is."""
    yield from (("embed", EMBED, 0), ("pos", POS, 0), ("final.norm", FINAL_NORM, 0), ("head", HEAD, 0))
    for i, l in enumerate(cfg.layers):
        yield f"l{i}.norm1", NORM, i
        for n, t in (("q", Q), ("k", K), ("v", V), ("o", O)):
            if t in (Q, O) or l.kv_from is None:
                yield f"l{i}.mix.{n}", t, i
        if l.ff:
            for n, t in (("gate", GATE), ("up", UP), ("down", DOWN)):
                yield f"l{i}.mlp.{n}", t, i


def map_balance(l: TofazenLayer, lq1, lk1, lq2, lk2) -> float:
    """The factor of the second map: exp(lq1 . lk1) - exp(lq2 . lk2) + diff."""
    dot = lambda a, b: float(np.dot(np.asarray(a, np.float64), np.asarray(b, np.float64)))
    return math.exp(dot(lq1, lk1)) - math.exp(dot(lq2, lk2)) + l.diff


class TofazenModel(StepModel):
    """Weights, caches and the step.  `dtype` BF16: bf16 weights, activations and caches with an f32 stream; F32: all f32.
    `lambdas`: one factor of the second map per layer (``map_balance``)."""

    abi = "tq_tofazen"

    def __init__(self, dev: QuantComputeDevice, cfg: TofazenConfig, lambdas, dtype: int = _lib.BF16, max_slots: int = 64,
                 max_seq: int | None = None):
        self.dev, self.cfg, self.dtype, self.max_slots = dev, cfg, dtype, max_slots
        self.max_seq = min(max_seq or cfg.max_positions, cfg.max_positions)
        cc = _CConfig(len(cfg.layers), cfg.width, cfg.vocab, cfg.max_positions, self.max_seq, max_slots, dtype, cfg.eps, cfg.residual_mult)
        cl = (_CLayer * len(cfg.layers))(*[
            _CLayer(l.heads, l.kv_heads, l.dim, l.vdim, l.ff, -1 if l.kv_from is None else l.kv_from, l.window, l.keep_first,
                    l.scale, lam, 1.0 - l.diff, l.limit) for l, lam in zip(cfg.layers, lambdas)])
        h = C.c_void_p()
        dev._check(dev._L.tq_tofazen_create(dev._ctx, C.byref(cc), cl, C.byref(h)))
        self.handle = h.value

    @classmethod
    def from_tensors(cls, dev: QuantComputeDevice, config: dict, tensors: dict, dtype: int = _lib.BF16, max_slots: int = 64,
                     max_seq: int | None = None) -> "TofazenModel":
        """From a parsed config.json and the tensors of the checkpoint (``read_safetensors``)."""
        cfg = TofazenConfig.from_dict(config)
        lambdas = [map_balance(l, *(need(tensors, f"l{i}.mix.{n}").to_f32() for n in ("lq1", "lk1", "lq2", "lk2"))) for i, l in enumerate(cfg.layers)]
        model = cls(dev, cfg, lambdas, dtype, max_slots, max_seq)
        try:
            for name, tensor, layer in tensor_names(cfg):
                model.put(tensor, layer, need(tensors, name))
        except Exception:
            model.destroy()
            raise
        return model

    def put(self, tensor: int, layer: int, view: TensorView) -> None:
        a, dt, rows, cols = host_array(view)
        self.put_pointer(tensor, layer, a.ctypes.data, dt, rows, cols)

    def put_pointer(self, tensor: int, layer: int, ptr: int, dtype: int, rows: int, cols: int) -> None:
        """`ptr`: host or device address of the row-major [rows, cols] tensor."""
        self._call("put", tensor, layer, C.c_void_p(ptr), dtype, rows, cols)
