"""Numuzen (``tq_numuzen_*`` in include/tangq.h): configuration, weight loading and the model.

A small decoder whose layers are sliding-window attention (whole-projection query/key norm, YaRN rotation, capped scores, a
sink, an output gate, values that are the raw keys) or gated linear attention, each with sigmoid-routed experts, norms before
and after every sublayer and tied embeddings.  No counterpart in the reference.
"""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass

from . import _lib
from .checkpoint import TensorView
from .device import QuantComputeDevice
from .stepmodel import NO_WINDOW, ConfigError, StepModel, host_array, need

# tq_numuzen_tensor
(EMBED, FINAL_NORM, NORM1, NORM1B, NORM2, NORM2B, Q, K, V, G, O, Q_NORM, K_NORM, O_NORM, A1, A2, A2_BIAS, ROUTER, GATE, UP, DOWN) = range(21)

# tq_numuzen_mixer
ATTENTION, GLA = range(2)


class _CConfig(C.Structure):
    _fields_ = [(n, C.c_uint32) for n in ("n_layers", "width", "vocab", "max_seq", "max_slots")] + [("dtype", C.c_int), ("eps", C.c_float)]


class _CLayer(C.Structure):
    _fields_ = [(n, C.c_uint32) for n in ("kind", "heads", "kv_heads", "dim", "vdim", "window", "rot_dims", "rank", "experts", "top", "ff")] + [
        (n, C.c_float) for n in ("scale", "softcap", "tau", "limit")] + [
        (n, C.c_double) for n in ("rot_base", "rot_factor", "rot_original", "rot_fast", "rot_slow")]


@dataclass
class Rotation:
    dims: int = 0
    base: float = 0.0
    factor: float = 0.0       # 0: no scaling
    original: float = 0.0
    fast: float = 0.0
    slow: float = 0.0


@dataclass
class Experts:
    count: int
    top: int
    ff: int
    limit: float


@dataclass
class NumuzenLayer:
    kind: int                 # ATTENTION or GLA
    heads: int
    dim: int
    vdim: int
    scale: float              # of the scores / of the recurrent queries
    kv_heads: int = 0
    window: int = NO_WINDOW
    softcap: float = 0.0
    rot: Rotation | None = None
    tau: float = 1.0
    rank: int = 0             # recurrent: rows of a1; the checkpoint gives it
    experts: Experts | None = None


@dataclass
class NumuzenConfig:
    vocab: int
    width: int
    eps: float
    layers: list

    @classmethod
    def from_dict(cls, c: dict) -> "NumuzenConfig":
        """From the parsed config.json."""
        try:
            return cls(int(c["vocab"]), int(c["width"]), float(c["norm"]["eps"]), [_layer(i, e) for i, e in enumerate(c["layers"])])
        except (KeyError, TypeError) as e:
            raise ConfigError(f"config.json lacks {e}") from None

    def cache_bytes_per_token(self, dtype: int) -> int:
        up8 = lambda n: (n + 7) // 8 * 8
        return sum(2 * l.kv_heads * up8(l.dim) for l in self.layers if l.kind == ATTENTION) * (4 if dtype == _lib.F32 else 2)

    def state_bytes(self) -> int:
        return 4 * sum(l.heads * l.dim * l.vdim for l in self.layers if l.kind == GLA)

    def bytes_per_slot(self, dtype: int, max_seq: int) -> int:
        """Device memory that one more concurrent sequence takes."""
        return max_seq * self.cache_bytes_per_token(dtype) + self.state_bytes()


def _layer(i: int, e: dict) -> NumuzenLayer:
    m, mlp = e["mixer"], e.get("mlp")
    experts = None
    if mlp is not None:
        if mlp["kind"] != "moe":
            raise ConfigError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
        experts = Experts(int(mlp["router"]["experts"]), int(mlp["router"]["top"]), int(mlp["expert"]["ff"]), float(mlp["expert"]["limit"]))
    heads, dim = int(m["heads"]), int(m["dim"])
    if e["type"] == "attention":
        if int(m["vdim"]) != dim:
            raise ConfigError(f"layer {i}: the values are the keys, so vdim must be dim")
        rot, mask = m.get("rot") or {"dims": 0, "base": 0.0}, m.get("mask") or {}
        sc = rot.get("scaling") or {}
        r = Rotation(int(rot["dims"]), float(rot["base"]), *((float(sc[k]) for k in ("factor", "original", "fast", "slow")) if sc else ()))
        return NumuzenLayer(ATTENTION, heads, dim, dim, float(m["scale"]), int(m["kv_heads"]), int(mask.get("size", NO_WINDOW)), float(m["softcap"]), r,
                            experts=experts)
    if e["type"] == "gla":
        return NumuzenLayer(GLA, heads, dim, int(m["vdim"]), dim ** -0.5, tau=float(m["tau"]), experts=experts)
    raise ConfigError(f"layer {i}: unknown mixer {e['type']!r}")


_MIXER = {ATTENTION: (("q", Q), ("k", K), ("g", G), ("o", O), ("q.norm", Q_NORM), ("k.norm", K_NORM)),
          GLA: (("q", Q), ("k", K), ("v", V), ("g", G), ("o", O), ("norm", O_NORM), ("a1", A1), ("a2", A2), ("a2.b", A2_BIAS))}


def tensor_names(cfg: NumuzenConfig):
    """(name, tensor, layer, expert) of every tensor of the checkpoint."""
    yield from (("embed", EMBED, 0, 0), ("final.norm", FINAL_NORM, 0, 0))
    for i, l in enumerate(cfg.layers):
        for n, t in (("norm1", NORM1), ("norm1b", NORM1B)) + ((("norm2", NORM2), ("norm2b", NORM2B)) if l.experts else ()):
            yield f"l{i}.{n}", t, i, 0
        for n, t in _MIXER[l.kind]:
            yield f"l{i}.mix.{n}", t, i, 0
        if l.experts:
            yield f"l{i}.mlp.router", ROUTER, i, 0
            for e in range(l.experts.count):
                for n, t in (("gate", GATE), ("up", UP), ("down", DOWN)):
                    yield f"l{i}.mlp.e{e}.{n}", t, i, e


class NumuzenModel(StepModel):
    """Weights, caches, states and the step.  `dtype` BF16: bf16 weights, activations and caches with an f32 stream and f32
    states; F32: all f32.  Recurrent layers of `cfg` need their `rank` set (``from_tensors`` reads it off the checkpoint)."""

    abi = "tq_numuzen"

    def __init__(self, dev: QuantComputeDevice, cfg: NumuzenConfig, dtype: int = _lib.BF16, max_slots: int = 64, max_seq: int | None = None):
        from .registry import DEFAULT_MAX_SEQ

        self.dev, self.cfg, self.dtype, self.max_slots = dev, cfg, dtype, max_slots
        self.max_seq = max_seq or DEFAULT_MAX_SEQ
        cc = _CConfig(len(cfg.layers), cfg.width, cfg.vocab, self.max_seq, max_slots, dtype, cfg.eps)
        cl = (_CLayer * len(cfg.layers))()
        for c, l in zip(cl, cfg.layers):
            r, x = l.rot or Rotation(), l.experts or Experts(0, 0, 0, 0.0)
            c.kind, c.heads, c.kv_heads, c.dim, c.vdim, c.window, c.rot_dims, c.rank = l.kind, l.heads, l.kv_heads, l.dim, l.vdim, l.window, r.dims, l.rank
            c.experts, c.top, c.ff, c.limit = x.count, x.top, x.ff, x.limit
            c.scale, c.softcap, c.tau = l.scale, l.softcap, l.tau
            c.rot_base, c.rot_factor, c.rot_original, c.rot_fast, c.rot_slow = r.base, r.factor, r.original, r.fast, r.slow
        h = C.c_void_p()
        dev._check(dev._L.tq_numuzen_create(dev._ctx, C.byref(cc), cl, C.byref(h)))
        self.handle = h.value

    @classmethod
    def from_tensors(cls, dev: QuantComputeDevice, config: dict, tensors: dict, dtype: int = _lib.BF16, max_slots: int = 64,
                     max_seq: int | None = None) -> "NumuzenModel":
        """From a parsed config.json and the tensors of the checkpoint (``read_safetensors``)."""
        cfg = NumuzenConfig.from_dict(config)
        for i, l in enumerate(cfg.layers):
            if l.kind == GLA:
                l.rank = int(need(tensors, f"l{i}.mix.a1").shape[0])
        model = cls(dev, cfg, dtype, max_slots, max_seq)
        try:
            for name, tensor, layer, expert in tensor_names(cfg):
                model.put(tensor, layer, need(tensors, name), expert)
        except Exception:
            model.destroy()
            raise
        return model

    def put(self, tensor: int, layer: int, view: TensorView, expert: int = 0) -> None:
        a, dt, rows, cols = host_array(view)
        self.put_pointer(tensor, layer, a.ctypes.data, dt, rows, cols, expert)

    def put_pointer(self, tensor: int, layer: int, ptr: int, dtype: int, rows: int, cols: int, expert: int = 0) -> None:
        """`ptr`: host or device address of the row-major [rows, cols] tensor."""
        self._call("put", tensor, layer, expert, C.c_void_p(ptr), dtype, rows, cols)
