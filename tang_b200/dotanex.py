"""Dotanex (``tq_dotanex_*`` in include/tangq.h): configuration, weight loading and the model.

A small decoder with several residual streams mixed around every sublayer.  Its mixers are sliding-window attention (per-head
query/key norm, banded rotation, a learned sink per head, values that are the raw keys), latent attention (low-rank queries, one
cached latent and one rotated key part per position, YaRN rotation, output gate) and lightning attention; its feed-forwards are
dense or softmax-routed experts with identity experts and a shared one.  Layers may share another layer's weights.  No
counterpart in the reference.
"""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass, replace

from . import _lib
from .checkpoint import TensorView
from .device import QuantComputeDevice
from .stepmodel import NO_WINDOW, ConfigError, StepModel, host_array, need

# tq_dotanex_tensor
(EMBED, FINAL_NORM, HEAD, NORM1, NORM2, HC1_IN, HC1_OUT, HC1_MIX, HC2_IN, HC2_OUT, HC2_MIX, Q, K, V, G, O, Q_NORM, K_NORM, SINK, O_NORM, DQ, DQ_NORM, UQ,
 DKV, DKV_NORM, UK, UV, ROUTER, CORRECTION, GATE, UP, DOWN, SHARED_GATE, SHARED_UP, SHARED_DOWN) = range(35)

# tq_dotanex_mixer, tq_dotanex_ff
ATTENTION, LATENT, LIGHTNING = range(3)
NONE, DENSE, MOE = range(3)


class _CConfig(C.Structure):
    _fields_ = [(n, C.c_uint32) for n in ("n_layers", "width", "vocab", "streams", "max_seq", "max_slots")] + [("dtype", C.c_int), ("eps", C.c_float), (
        "expand_bytes", C.c_size_t)]


class _CLayer(C.Structure):
    _fields_ = [("kind", C.c_uint32), ("weights_of", C.c_int32)] + [(n, C.c_uint32) for n in (
        "heads", "kv_heads", "dim", "vdim", "window", "rot_dims", "q_rank", "kv_rank", "rot_dim", "ff_kind", "ff", "experts", "identity", "top",
        "shared_ff")] + [(n, C.c_float) for n in ("scale", "limit", "shared_limit")] + [(n, C.c_double) for n in (
            "rot_base", "rot_factor", "rot_original", "rot_low", "rot_high", "rot_fast", "rot_slow")] + [("decay", C.POINTER(C.c_float))]


@dataclass(frozen=True)
class Rotation:
    dims: int = 0
    base: float = 0.0
    factor: float = 0.0       # 0: no scaling
    original: float = 0.0
    low: float = 0.0          # attention
    high: float = 0.0
    fast: float = 0.0         # latent attention
    slow: float = 0.0


@dataclass(frozen=True)
class FeedForward:
    kind: int = NONE
    ff: int = 0               # of the dense one, or of an expert
    experts: int = 0
    identity: int = 0
    top: int = 0
    limit: float = 0.0
    shared_ff: int = 0        # 0: no shared expert
    shared_limit: float = 0.0


@dataclass(frozen=True)
class DotanexLayer:
    kind: int
    heads: int
    dim: int                  # latent attention: without the rotated part
    vdim: int
    scale: float = 0.0
    kv_heads: int = 0
    window: int = NO_WINDOW
    rot: Rotation = Rotation()
    q_rank: int = 0
    kv_rank: int = 0
    rot_dim: int = 0
    decay: tuple = ()
    mlp: FeedForward = FeedForward()
    weights_of: int = -1      # -1: tensors of its own


def _up(n: int, to: int) -> int:
    return (n + to - 1) // to * to


@dataclass
class DotanexConfig:
    vocab: int
    width: int
    streams: int
    eps: float
    layers: list

    @classmethod
    def from_dict(cls, c: dict) -> "DotanexConfig":
        """From the parsed config.json."""
        try:
            layers = [_layer(i, e) for i, e in enumerate(c["layers"])]
            cfg = cls(int(c["vocab"]), int(c["width"]), int(c["streams"]), float(c["norm"]["eps"]), layers)
        except (KeyError, TypeError) as e:
            raise ConfigError(f"config.json lacks {e}") from None
        for i, l in enumerate(layers):
            if l.weights_of >= 0:
                if l.weights_of >= len(layers) or layers[l.weights_of].weights_of >= 0 or replace(l, weights_of=-1) != layers[l.weights_of]:
                    raise ConfigError(f"layer {i}: weights_of must name a layer with tensors of its own and the same entry")
        return cfg

    def cache_bytes_per_token(self, dtype: int) -> int:
        values = sum(2 * l.kv_heads * _up(l.dim, 8) for l in self.layers if l.kind == ATTENTION)
        values += sum(_up(l.kv_rank, 16) + _up(l.rot_dim, 16) for l in self.layers if l.kind == LATENT)
        return values * (4 if dtype == _lib.F32 else 2)

    def state_bytes(self) -> int:
        return 4 * sum(l.heads * l.dim * l.vdim for l in self.layers if l.kind == LIGHTNING)

    def bytes_per_slot(self, dtype: int, max_seq: int) -> int:
        """Device memory that one more concurrent sequence takes."""
        return max_seq * self.cache_bytes_per_token(dtype) + self.state_bytes()


def _rotation(m: dict, keys) -> Rotation:
    rot = m.get("rot") or {"dims": 0, "base": 0.0}
    sc = rot.get("scaling") or {}
    return Rotation(int(rot["dims"]), float(rot["base"]), **{k: float(sc[k]) for k in keys if sc})


def _feed_forward(i: int, mlp: dict | None) -> FeedForward:
    if mlp is None:
        return FeedForward()
    if mlp["kind"] == "dense":
        return FeedForward(DENSE, int(mlp["ff"]))
    if mlp["kind"] != "moe":
        raise ConfigError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
    r, e, s = mlp["router"], mlp["expert"], mlp.get("shared")
    return FeedForward(MOE, int(e["ff"]), int(r["experts"]), int(r.get("identity") or 0), int(r["top"]), float(e["limit"]),
                       *((int(s["ff"]), float(s["limit"])) if s else ()))


def _layer(i: int, e: dict) -> DotanexLayer:
    m = e["mixer"]
    of = e.get("weights_of")
    base = dict(heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), mlp=_feed_forward(i, e.get("mlp")), weights_of=-1 if of is None else int(of))
    if e["type"] == "attention":
        if base["vdim"] != base["dim"]:
            raise ConfigError(f"layer {i}: the values are the keys, so vdim must be dim")
        return DotanexLayer(ATTENTION, scale=float(m["scale"]), kv_heads=int(m["kv_heads"]), window=int((m.get("mask") or {}).get("size", NO_WINDOW)),
                            rot=_rotation(m, ("factor", "low", "high", "original")), **base)
    if e["type"] == "latent_attention":
        rot = _rotation(m, ("factor", "original", "fast", "slow"))
        if rot.dims != int(m["rot_dim"]):
            raise ConfigError(f"layer {i}: all of rot_dim is rotated, so rot.dims must be rot_dim")
        return DotanexLayer(LATENT, scale=float(m["scale"]), rot=rot, q_rank=int(m["q_rank"]), kv_rank=int(m["kv_rank"]), rot_dim=int(m["rot_dim"]), **base)
    if e["type"] == "lightning":
        decay = tuple(float(d) for d in m["decay"])
        if len(decay) != base["heads"]:
            raise ConfigError(f"layer {i}: {len(decay)} decays for {base['heads']} heads")
        return DotanexLayer(LIGHTNING, decay=decay, **base)
    raise ConfigError(f"layer {i}: unknown mixer {e['type']!r}")


_MIXER = {ATTENTION: (("q", Q), ("k", K), ("q.norm", Q_NORM), ("k.norm", K_NORM), ("sink", SINK), ("o", O)),
          LATENT: (("dq", DQ), ("dq.norm", DQ_NORM), ("uq", UQ), ("dkv", DKV), ("dkv.norm", DKV_NORM), ("uk", UK), ("uv", UV), ("g", G), ("o", O)),
          LIGHTNING: (("q", Q), ("k", K), ("v", V), ("g", G), ("norm", O_NORM), ("o", O))}
_FF = (("gate", GATE), ("up", UP), ("down", DOWN))


def tensor_names(cfg: DotanexConfig):
    """(name, tensor, layer, expert) of every tensor of the checkpoint."""
    yield from (("embed", EMBED, 0, 0), ("final.norm", FINAL_NORM, 0, 0), ("head", HEAD, 0, 0))
    for i, l in enumerate(cfg.layers):
        if l.weights_of >= 0:
            continue
        names = [("norm1", NORM1), ("hc1.in", HC1_IN), ("hc1.out", HC1_OUT), ("hc1.mix", HC1_MIX)]
        if l.mlp.kind != NONE:
            names += [("norm2", NORM2), ("hc2.in", HC2_IN), ("hc2.out", HC2_OUT), ("hc2.mix", HC2_MIX)]
        names += [(f"mix.{n}", t) for n, t in _MIXER[l.kind]]
        if l.mlp.kind == DENSE:
            names += [(f"mlp.{n}", t) for n, t in _FF]
        elif l.mlp.kind == MOE:
            names += [("mlp.router", ROUTER), ("mlp.correction", CORRECTION)]
            if l.mlp.shared_ff:
                names += [("mlp.shared.gate", SHARED_GATE), ("mlp.shared.up", SHARED_UP), ("mlp.shared.down", SHARED_DOWN)]
        for n, t in names:
            yield f"l{i}.{n}", t, i, 0
        for e in range(l.mlp.experts):
            for n, t in _FF:
                yield f"l{i}.mlp.e{e}.{n}", t, i, e


class DotanexModel(StepModel):
    """Weights, caches, states and the step.  `dtype` BF16: bf16 weights, activations and caches with f32 streams and states; F32:
    all f32.  ``trace`` receives the sum of the streams after each layer.  `expand_bytes`: see tq_dotanex_config."""

    abi = "tq_dotanex"

    def __init__(self, dev: QuantComputeDevice, cfg: DotanexConfig, dtype: int = _lib.BF16, max_slots: int = 64, max_seq: int | None = None,
                 expand_bytes: int = 0):
        from .registry import DEFAULT_MAX_SEQ

        self.dev, self.cfg, self.dtype, self.max_slots = dev, cfg, dtype, max_slots
        self.max_seq = max_seq or DEFAULT_MAX_SEQ
        cc = _CConfig(len(cfg.layers), cfg.width, cfg.vocab, cfg.streams, self.max_seq, max_slots, dtype, cfg.eps, expand_bytes)
        cl, keep = (_CLayer * len(cfg.layers))(), []
        for c, l in zip(cl, cfg.layers):
            for n in ("kind", "weights_of", "heads", "kv_heads", "dim", "vdim", "window", "q_rank", "kv_rank", "rot_dim", "scale"):
                setattr(c, n, getattr(l, n))
            for n in ("ff", "experts", "identity", "top", "shared_ff", "limit", "shared_limit"):
                setattr(c, n, getattr(l.mlp, n))
            for n in ("dims", "base", "factor", "original", "low", "high", "fast", "slow"):
                setattr(c, f"rot_{n}", getattr(l.rot, n))
            c.ff_kind = l.mlp.kind
            if l.decay:
                keep.append((C.c_float * len(l.decay))(*l.decay))
                c.decay = C.cast(keep[-1], C.POINTER(C.c_float))
        h = C.c_void_p()
        dev._check(dev._L.tq_dotanex_create(dev._ctx, C.byref(cc), cl, C.byref(h)))
        self.handle = h.value

    @classmethod
    def from_tensors(cls, dev: QuantComputeDevice, config: dict, tensors: dict, dtype: int = _lib.BF16, max_slots: int = 64,
                     max_seq: int | None = None, expand_bytes: int = 0) -> "DotanexModel":
        """From a parsed config.json and the tensors of the checkpoint (``read_safetensors``)."""
        cfg = DotanexConfig.from_dict(config)
        model = cls(dev, cfg, dtype, max_slots, max_seq, expand_bytes)
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
