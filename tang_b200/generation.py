"""The generation loop shared by the models (``generate``, crates/tang-infer/src/sampling.rs:229-256)."""
from __future__ import annotations

import ctypes as C

import numpy as np

from . import _lib
from .device import SamplerConfig


def decode_loop(dev, decode, prompts, n_new: int, vocab: int, sampling=None, seed: int = 42, comm_world: int = 1) -> np.ndarray:
    """Draws `n_new` tokens for every prompt (sequences of ids, any lengths) whose tokens but the last are in the model's
    cache already.  decode(tokens, positions, logits) launches the model's step for one new token per sequence; step ->
    ``Sampler::sample`` -> advance runs once eagerly (workspaces) and is then replayed as one CUDA graph, the logits and the
    growing histories staying on the device.  Every sequence owns an LCG seeded with `seed`; the repetition penalty sees
    prompt and generated tokens.  Returns int32 [batch, n_new]."""
    L = dev._L
    lens = np.array([len(p) for p in prompts], np.int32)
    B, ld = len(prompts), int(lens.max()) + n_new
    cfg = sampling if sampling is not None else SamplerConfig(0.0, 0, 1.0, 1.0)
    hist = np.zeros((B, ld), np.int32)
    for row, p in zip(hist, prompts):
        row[:len(p)] = p
    logits = dev.alloc(B * vocab, _lib.F32)
    tok = dev.upload(np.array([p[-1] for p in prompts], np.int32), _lib.I32)
    pos = dev.upload(lens - 1, _lib.I32)
    chosen = dev.alloc(B, _lib.I32)
    hist_d = dev.upload(hist, _lib.I32)
    lens_d = dev.upload(lens, _lib.I32)
    rng = dev.upload(np.full(B, seed, np.uint64).view(np.float64), _lib.F64)

    def one():
        decode(tok, pos, logits)
        dev._check(L.tq_sample(dev._ctx, C.c_void_p(logits.ptr), comm_world, B, vocab // comm_world, C.byref(cfg),
                               C.c_void_p(rng.ptr), C.c_void_p(hist_d.ptr), C.c_void_p(lens_d.ptr), ld, C.c_void_p(chosen.ptr)))
        dev._check(L.tq_generate_advance(dev._ctx, C.c_void_p(chosen.ptr), B, C.c_void_p(tok.ptr), C.c_void_p(pos.ptr),
                                         C.c_void_p(hist_d.ptr), ld, C.c_void_p(0), C.c_void_p(lens_d.ptr)))

    one()
    if n_new > 1:
        dev.sync()
        dev.begin_capture()
        one()
        graph = dev.end_capture()
        for _ in range(n_new - 1):
            graph.launch()
        dev.sync()
        graph.free()
    dev.sync()
    out = hist_d.to_vec().reshape(B, ld)
    return np.stack([out[b, n:n + n_new] for b, n in enumerate(lens)])


def check_lengths(prompts, n_new: int, max_seq: int) -> None:
    if n_new < 1 or not len(prompts) or any(len(p) < 1 for p in prompts):
        raise _lib.TangqError(_lib.TQ_EINVAL, "generate: need at least one prompt token and one new token")
    if max(len(p) for p in prompts) + n_new > max_seq:
        raise _lib.TangqError(_lib.TQ_EINVAL, "generate: prompt + new tokens exceed max_seq")
