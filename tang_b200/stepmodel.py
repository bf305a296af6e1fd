"""What checkpoint models over ragged steps share: ``step`` / ``decode`` / ``trace`` over their C entry points, loading a
tensor, and ``generate``."""
from __future__ import annotations

import ctypes as C

import numpy as np

from . import _lib
from .checkpoint import SafetensorsError, TensorView
from .device import Buffer
from .generation import check_lengths, decode_loop


class ConfigError(ValueError):
    """A configuration that is not of the design it names."""


NO_WINDOW = 0x7FFFFFFF


def need(tensors: dict, name: str) -> TensorView:
    if name not in tensors:
        raise SafetensorsError(f"tensor {name!r} is missing")
    return tensors[name]


def host_array(view: TensorView):
    """(contiguous array, its dtype code, rows, columns) of a checkpoint tensor; a vector is one row."""
    if view.dtype == "BF16":
        a, dt = np.ascontiguousarray(view.data), _lib.BF16
    else:
        a, dt = np.ascontiguousarray(view.to_f32()), _lib.F32
    rows, cols = view.shape if len(view.shape) == 2 else (1, int(np.prod(view.shape)))
    return a, dt, rows, cols


class StepModel:
    """Subclasses set ``abi`` (the prefix of their C entry points) and, when they are made, dev, cfg, dtype, max_slots, max_seq
    and handle."""

    abi = ""

    def _call(self, name: str, *args) -> None:
        self.dev._check(getattr(self.dev._L, f"{self.abi}_{name}")(C.c_void_p(self.handle), *args))

    def step(self, tokens: Buffer, rows: int, seq_rows: Buffer | None, starts: Buffer, slots: Buffer | None, n_seqs: int, max_q: int,
             max_len: int, logit_rows: Buffer | None, n_logits: int, logits: Buffer | None) -> None:
        """One step over a ragged batch (``tq_tofazen_step``); asynchronous."""
        ptr = lambda b: C.c_void_p(b.ptr if b is not None else 0)
        self._call("step", ptr(tokens), rows, ptr(seq_rows), ptr(starts), ptr(slots), n_seqs, max_q, max_len, ptr(logit_rows), n_logits, ptr(logits))

    def decode(self, token_ids: Buffer, positions: Buffer, batch: int, max_len: int, logits: Buffer, slots: Buffer | None = None) -> None:
        """One new token for each of `batch` sequences (slots 0 .. batch-1 unless given)."""
        self.step(token_ids, batch, None, positions, slots, batch, 1, max_len, None, batch, logits)

    def trace(self, streams: Buffer | None) -> None:
        """While set, every step leaves the f32 stream after each layer in `streams` [layers, rows, width]."""
        self._call("trace", C.c_void_p(streams.ptr if streams is not None else 0))

    def generate(self, prompts, n_new: int, sampling=None, seed: int = 42) -> np.ndarray:
        """``generate`` for a batch of prompts of any lengths: the prompts run as one ragged batch (all tokens but the
        last of each), then decode -> sample -> advance as one replayed graph.  Returns int32 [batch, n_new]."""
        from .engine import Engine

        prompts = [np.asarray(p, np.int32) for p in prompts]
        check_lengths(prompts, n_new, self.max_seq)
        engine = Engine(self)
        heads = [(i, p[:-1], ()) for i, p in enumerate(prompts)]
        slots = [engine.open(i) for i in range(len(prompts))]
        if any(len(t) for _, t, _ in heads):
            engine.step([h for h in heads if len(h[1])])
        B, longest = len(prompts), max(len(p) for p in prompts)
        slot_buf = self.dev.upload(np.array(slots, np.int32), _lib.I32)
        return decode_loop(self.dev, lambda tok, pos, logits: self.decode(tok, pos, B, longest + n_new, logits, slot_buf), prompts, n_new,
                           self.cfg.vocab, sampling, seed)

    def generate_greedy(self, prompts, n_new: int) -> np.ndarray:
        return self.generate(prompts, n_new, None)

    def destroy(self) -> None:
        if self.handle:
            self._call("destroy")
            self.handle = 0
