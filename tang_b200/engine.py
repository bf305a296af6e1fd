"""Cache slots and ragged batching over a model that has ``step`` (``StepModel``).

Requests are named by the caller; each holds one cache slot from ``open`` (or its first ``step``) to ``close``.  A step
takes the next tokens of any set of requests, packs them into one batch without padding -- in portions of at most
`max_rows` rows when prompts are long -- and returns the logits that were asked for.
"""
from __future__ import annotations

import numpy as np

from . import _lib
from ._lib import TQ_EINVAL, TQ_ENOMEM, TangqError


class SlotPool:
    """Which request owns which cache slot, and how many positions it holds."""

    def __init__(self, n_slots: int):
        self.free = list(range(n_slots - 1, -1, -1))
        self.slot, self.length = {}, {}

    def open(self, request) -> int:
        if request in self.slot:
            raise TangqError(TQ_EINVAL, f"request {request!r} is open already")
        if not self.free:
            raise TangqError(TQ_ENOMEM, "no free cache slot")
        self.slot[request], self.length[request] = self.free.pop(), 0
        return self.slot[request]

    def close(self, request) -> None:
        self.free.append(self.slot.pop(request))
        del self.length[request]


def portions(lengths, max_rows: int):
    """Cuts sequences of the given lengths into batches of at most max_rows rows: a list of lists of
    (sequence, first token, number of tokens), every sequence's tokens in order."""
    out, batch, used = [], [], 0
    for s, n in enumerate(lengths):
        at = 0
        while at < n:
            take = min(n - at, max_rows - used)
            if take:
                batch.append((s, at, take))
                at += take
                used += take
            if used == max_rows:
                out.append(batch)
                batch, used = [], 0
    if batch:
        out.append(batch)
    return out


class Engine:
    def __init__(self, model, max_rows: int = 16384):
        self.model, self.dev, self.max_rows = model, model.dev, max_rows
        self.pool = SlotPool(model.max_slots)
        self._ints = self._logits = None

    def open(self, request) -> int:
        return self.pool.open(request)

    def close(self, request) -> None:
        self.pool.close(request)

    def step(self, entries) -> np.ndarray:
        """entries: (request, next tokens, places among them whose logits are wanted).  Returns f32 [wanted, vocab] in the
        order of the entries and of their places."""
        vocab, max_seq = self.model.cfg.vocab, self.model.max_seq
        entries = [(r, np.asarray(t, np.int32).reshape(-1), list(w)) for r, t, w in entries]
        if len({r for r, _, _ in entries}) != len(entries):
            raise TangqError(TQ_EINVAL, "a step takes each request once")
        for r, t, w in entries:
            if any(not 0 <= i < len(t) for i in w) or not len(t):
                raise TangqError(TQ_EINVAL, f"request {r!r}: no tokens, or a wanted place outside them")
            if len(t) and (t.min() < 0 or t.max() >= vocab):
                raise TangqError(TQ_EINVAL, f"request {r!r}: token outside the vocabulary")
            if self.pool.length.get(r, 0) + len(t) > max_seq:
                raise TangqError(TQ_EINVAL, f"request {r!r}: more than {max_seq} positions")
        for r, _, _ in entries:
            if r not in self.pool.slot:
                self.pool.open(r)
        first = np.cumsum([0] + [len(w) for _, _, w in entries])
        out = np.empty((int(first[-1]), vocab), np.float32)
        for batch in portions([len(t) for _, t, _ in entries], self.max_rows):
            where, rows = [], []                      # output row / batch row of every wanted place of this batch
            row = 0
            for s, at, n in batch:
                for k, place in enumerate(entries[s][2]):
                    if at <= place < at + n:
                        where.append(int(first[s]) + k)
                        rows.append(row + place - at)
                row += n
            got = self._run([(entries[s][0], entries[s][1][at:at + n]) for s, at, n in batch], rows)
            if where:
                out[where] = got
        return out

    def _run(self, batch, logit_rows) -> np.ndarray | None:
        dev, pool, vocab = self.dev, self.pool, self.model.cfg.vocab
        counts = [len(t) for _, t in batch]
        B, R, n = len(batch), sum(counts), len(logit_rows)
        starts = [pool.length[r] for r, _ in batch]
        parts = [np.concatenate([t for _, t in batch]), np.cumsum([0] + counts), starts, [pool.slot[r] for r, _ in batch], logit_rows]
        # one upload for all the integers of the step
        ints = np.concatenate([np.asarray(p, np.int32) for p in parts])
        if self._ints is None or self._ints.n < ints.size:
            self._ints = dev.alloc(max(4096, 2 * ints.size), _lib.I32)
        dev.upload_into(self._ints, ints)
        views, off = [], 0
        for p in parts:
            views.append(self._view(self._ints, off, len(p)))
            off += len(p)
        if n and (self._logits is None or self._logits.n < n * vocab):
            self._logits = dev.alloc(n * vocab, _lib.F32)
        tok, seq_rows, starts_b, slots_b, rows_b = views
        max_q = max(counts)
        self.model.step(tok, R, None if max_q == 1 else seq_rows, starts_b, slots_b, B, max_q, max(s + c for s, c in zip(starts, counts)),
                        rows_b if n else None, n, self._logits if n else None)
        for (r, _), c in zip(batch, counts):
            pool.length[r] += c
        dev.sync()
        return dev.download(self._view(self._logits, 0, n * vocab)).reshape(n, vocab) if n else None

    def _view(self, buf, first: int, n: int):
        from .device import Buffer, _SIZE_OF

        return Buffer(self.dev, buf.ptr + first * _SIZE_OF[buf.dtype], n, buf.dtype, owns=False)
