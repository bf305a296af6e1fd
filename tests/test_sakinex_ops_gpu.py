"""The mechanisms of the Sakinex family one by one on the device, against the numpy implementation: short convolutions, convolved
heads with their caches and pooled blocks, attention over pooled blocks and a window, minGRU, the stream step, biased routing.
What keeps a state runs in steps of every kind over slots that another sequence has used."""
import ctypes as C

import numpy as np
import pytest

import sakinex_oracle as X
from util import bf16_round

pytestmark = pytest.mark.gpu

F32, BF16, I32 = 0, 1, 5
MAX_SEQ = 320


class AttnConfig(C.Structure):
    _fields_ = [(n, C.c_uint32) for n in ("heads", "kv_heads", "dim", "vdim", "window")] + [(n, C.c_float) for n in ("scale", "softcap", "sink")]


class HeadsConfig(C.Structure):
    _fields_ = [(n, C.c_uint32) for n in ("heads", "kv_heads", "dim", "vdim", "k0", "v0", "channels", "taps", "rot_dims")] + [("norm", C.c_int)] + [
        (n, C.c_uint32) for n in ("pool", "pool_rows")] + [(n, C.c_float) for n in ("rot_mult", "eps")]


@pytest.fixture(scope="module")
def dev():
    import tang_b200

    d = tang_b200.QuantComputeDevice(0)
    yield d
    d.close()


KEEP = []          # buffers of the running test: a temporary must outlive the launch that reads it


@pytest.fixture(autouse=True)
def _release(dev):
    yield
    dev.sync()
    KEEP.clear()


def ptr(b):
    KEEP.append(b)
    return C.c_void_p(b.ptr if b is not None else 0)


def up(dev, x, dt=F32):
    """Upload of an array in the given format; returns (buffer, the values it holds)."""
    x = np.ascontiguousarray(x, np.float32)
    if dt == F32:
        return dev.upload(x.reshape(-1), F32), x.astype(np.float64)
    bits, val = bf16_round(x)
    return dev.upload(bits.reshape(-1), BF16), val.reshape(x.shape).astype(np.float64)


def down(buf, dt, shape):
    a = np.asarray(buf.to_vec())
    if dt == BF16 and a.dtype == np.uint16:
        a = (a.astype(np.uint32) << 16).view(np.float32)
    return np.asarray(a, np.float64).reshape(shape)


def ints(dev, x):
    return dev.upload(np.asarray(x, np.int32).reshape(-1), I32)


def rel(got, want):
    """Largest error, relative to the element and the root mean square (an output in bf16 carries 0.002 of its element)."""
    return (np.abs(got - want) / (np.abs(want) + np.sqrt(np.mean(np.square(want))) + 1e-30)).max()


def pad(x, to):
    """Zeros behind the last axis up to a multiple of `to`."""
    return np.pad(x, [(0, 0)] * (x.ndim - 1) + [(0, -x.shape[-1] % to)])


class Batch:
    """Sequences of (slot, start, rows) over caches of max_seq rows."""

    def __init__(self, dev, seqs, max_seq=MAX_SEQ):
        self.seqs, self.max_seq = seqs, max_seq
        counts = [n for _, _, n in seqs]
        self.rows, self.max_q, self.max_len = sum(counts), max(counts), max(s + n for _, s, n in seqs)
        self.pos = np.concatenate([np.arange(s, s + n) for _, s, n in seqs])
        self.crow = np.concatenate([slot * max_seq + np.arange(s, s + n) for slot, s, n in seqs])
        self.first = np.cumsum([0] + counts)
        self.pos_d, self.crow_d = ints(dev, self.pos), ints(dev, self.crow)
        self.rows_d = ints(dev, self.first) if self.max_q > 1 else None

    def tail(self):
        """(row offsets, positions, cache rows, sequences, rows, longest) as the entry points take them."""
        return ptr(self.rows_d), ptr(self.pos_d), ptr(self.crow_d), len(self.seqs), self.rows, self.max_q


# Steps over three slots: prompts, portions down to one and two rows among longer ones, single rows, and slots that are used again.
# A sequence is (slot, generation).
STEPS = [[(0, 0, 70), (2, 0, 1), (1, 0, 5)], [(1, 0, 2), (0, 0, 1), (2, 0, 33)], [(0, 0, 1), (1, 0, 1), (2, 0, 1)], [(2, 0, 1)], [(1, 1, 2), (0, 0, 60)],
         [(1, 1, 1), (0, 1, 1), (2, 0, 1)], [(0, 1, 1), (1, 1, 1)], [(0, 1, 1), (1, 1, 130)], [(2, 1, 3), (0, 1, 2)], [(2, 1, 1), (1, 1, 1), (0, 1, 1)]]


def walk(steps=STEPS):
    """(sequences of a step as (slot, start, rows), their names) for every step."""
    at = {}
    for step in steps:
        seqs = []
        for slot, gen, n in step:
            seqs.append((slot, at.get((slot, gen), 0), n))
            at[slot, gen] = at.get((slot, gen), 0) + n
        yield seqs, [(slot, gen) for slot, gen, _ in step]


def lengths(steps=STEPS):
    out = {}
    for step in steps:
        for slot, gen, n in step:
            out[slot, gen] = out.get((slot, gen), 0) + n
    return out


@pytest.mark.parametrize("dt,tol", [(F32, 2e-6), (BF16, 6e-3)])
@pytest.mark.parametrize("channels,taps", [(72, 1), (72, 2), (256, 3), (1024, 4), (136, 7), (37, 3), (8, 5)])
def test_short_convolution(dev, dt, tol, channels, taps):
    rng = np.random.default_rng(channels + taps)
    w, wv = up(dev, rng.standard_normal((taps, channels)))
    state = up(dev, rng.standard_normal((3, max(taps - 1, 1), channels)) * 50, dt)[0]       # (what others left)
    x = {s: bf16_round(rng.standard_normal((n, channels)).astype(np.float32))[1].astype(np.float64) for s, n in lengths().items()}
    want = {s: r + X.conv(r, wv.T, np.zeros((taps - 1, channels)))[0] for s, r in x.items()}
    ld = (channels + 7) // 8 * 8 + 8
    for seqs, names in walk():
        b = Batch(dev, seqs)
        rows = np.concatenate([x[s][a:a + n] for s, (_, a, n) in zip(names, seqs)])
        xd = up(dev, np.pad(rows, [(0, 0), (0, ld - channels)]), dt)[0]
        out = up(dev, np.full((b.rows, ld), 7.0), dt)[0]
        r, p, c, n_seqs, n_rows, max_q = b.tail()
        dev._check(dev._L.tq_conv_residual(dev._ctx, dt, channels, taps, ptr(w), ptr(state), MAX_SEQ, 3 * MAX_SEQ, ptr(xd), ld, r, p, c, n_seqs, n_rows, max_q, b.max_len,
                                           ptr(out), ld))
        got = down(out, dt, (b.rows, ld))
        assert (got[:, channels:] == 7).all()
        assert rel(got[:, :channels], np.concatenate([want[s][a:a + n] for s, (_, a, n) in zip(names, seqs)])) < tol


@pytest.mark.parametrize("dt,tol", [(F32, 6e-5), (BF16, 1.5e-2)])
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,taps,rot,pool,norm", [
    (4, 2, 32, 32, 3, 32, 4, True), (5, 1, 33, 21, 4, 10, 3, True), (12, 3, 64, 128, 2, 32, 16, True), (3, 3, 16, 8, 1, 0, 1, True), (2, 2, 24, 40, 6, 8, 7, True),
    (2, 1, 128, 64, 0, 128, 64, True), (6, 2, 16, 24, 3, 16, 0, False), (2, 1, 256, 256, 4, 64, 10, True), (3, 1, 9, 7, 0, 4, 5, True)])
def test_convolved_heads_caches_and_pooled_blocks(dev, dt, tol, heads, kv_heads, dim, vdim, taps, rot, pool, norm):
    rng = np.random.default_rng(dim + vdim)
    up16 = lambda n: (n + 15) // 16 * 16
    up8 = lambda n: (n + 7) // 8 * 8
    eps, mult = 1e-5, 1.25
    k0, v0 = up16(heads * dim), up16(heads * dim) + up16(kv_heads * dim)
    ch = v0 + up16(kv_heads * vdim)
    cols = np.concatenate([np.arange(heads * dim), k0 + np.arange(kv_heads * dim), v0 + np.arange(kv_heads * vdim)])
    w = np.zeros((max(taps, 1), ch))
    w[:, cols] = rng.standard_normal((max(taps, 1), len(cols)))
    wd, wv = up(dev, w) if taps else (None, None)
    state = up(dev, rng.standard_normal((3, max(taps - 1, 1), ch)) * 50, dt)[0]
    fr, fv = up(dev, np.append(rng.random(rot // 2), 0.0))
    x = {s: np.zeros((n, ch)) for s, n in lengths().items()}
    for s in x:
        x[s][:, cols] = bf16_round(rng.standard_normal((len(x[s]), len(cols))).astype(np.float32))[1]
    full = {s: X.conv(r, wv.T, np.zeros((taps - 1, ch)))[0] if taps else r for s, r in x.items()}

    def turned(rows, n_heads):
        y = np.array([X.rotate(r, t, fv[:rot // 2], mult) for t, r in enumerate(rows.reshape(len(rows), n_heads, dim))])
        return X.rms(y, eps) if norm else y

    q = {s: turned(r[:, :heads * dim], heads) for s, r in full.items()}
    k = {s: turned(r[:, k0:k0 + kv_heads * dim], kv_heads) for s, r in full.items()}
    v = {s: r[:, v0:v0 + kv_heads * vdim].reshape(-1, kv_heads, vdim) for s, r in full.items()}
    prow = MAX_SEQ // pool if pool else 0
    zeros = lambda *shape: up(dev, np.zeros(shape), dt)[0]
    keys, vals = zeros(3 * MAX_SEQ, kv_heads, up8(dim)), zeros(3 * MAX_SEQ, kv_heads, up8(vdim))
    pk, pv = zeros(3 * prow + 1, kv_heads, up8(dim)), zeros(3 * prow + 1, kv_heads, up8(vdim))
    cfg = HeadsConfig(heads, kv_heads, dim, vdim, k0, v0, ch, taps, rot, int(norm), pool, prow, mult, eps)
    for seqs, names in walk():
        b = Batch(dev, seqs)
        raw = up(dev, np.concatenate([x[s][a:a + n] for s, (_, a, n) in zip(names, seqs)]), dt)[0]
        out = dev.alloc(b.rows * up8(heads * dim), dt)
        r, p, c, n_seqs, n_rows, max_q = b.tail()
        dev._check(dev._L.tq_conv_heads(dev._ctx, C.byref(cfg), dt, ptr(raw), ch, ptr(wd), ptr(state), ptr(fr), MAX_SEQ, 3 * MAX_SEQ, r, p, c, n_seqs, n_rows, max_q,
                                        b.max_len, ptr(out), up8(heads * dim), ptr(keys), ptr(vals), ptr(pk), ptr(pv)))
        got = down(out, dt, (b.rows, up8(heads * dim)))[:, :heads * dim].reshape(b.rows, heads, dim)
        assert rel(got, np.concatenate([q[s][a:a + n] for s, (_, a, n) in zip(names, seqs)])) < tol
        gk, gv = down(keys, dt, (3, MAX_SEQ, kv_heads, up8(dim))), down(vals, dt, (3, MAX_SEQ, kv_heads, up8(vdim)))
        gpk, gpv = (down(buf, dt, (3 * prow + 1, kv_heads, up8(e))) for buf, e in ((pk, dim), (pv, vdim)))
        for s, (slot, a, n) in zip(names, seqs):
            end = a + n
            assert rel(gk[slot, :end, :, :dim], k[s][:end]) < tol and rel(gv[slot, :end, :, :vdim], v[s][:end]) < tol
            for blk in range((end - 1) // pool if pool else 0):      # complete one row before the last one
                row = slot * prow + blk
                for g, cache, d in ((gpk, gk, dim), (gpv, gv, vdim)):
                    want = X.pooled(cache[slot, :end, :, :d], blk, pool)
                    assert np.abs(g[row, :, :d] - want).max() < (1e-6 if dt == F32 else 8e-3 * np.abs(want).max()), (s, blk)
        assert not gk[..., dim:].any() and not gv[..., vdim:].any() and not gpk[3 * prow:].any() and not gpv[3 * prow:].any()


@pytest.mark.parametrize("dt,tol", [(F32, 1e-5), (BF16, 2e-2)])      # (in bf16 the pooled rows carry 0.002)
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,window,pool", [(4, 2, 32, 32, 20, 4), (6, 1, 40, 24, 65, 16), (18, 1, 16, 16, 64, 1), (3, 3, 136, 40, 1, 2), (8, 2, 128, 128, 100, 7),
                                                                 (2, 1, 264, 16, 33, 5), (2, 2, 8, 80, 3, 40), (1, 1, 64, 256, 128, 64)])
@pytest.mark.parametrize("seqs", [[(0, 0, 70), (1, 33, 5), (2, 200, 1)], [(0, 319, 1), (1, 0, 1), (2, 64, 1)], [(1, 0, 320)], [(2, 107, 130), (0, 64, 2)]])
def test_attention_over_pooled_blocks_and_a_window(dev, dt, tol, heads, kv_heads, dim, vdim, window, pool, seqs):
    rng = np.random.default_rng(dim + window)
    b = Batch(dev, seqs)
    prow, scale, factor = MAX_SEQ // pool, 1.3 * dim ** -0.5, 0.6
    q, qv = up(dev, rng.standard_normal((b.rows, heads, dim)) * 2, dt)
    keys, values = rng.standard_normal((3 * MAX_SEQ, kv_heads, dim)), rng.standard_normal((3 * MAX_SEQ, kv_heads, vdim))
    # blocks that nobody sees yet hold what would show
    pk, pv = np.full((3 * prow, kv_heads, dim), 3.0), np.full((3 * prow, kv_heads, vdim), 100.0)
    k, kv = up(dev, pad(keys, 8), dt)
    v, vv = up(dev, pad(values, 8), dt)
    for slot, s, n in seqs:
        for blk in X.seen_blocks(s + n - 1, window, pool):
            pk[slot * prow + blk] = X.pooled(kv[slot * MAX_SEQ:, :, :dim], blk, pool)
            pv[slot * prow + blk] = X.pooled(vv[slot * MAX_SEQ:, :, :vdim], blk, pool)
    pkd, pvd = up(dev, pad(pk, 8), dt)[0], up(dev, pad(pv, 8), dt)[0]
    cfg = AttnConfig(heads, kv_heads, dim, vdim, window, scale, 0.0, -np.inf)
    out = dev.alloc(b.rows * heads * vdim, dt)
    r, p, c, n_seqs, n_rows, max_q = b.tail()
    dev._check(dev._L.tq_window_attention_pooled(dev._ctx, C.byref(cfg), None, dt, ptr(q), heads * dim, None, 0, ptr(k), ptr(v), 3 * MAX_SEQ, pool, ptr(pkd), ptr(pvd), prow,
                                                 MAX_SEQ, factor, r, p, c, n_seqs, n_rows, max_q, b.max_len, ptr(out), heads * vdim))
    got = down(out, dt, (b.rows, heads, vdim))
    for i, (slot, start, n) in enumerate(seqs):
        rows = slice(slot * MAX_SEQ, slot * MAX_SEQ + start + n)
        want = factor * X.attention(qv[b.first[i]:b.first[i + 1]], kv[rows, :, :dim], vv[rows, :, :vdim], start, scale, window, pool)
        assert rel(got[b.first[i]:b.first[i + 1]], want) < tol


@pytest.mark.parametrize("heads,kv_heads,dim", [(2, 1, 24), (16, 2, 64)])
def test_a_long_row_of_pooled_blocks_is_split_over_ctas(dev, heads, kv_heads, dim):
    """Many tiles of blocks in one decode step, one of them far away holding nearly all the weight."""
    rng = np.random.default_rng(dim)
    n, window, pool = 4096, 70, 4
    b = Batch(dev, [(0, n - 1, 1)], n)
    q, qv = up(dev, rng.standard_normal((1, heads, dim)), BF16)
    pk, pkv = up(dev, rng.standard_normal((n // pool, kv_heads, dim)), BF16)
    for at in (0, 63, 64, 500, (n - window) // pool - 1, (n - window) // pool):
        near = rng.standard_normal((n, kv_heads, dim))
        blocks = pkv.copy()
        blocks[at] = 3 * qv[0, ::heads // kv_heads]
        k, kv = up(dev, near, BF16)
        pkd, blocks = up(dev, blocks, BF16)
        out = dev.alloc(heads * dim, BF16)
        cfg = AttnConfig(heads, kv_heads, dim, dim, window, dim ** -0.5, 0.0, -np.inf)
        dev._check(dev._L.tq_window_attention_pooled(dev._ctx, C.byref(cfg), None, BF16, ptr(q), heads * dim, None, 0, ptr(k), ptr(k), n, pool, ptr(pkd), ptr(pkd), n // pool,
                                                     n, 1.0, None, ptr(b.pos_d), ptr(b.crow_d), 1, 1, 1, n, ptr(out), heads * dim))
        seen = np.concatenate([blocks[:(n - window) // pool], kv[n - window:]])
        got = down(out, BF16, (heads, dim))
        for h in range(heads):
            s = seen[:, h // (heads // kv_heads)] @ qv[0, h] * dim ** -0.5
            e = np.exp(s - s.max())
            assert rel(got[h], e / e.sum() @ seen[:, h // (heads // kv_heads)]) < 1e-2, (at, h)


@pytest.mark.parametrize("dt,tol", [(F32, 3e-6), (BF16, 6e-3)])
@pytest.mark.parametrize("width", [1, 13, 32, 96, 514])
def test_min_gru(dev, dt, tol, width):
    rng = np.random.default_rng(width)
    factor, up16 = 1.1, (width + 15) // 16 * 16
    zb, zbv = up(dev, rng.standard_normal(width) - 2)
    ub, ubv = up(dev, rng.standard_normal(width))
    state = up(dev, rng.standard_normal((3, (width + 1) // 2 * 2)) * 50)[0]
    steps = STEPS + [[(2, 2, 300)], [(2, 2, 1)], [(2, 2, 2)]]
    x = {s: bf16_round((rng.standard_normal((n, 3, width)) * 2).astype(np.float32))[1].astype(np.float64) for s, n in lengths(steps).items()}
    # a gate that is shut over long stretches carries the first rows' state far
    for s in x:
        x[s][5:, 0, ::3] -= 6
    want = {s: X.min_gru(r[:, 0] + zbv, r[:, 1] + ubv, np.zeros(width))[0] * X.silu(r[:, 2]) * factor for s, r in x.items()}
    for seqs, names in walk(steps):
        b = Batch(dev, seqs)
        rows = np.concatenate([x[s][a:a + n] for s, (_, a, n) in zip(names, seqs)])
        xd = up(dev, np.pad(rows, [(0, 0), (0, 0), (0, up16 - width)]), dt)[0]
        KEEP.append(xd)
        out = up(dev, np.full((b.rows, up16), 7.0), dt)[0]
        at = lambda i: C.c_void_p(xd.ptr + i * up16 * (4 if dt == F32 else 2))
        r, p, c, n_seqs, n_rows, max_q = b.tail()
        dev._check(dev._L.tq_min_gru(dev._ctx, dt, width, at(0), at(1), at(2), 3 * up16, ptr(zb), ptr(ub), factor, ptr(state), MAX_SEQ, 3 * MAX_SEQ, r, p, c, n_seqs, n_rows,
                                     max_q, ptr(out), up16))
        got = down(out, dt, (b.rows, up16))
        assert (got[:, width:] == 7).all()
        assert rel(got[:, :width], np.concatenate([want[s][a:a + n] for s, (_, a, n) in zip(names, seqs)])) < tol


@pytest.mark.parametrize("dt,tol", [(F32, 3e-6), (BF16, 2e-2)])      # (in bf16 every input of the convolution carries 0.002)
@pytest.mark.parametrize("width,taps", [(72, 3), (101, 2), (1024, 4), (4100, 1), (264, 6)])
def test_stream_step(dev, dt, tol, width, taps):
    """Residual with a factor, weighted expert rows, a row behind a sigmoid gate, rows added afterwards, the next norm and its convolution,
    token by token over slots that are used again."""
    rng = np.random.default_rng(width)
    eps, ld, n_y, mult = 1e-4, (width + 7) // 8 * 8, 3, 0.37
    gain, gv = up(dev, rng.standard_normal(width))
    w, wv = up(dev, rng.standard_normal((taps, width)) * 0.5)
    state = up(dev, rng.standard_normal((4, max(taps - 1, 1), width)) * 50, dt)[0]
    one, fac = up(dev, [1.0])[0], up(dev, [mult])[0]
    mult = float(np.float32(mult))
    seen = {}
    for t in range(9):
        slots = [3, 0, 1] if t < 5 else [1, 3]
        start = {s: t if t < 5 or s == 3 else t - 5 for s in slots}
        b = Batch(dev, [(s, start[s], 1) for s in slots], 16)
        rows = len(slots)
        x, xv = up(dev, rng.standard_normal((rows, width)))
        y, yv = up(dev, rng.standard_normal((rows * n_y, width)))
        order = rng.permutation(rows * n_y).reshape(rows, n_y)
        wt, wtv = up(dev, rng.random((rows, n_y)))
        more, mv = up(dev, rng.standard_normal((rows, width)))
        gate, gtv = up(dev, rng.standard_normal((rows, 5)))
        inj, iv = up(dev, rng.standard_normal((rows, width)))
        out, total = up(dev, np.full((rows, ld), 7.0), dt)[0], dev.alloc(rows * width, F32)
        at_gate = C.c_void_p(gate.ptr + 8)
        KEEP.append(gate)
        inject = t % 2 == 0
        dev._check(dev._L.tq_stream_step(dev._ctx, ptr(x), ptr(x), ptr(y), ptr(ints(dev, order)), ptr(wt), n_y, ptr(more), at_gate, 5, ptr(inj if inject else None), ptr(one),
                                         ptr(fac), ptr(gain), rows, width, eps, ptr(w), ptr(state), taps, 16, ptr(b.pos_d), ptr(b.crow_d), ptr(out), dt, ld, ptr(total)))
        new = xv + mult * ((yv[order] * wtv[..., None]).sum(1) + mv * X.sigmoid(gtv[:, 2:3]))
        assert rel(down(total, F32, (rows, width)), new) < 1e-5
        if inject:
            new = new + iv
        assert rel(down(x, F32, (rows, width)), new) < 1e-5
        h = X.rms(new, eps) * gv
        got = down(out, dt, (rows, ld))
        assert (got[:, width:] == 7).all()
        for i, s in enumerate(slots):
            before = seen.get(s, np.zeros((taps - 1, width))) if start[s] else np.zeros((taps - 1, width))
            c, seen[s] = X.conv(h[i:i + 1], wv.T, before)
            assert rel(got[i, :width], h[i] + c[0]) < tol, (t, s)


@pytest.mark.parametrize("rows,experts,top,chunk", [(1, 3, 2, 8), (5, 12, 3, 4), (40, 40, 6, 16), (700, 64, 4, 32), (300, 2, 1, 8), (90, 300, 9, 16)])
def test_biased_routing(dev, rows, experts, top, chunk):
    """Softmax over the chosen logits; the logits' rows have something else behind them."""
    rng = np.random.default_rng(rows)
    pairs, ld = rows * top, experts + 3
    z = np.concatenate([rng.standard_normal((rows, experts)) * 2, np.full((rows, 3), 99.0)], 1).astype(np.float32)
    bias = (rng.standard_normal(experts) * 2).astype(np.float32)
    jobs_max = min(pairs, experts + pairs // chunk)
    e, slot, srow = (dev.upload(np.full(pairs, -7, np.int32), I32) for _ in range(3))
    w, jobs, nj = dev.alloc(pairs, F32), dev.upload(np.zeros(4 * jobs_max, np.int32), I32), dev.upload(np.zeros(1, np.int32), I32)
    dev._check(dev._L.tq_route_biased(dev._ctx, ptr(up(dev, z)[0]), ld, rows, experts, top, 1, 1, ptr(up(dev, bias)[0]), None, 0, chunk, ptr(e), ptr(w), ptr(slot), ptr(srow),
                                      ptr(jobs), ptr(nj)))
    ge, gw, gs, gr = e.to_vec().reshape(rows, top), w.to_vec().reshape(rows, top), slot.to_vec(), srow.to_vec()
    moved = 0
    for r in range(rows):
        full = (z[r, :experts] + bias).astype(np.float64)
        want_e, want_w = X.choose(full, top)
        assert ge[r].tolist() == want_e
        assert np.allclose(gw[r], want_w, rtol=3e-5)
        moved += want_e != X.choose(z[r, :experts].astype(np.float64), top)[0]
    assert moved
    assert np.array_equal(np.sort(gs), np.arange(pairs)) and np.array_equal(gr[gs], np.repeat(np.arange(rows), top))
    seen, owner = np.zeros(pairs, int), np.zeros(pairs, int)
    owner[gs] = ge.reshape(-1)
    for ex, first, count, shift in jobs.to_vec().reshape(-1, 4)[:int(nj.to_vec()[0])]:
        assert 0 < count <= chunk and shift == 0 and (owner[first:first + count] == ex).all()
        seen[first:first + count] += 1
    assert (seen == 1).all()
