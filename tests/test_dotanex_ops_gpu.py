"""The mechanisms of the Dotanex family one by one on the device, against the numpy implementation: residual streams, per-head
norms and rotations, sinks per head, absorbed latent attention, lightning attention, corrected routing with identity experts."""
import ctypes as C

import numpy as np
import pytest

import dotanex_oracle as X
from util import bf16_round

pytestmark = pytest.mark.gpu

F32, BF16, I32 = 0, 1, 5


class AttnConfig(C.Structure):
    _fields_ = [(n, C.c_uint32) for n in ("heads", "kv_heads", "dim", "vdim", "window")] + [(n, C.c_float) for n in ("scale", "softcap", "sink")]


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

    def __init__(self, dev, seqs, max_seq):
        self.seqs, self.max_seq = seqs, max_seq
        counts = [n for _, _, n in seqs]
        self.rows, self.max_q, self.max_len = sum(counts), max(counts), max(s + n for _, s, n in seqs)
        self.pos = np.concatenate([np.arange(s, s + n) for _, s, n in seqs])
        self.crow = np.concatenate([slot * max_seq + np.arange(s, s + n) for slot, s, n in seqs])
        self.first = np.cumsum([0] + counts)
        self.pos_d, self.crow_d = ints(dev, self.pos), ints(dev, self.crow)
        self.rows_d = ints(dev, self.first) if self.max_q > 1 else None


@pytest.mark.parametrize("dt,tol", [(F32, 3e-6), (BF16, 4e-3)])
@pytest.mark.parametrize("streams", [1, 2, 3, 4, 5, 16])
@pytest.mark.parametrize("rows,width", [(3, 72), (1, 1001), (700, 130), (5, 4100)])
def test_streams(dev, dt, tol, streams, rows, width):
    """All streams equal at first or not, a plain sublayer output, and the weighted rows of experts with the sublayer's input for
    identity experts (overwritten by the next input) and a shared row."""
    rng = np.random.default_rng(streams * 1000 + width)
    eps, ld = 1e-4, (width + 7) // 8 * 8
    mix, wo, wi, gain = (rng.standard_normal(s) for s in ((streams, streams), streams, streams, width))
    mix_d, wo_d, wi_d, gain_d = (up(dev, a)[0] for a in (mix, wo, wi, gain))
    mix, wo, wi, gain = (a.astype(np.float32).astype(np.float64) for a in (mix, wo, wi, gain))
    n_y = 3
    for equal in (False, True):
        for experts in (False, True):
            x, xv = up(dev, rng.standard_normal((rows, 1 if equal else streams, width)))
            xs = np.repeat(xv, streams, 1).transpose(1, 0, 2) if equal else xv.transpose(1, 0, 2)
            h, hv = up(dev, rng.standard_normal((rows, ld)), dt)
            if experts:
                y, yv = up(dev, rng.standard_normal((rows * n_y, width)))
                slots = rng.permutation(rows * n_y).reshape(rows, n_y)
                slots[rng.random((rows, n_y)) < 0.3] = -1
                wt, wtv = up(dev, rng.random((rows, n_y)))
                more, mv = up(dev, rng.standard_normal((rows, width)))
                parts = np.where(slots[..., None] < 0, hv[:, None, :width], yv[slots])
                ys = (parts * wtv[..., None]).sum(1) + mv
            else:
                (y, ys), slots, wt, more = up(dev, rng.standard_normal((rows, width))), None, None, None
            out = x if not equal else dev.alloc(rows * streams * width, F32)
            total = dev.alloc(rows * width, F32)
            dev._check(dev._L.tq_stream_mix(dev._ctx, streams, 1 if equal else streams, ptr(x), ptr(out), ptr(y), ptr(ints(dev, slots) if experts else None), ptr(wt),
                                            n_y, ptr(h if experts else None), ptr(more), ptr(mix_d), ptr(wo_d), ptr(wi_d), ptr(gain_d), rows, width, eps, ptr(h), dt,
                                            ld, ptr(total)))
            new = X.write_streams(xs, mix, wo, ys)
            assert rel(down(out, F32, (rows, streams, width)).transpose(1, 0, 2), new) < 1e-5
            assert rel(down(total, F32, (rows, width)), new.sum(0)) < 1e-5
            got = down(h, dt, (rows, ld))
            assert rel(got[:, :width], X.rms(X.read_streams(new, wi), eps) * gain) < max(tol, 1e-5)
            assert np.array_equal(got[:, width:], hv[:, width:])


@pytest.mark.parametrize("dt,tol", [(F32, 6e-5), (BF16, 8e-3)])      # (an f32 angle of 300 carries 1.5e-5)
@pytest.mark.parametrize("heads,kv_heads,dim,first,rot,interleaved,norm", [
    (4, 2, 32, 0, 16, False, True), (3, 1, 33, 0, 10, False, True), (20, 4, 128, 0, 128, False, True), (5, 0, 24, 16, 8, True, False), (7, 0, 13, 7, 6, True, False),
    (33, 0, 192, 128, 64, True, False), (2, 2, 8, 0, 0, False, True)])
def test_head_norm_and_rotation(dev, dt, tol, heads, kv_heads, dim, first, rot, interleaved, norm):
    rng = np.random.default_rng(dim)
    b = Batch(dev, [(1, 5, 9), (0, 300, 1), (2, 0, 40)], 320)
    eps, mult, ld = 1e-5, 1.25, (dim + 7) // 8 * 8
    f = X.plain_frequencies(rot, 500.0) if rot else np.zeros(0)
    # head by head: [head][row][ld]
    q, qv = up(dev, rng.standard_normal((heads, b.rows, ld)), dt)
    raw, rv = up(dev, pad(rng.standard_normal((960, max(kv_heads, 1), dim)), 8), dt)
    keys = dev.upload(np.zeros(960 * max(kv_heads, 1) * ld, np.float32 if dt == F32 else np.uint16), dt)
    qg, qgv = up(dev, rng.standard_normal(dim), dt)
    kg, kgv = up(dev, rng.standard_normal(dim), dt)
    fr, fv = up(dev, np.append(f, 0.0))
    dev._check(dev._L.tq_head_norm_rope(dev._ctx, dt, heads, kv_heads, dim, ptr(q), ld, b.rows * ld, ptr(raw if kv_heads else None), ptr(keys if kv_heads else None), 960,
                                        ptr(qg if norm else None), ptr(kg if norm else None), first, rot, int(interleaved), ptr(fr), mult, eps, ptr(b.pos_d),
                                        ptr(b.crow_d), b.rows))
    got, gk = down(q, dt, (heads, b.rows, ld)), down(keys, dt, (960, max(kv_heads, 1), ld))
    spin = X.rotate_neighbours if interleaved else X.rotate_halves

    def want(x, gain, pos):
        y = X.rms(x, eps) * gain if norm else x.copy()
        y[..., first:] = spin(y[..., first:], pos, fv[:rot // 2], mult)
        return y

    for r in range(b.rows):
        assert rel(got[:, r, :dim], want(qv[:, r, :dim], qgv, b.pos[r])) < tol
        if kv_heads:
            assert rel(gk[b.crow[r], :, :dim], want(rv[b.crow[r], :, :dim], kgv, b.pos[r])) < tol
    if kv_heads:
        other = np.setdiff1d(np.arange(960), b.crow)
        assert not gk[other].any()


@pytest.mark.parametrize("dt,tol", [(F32, 5e-6), (BF16, 8e-3)])
@pytest.mark.parametrize("heads,kv_heads,dim,window", [(4, 2, 32, 20), (6, 1, 40, 65), (20, 1, 16, 64), (3, 3, 136, 1), (8, 2, 128, 300), (2, 1, 264, 90)])
@pytest.mark.parametrize("seqs", [[(0, 0, 70), (1, 33, 5), (2, 200, 1)], [(0, 319, 1), (1, 0, 1), (2, 64, 1)]])
def test_sinks_per_head(dev, dt, tol, heads, kv_heads, dim, window, seqs):
    rng = np.random.default_rng(dim + window)
    b = Batch(dev, seqs, 320)
    sinks = rng.standard_normal(heads) * 3
    sinks[0], sinks[-1] = 12.0, -20.0
    sink_d, sinks = up(dev, sinks)
    q, qv = up(dev, rng.standard_normal((b.rows, heads, dim)) * 2, dt)
    k, kv = up(dev, pad(rng.standard_normal((960, kv_heads, dim)), 8), dt)
    v, vv = up(dev, pad(rng.standard_normal((960, kv_heads, dim)), 8), dt)
    cfg = AttnConfig(heads, kv_heads, dim, dim, window, dim ** -0.5, 0.0, 0.0)
    out = dev.alloc(b.rows * heads * dim, dt)
    dev._check(dev._L.tq_window_attention_sinks(dev._ctx, C.byref(cfg), ptr(sink_d), dt, ptr(q), heads * dim, None, 0, ptr(k), ptr(v), 960, ptr(b.rows_d),
                                                ptr(b.pos_d), ptr(b.crow_d), len(seqs), b.rows, b.max_q, b.max_len, ptr(out), heads * dim))
    got = down(out, dt, (b.rows, heads, dim))
    for i, (slot, start, n) in enumerate(seqs):
        rows = slice(slot * 320, slot * 320 + start + n)
        want = X.attention(qv[b.first[i]:b.first[i + 1]], kv[rows, :, :dim], vv[rows, :, :dim], start, dim ** -0.5, window, sinks)
        assert rel(got[b.first[i]:b.first[i + 1]], want) < tol


@pytest.mark.parametrize("heads,dim,rot,rank", [(3, 20, 8, 28), (16, 64, 32, 64), (17, 7, 6, 13), (40, 16, 16, 128), (8, 24, 64, 200), (20, 128, 64, 512)])
@pytest.mark.parametrize("starts", [[0], [319, 0, 64, 63, 128], [700]])
@pytest.mark.parametrize("rotate", [False, True])
def test_absorbed_latent_attention(dev, heads, dim, rot, rank, starts, rotate):
    rng = np.random.default_rng(rank + len(starts))
    n, max_seq = len(starts), 720
    b = Batch(dev, [(n - 1 - i, s, 1) for i, s in enumerate(starts)], max_seq)
    cp, rp, ldq, scale, mult = -(-rank // 16) * 16, -(-rot // 16) * 16, (dim + rot + 7) // 8 * 8, 0.7 * (dim + rot) ** -0.5, 1.3
    c = pad(rng.standard_normal((n * max_seq, rank)), 16)
    r = pad(rng.standard_normal((n * max_seq, rot)), 16)
    cache, cv = up(dev, np.concatenate([c, r], 1), BF16)
    ql, qlv = up(dev, pad(rng.standard_normal((heads, n, rank)) * 0.5, 16) + 7.0 * (np.arange(cp) >= rank), BF16)     # (padding of the queries may hold anything)
    q, qv = up(dev, rng.standard_normal((heads, n, ldq)) * 2, BF16)
    fr, f = up(dev, X.plain_frequencies(rot, 300.0))
    out = dev.upload(np.zeros(heads * n * cp, np.uint16), BF16)
    dev._check(dev._L.tq_latent_decode(dev._ctx, heads, dim, rot, rank, scale, rot, ptr(fr), mult, int(rotate), ptr(ql), ptr(q), ldq, ptr(cache), n * max_seq,
                                       ptr(b.pos_d), ptr(b.crow_d), n, b.max_len, ptr(out)))
    got = down(out, BF16, (heads, n, cp))
    for i, s in enumerate(starts):
        rows = cv[(n - 1 - i) * max_seq:][:s + 1]
        turned = qv[:, i, dim:dim + rot]
        if rotate:
            turned = bf16_round(X.rotate_neighbours(turned, s, f, mult).astype(np.float32))[1].astype(np.float64)
        full = np.concatenate([qlv[:, i, :rank], turned], 1)[None]
        keys = np.concatenate([rows[:, :rank], rows[:, cp:cp + rot]], 1)[:, None]
        assert rel(got[:, i, :rank], X.attention(full, keys, rows[:, None, :rank], s, scale)[0]) < 2e-2


@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("heads,dim,vdim", [(3, 20, 24), (2, 64, 128), (1, 7, 9), (4, 16, 16), (2, 256, 256), (3, 32, 48), (5, 160, 64)])
@pytest.mark.parametrize("seqs", [[(1, 0, 200), (0, 37, 64), (2, 5, 1)], [(2, 0, 1), (0, 9, 1)], [(1, 3, 7), (0, 0, 2)], [(0, 64, 129)]])
def test_lightning(dev, dt, heads, dim, vdim, seqs):
    rng = np.random.default_rng(dim + vdim + len(seqs))
    b = Batch(dev, seqs, 400)
    eps = 1e-5
    decay_d, decay = up(dev, np.array([1.0, 0.6, 0.0, 0.97, 0.999])[:heads])
    kc, vc, gc = (heads * dim + 7) // 8 * 8, 0, 0
    vc = 2 * kc
    gc = vc + (heads * vdim + 7) // 8 * 8
    ld = gc + (heads * vdim + 7) // 8 * 8
    buf, bv = up(dev, rng.standard_normal((b.rows, ld)), dt)
    es = 4 if dt == F32 else 2
    state0 = rng.standard_normal((3, heads, dim, vdim)) * 3
    st, sv = up(dev, state0)
    nw, nv = up(dev, rng.standard_normal(heads * vdim))
    out = dev.alloc(b.rows * heads * vdim, dt)
    at = lambda c: C.c_void_p(buf.ptr + c * es)
    KEEP.append(buf)
    dev._check(dev._L.tq_lightning(dev._ctx, dt, heads, dim, vdim, eps, ptr(decay_d), at(0), at(kc), at(vc), at(gc), ld, ptr(nw), ptr(st), 400, 1200, ptr(b.rows_d),
                                   ptr(b.pos_d), ptr(b.crow_d), len(seqs), b.rows, b.max_q, ptr(out), heads * vdim))
    got, gs = down(out, dt, (b.rows, heads * vdim)), down(st, F32, state0.shape)
    want_s = sv.copy()
    for i, (slot, start, n) in enumerate(seqs):
        rows = bv[b.first[i]:b.first[i + 1]]
        q, k, v = rows[:, :heads * dim].reshape(n, heads, dim), rows[:, kc:kc + heads * dim].reshape(n, heads, dim), rows[:, vc:vc + heads * vdim].reshape(n, heads, vdim)
        o = np.zeros((n, heads, vdim))
        for h in range(heads):
            o[:, h], want_s[slot, h] = X.lightning(q[:, h], k[:, h], v[:, h], decay[h], np.zeros((dim, vdim)) if start == 0 else sv[slot, h])
        want = X.rms(o.reshape(n, heads * vdim), eps) * nv * X.sigmoid(rows[:, gc:gc + heads * vdim])
        assert rel(got[b.first[i]:b.first[i + 1]], want) < (1e-5 if dt == F32 else 6e-3)
    assert rel(gs, want_s) < (1e-5 if dt == F32 else 1e-4)


@pytest.mark.parametrize("rows,experts,identity,top,chunk", [(1, 3, 2, 2, 8), (5, 12, 0, 3, 4), (40, 20, 20, 6, 16), (700, 60, 8, 4, 32), (300, 1, 3, 2, 8), (90, 300, 30, 9, 16)])
def test_corrected_routing_with_identity_experts(dev, rows, experts, identity, top, chunk):
    rng = np.random.default_rng(rows)
    n, pairs = experts + identity, rows * top
    z = rng.standard_normal((rows, n)).astype(np.float32) * 2
    corr = (rng.standard_normal(n) * 0.2).astype(np.float32)
    jobs_max = min(pairs, experts + pairs // chunk)
    e, slot, srow = (dev.upload(np.full(pairs, -7, np.int32), I32) for _ in range(3))
    w, jobs, nj = dev.alloc(pairs, F32), dev.upload(np.zeros(4 * jobs_max, np.int32), I32), dev.upload(np.zeros(1, np.int32), I32)
    dev._check(dev._L.tq_route_rule(dev._ctx, ptr(up(dev, z)[0]), rows, n, top, 1, 1, ptr(up(dev, corr)[0]), identity, chunk, ptr(e), ptr(w), ptr(slot), ptr(srow),
                                    ptr(jobs), ptr(nj)))
    ge, gw, gs, gr = e.to_vec().reshape(rows, top), w.to_vec().reshape(rows, top), slot.to_vec().reshape(rows, top), srow.to_vec()
    moved = 0
    for r in range(rows):
        want_e, want_w = X.choose(z[r].astype(np.float64), corr.astype(np.float64), top)
        assert ge[r].tolist() == want_e
        assert np.allclose(gw[r], want_w, rtol=3e-5)
        moved += want_e != X.choose(z[r].astype(np.float64), 0 * corr, top)[0]
    assert rows < 5 or moved
    real = ge < experts
    assert (gs[~real] == -1).all() and np.array_equal(np.sort(gs[real]), np.arange(real.sum()))
    row_of = np.repeat(np.arange(rows)[:, None], top, 1)
    assert np.array_equal(gr[gs[real]], row_of[real])
    seen = np.zeros(pairs, int)
    owner = np.full(pairs, -1)
    owner[gs[real]] = ge[real]
    for ex, first, count, shift in jobs.to_vec().reshape(-1, 4)[:int(nj.to_vec()[0])]:
        assert 0 < count <= chunk and shift == 0 and (owner[first:first + count] == ex).all()
        seen[first:first + count] += 1
    assert (seen[:real.sum()] == 1).all() and not seen[real.sum():].any()
