"""The mechanisms of the Numuzen family one by one on the device, against the numpy implementation: norm and rotation of
queries and keys, windowed attention with capped scores, sink and gate, gated linear attention, post-norm, routing, grouped
linear layers."""
import ctypes as C

import numpy as np
import pytest

import numuzen_oracle as N
from util import bf16_round

pytestmark = pytest.mark.gpu

F32, BF16, I32 = 0, 1, 5


class AttnConfig(C.Structure):
    _fields_ = [(n, C.c_uint32) for n in ("heads", "kv_heads", "dim", "vdim", "window")] + [(n, C.c_float) for n in ("scale", "softcap", "sink")]


class GlaConfig(C.Structure):
    _fields_ = [(n, C.c_uint32) for n in ("heads", "dim", "vdim", "rank")] + [(n, C.c_float) for n in ("tau", "q_scale", "eps")]


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


def up(dev, x, dt):
    """Upload of an array in the given format; returns (buffer, the values it holds)."""
    x = np.ascontiguousarray(x, np.float32)
    if dt == F32:
        return dev.upload(x.reshape(-1), F32), x.astype(np.float64)
    bits, val = bf16_round(x)
    return dev.upload(bits.reshape(-1), BF16), val.reshape(x.shape).astype(np.float64)


def down(buf, dt, shape):
    a = buf.to_vec()
    if dt == BF16:
        a = np.asarray(a)
        a = (a.astype(np.uint32) << 16).view(np.float32) if a.dtype == np.uint16 else a
    return np.asarray(a, np.float64).reshape(shape)


def ints(dev, x):
    return dev.upload(np.asarray(x, np.int32).reshape(-1), I32)


def rel(got, want):
    """Largest error, relative to the element and the root mean square (an output in bf16 carries 0.002 of its element)."""
    return (np.abs(got - want) / (np.abs(want) + np.sqrt(np.mean(np.square(want))) + 1e-30)).max()


def pad8(n):
    return (n + 7) // 8 * 8


def packed(x):
    """[rows, heads, dim] -> [rows, heads, dim rounded up to 8] with zeros."""
    return np.pad(x, ((0, 0), (0, 0), (0, pad8(x.shape[2]) - x.shape[2])))


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


ATTN = [  # heads, kv_heads, dim, vdim, window, softcap, sink, gate
    (4, 2, 32, 32, 20, 15.0, 0.0, True),
    (6, 1, 40, 40, 65, 8.0, 0.0, True),
    (3, 3, 72, 72, 1, 30.0, 0.0, True),
    (20, 1, 16, 16, 64, 5.0, 0.0, False),
    (5, 1, 33, 51, 7, 0.0, 1.5, True),
    (8, 2, 128, 128, 300, 25.0, 0.0, True),
    (2, 1, 200, 256, 90, 0.0, None, False),
    (2, 2, 264, 40, 33, 12.0, -2.0, True),
    (4, 4, 24, 100, 1 << 30, 9.0, 0.0, True),
]


@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("case", ATTN, ids=[str(c[:5]) for c in ATTN])
@pytest.mark.parametrize("kind", ["prompts", "decode"])
def test_window_attention(dev, case, dt, kind):
    H, G, D, V, window, softcap, sink, gated = case
    rng = np.random.default_rng(H * 1000 + D)
    max_seq, slots = 400, 4
    seqs = [(2, 0, 130), (0, 37, 60), (3, 300, 2), (1, 63, 1)] if kind == "prompts" else [(2, 0, 1), (0, 370, 1), (3, 127, 1), (1, 64, 1)]
    b = Batch(dev, seqs, max_seq)
    q, qv = up(dev, rng.standard_normal((b.rows, H, D)) * 1.5, dt)
    g, gv = up(dev, rng.standard_normal((b.rows, H, V)), dt)
    k, kv = up(dev, packed(rng.standard_normal((slots * max_seq, G, D))), dt)
    v, vv = up(dev, packed(rng.standard_normal((slots * max_seq, G, V))), dt)
    out = dev.alloc(b.rows * H * V, dt)
    scale = D ** -0.5 * 2
    a = AttnConfig(H, G, D, V, window, scale, softcap, -np.inf if sink is None else sink)
    dev._check(dev._L.tq_window_attention(dev._ctx, C.byref(a), dt, ptr(q), H * D, ptr(g) if gated else None, H * V, ptr(k), ptr(v), slots * max_seq, ptr(b.rows_d),
                                          ptr(b.pos_d), ptr(b.crow_d), len(seqs), b.rows, b.max_q, b.max_len, ptr(out), H * V))
    got = down(out, dt, (b.rows, H, V))
    for i, (slot, start, n) in enumerate(seqs):
        rows = slice(b.first[i], b.first[i + 1])
        at = slice(slot * max_seq, slot * max_seq + start + n)
        want = N.attention(qv[rows], kv[at, :, :D], vv[at, :, :V], start, scale, softcap, window, sink)
        if gated:
            want = want * N.sigmoid(gv[rows])
        assert rel(got[rows], want) < (3e-5 if dt == F32 else 6e-3), (i, rel(got[rows], want))


@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("heads,kv_heads,window", [(4, 1, 1000), (24, 1, 700), (2, 2, 5000), (8, 1, 129)])
def test_one_loud_key_among_many(dev, dt, heads, kv_heads, window):
    """A single key that the query matches, just inside and just outside the window and at tile borders, among hundreds."""
    D, n = 32, 1500
    rng = np.random.default_rng(5)
    pos = n - 1
    for j in sorted({max(0, pos - window + 1), max(0, pos - window), 0, 64, 63, 1023, 1024, pos - 1, pos}):
        kx, vx = rng.standard_normal((n, kv_heads, D)) * 0.1, rng.standard_normal((n, kv_heads, D))
        q0 = rng.standard_normal((1, heads, D))
        for h in range(heads):
            kx[j, h // (heads // kv_heads)] += q0[0, h] * 0.7
        k, kv = up(dev, kx, dt)
        v, vv = up(dev, vx, dt)
        for rows in (1, 3):                               # decoded alone, and as the last of a portion
            b = Batch(dev, [(0, n - rows, rows)], n)
            q, qv = up(dev, np.repeat(q0, rows, 0), dt)
            out = dev.alloc(rows * heads * D, dt)
            a = AttnConfig(heads, kv_heads, D, D, window, 0.5, 40.0, 0.0)
            dev._check(dev._L.tq_window_attention(dev._ctx, C.byref(a), dt, ptr(q), heads * D, None, 0, ptr(k), ptr(v), n, ptr(b.rows_d), ptr(b.pos_d),
                                                  ptr(b.crow_d), 1, rows, rows, n, ptr(out), heads * D))
            want = N.attention(qv, kv, vv, n - rows, 0.5, 40.0, window)
            got = down(out, dt, want.shape)
            assert rel(got[-1], want[-1]) < (3e-5 if dt == F32 else 6e-3), (j, rows)


@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("H,G,D,rot", [(4, 2, 32, 16), (3, 1, 33, 10), (5, 5, 24, 24), (8, 2, 128, 2), (2, 1, 40, 0)])
def test_query_key_norm_and_rotation(dev, dt, H, G, D, rot):
    rng = np.random.default_rng(D)
    max_seq = 3000
    b = Batch(dev, [(1, 2900, 5), (0, 0, 3)], max_seq)
    scaling = {"factor": 4.0, "original": 128, "fast": 8.0, "slow": 1.0}
    r = {"dims": rot, "base": 5000.0, "scaling": scaling}
    f, mult = (N.frequencies(r) if rot else (np.zeros(1), 1.0))
    q, qv = up(dev, rng.standard_normal((b.rows, H, D)), dt)
    raw_all = np.zeros((2 * max_seq, G, pad8(D)))
    raw_all[b.crow] = packed(rng.standard_normal((b.rows, G, D)))
    raw, rv = up(dev, raw_all, dt)
    keys = dev.alloc(2 * max_seq * G * pad8(D), dt)
    dev.memset(keys)
    qg, qgv = up(dev, 1 + 0.3 * rng.standard_normal(H * D), dt)
    kg, kgv = up(dev, 1 + 0.3 * rng.standard_normal(G * D), dt)
    fr = dev.upload(f.astype(np.float32), F32)
    eps = 1e-3
    dev._check(dev._L.tq_qk_norm_rope(dev._ctx, dt, H, G, D, ptr(q), H * D, ptr(raw), ptr(keys), 2 * max_seq, ptr(qg), ptr(kg), rot, ptr(fr), mult, eps,
                                      ptr(b.pos_d), ptr(b.crow_d), b.rows))
    got_q, got_k = down(q, dt, (b.rows, H, D)), down(keys, dt, (2 * max_seq, G, pad8(D)))
    turn = lambda x, p: N.rotate(x, p, r) if rot else x
    want_q = np.array([turn((N.rms(qv[i].reshape(-1), eps) * qgv).reshape(H, D), p) for i, p in enumerate(b.pos)])
    want_k = np.array([turn((N.rms(rv[c, :, :D].reshape(-1), eps) * kgv).reshape(G, D), p) for c, p in zip(b.crow, b.pos)])
    tol = 5e-4 if dt == F32 else 6e-3                     # (an angle of 2900 radians carries 1e-4 of f32 rounding)
    assert rel(got_q, want_q) < tol and rel(got_k[b.crow, :, :D], want_k) < tol
    assert not got_k[:, :, D:].any() and not np.delete(got_k, b.crow, 0).any()


@pytest.mark.parametrize("width,n_y,dt", [(64, 1, F32), (72, 3, BF16), (101, 2, BF16), (101, 2, F32), (2500, 2, F32), (4096, 4, BF16), (8000, 1, BF16)])
def test_add_norm(dev, width, n_y, dt):
    rng = np.random.default_rng(width)
    rows, n, eps = 7, 40, 1e-4
    x, y = rng.standard_normal((rows, width)), rng.standard_normal((n, width)) * 0.1
    slot = rng.permutation(n)[:rows * n_y].reshape(rows, n_y)
    slot[2, 0] = -1
    gp, gn = rng.standard_normal(width), rng.standard_normal(width)
    (xd, xv), (yd, yv), (gpd, gpv), (gnd, gnv) = (up(dev, a, F32) for a in (x, y, gp, gn))
    out = dev.alloc(rows * width, dt)
    ld = width
    dev._check(dev._L.tq_add_norm(dev._ctx, ptr(xd), ptr(yd), ptr(ints(dev, slot)), n_y, ptr(gpd), ptr(gnd), rows, width, eps, ptr(out), dt, ld))
    s = np.array([sum(yv[j] for j in r if j >= 0) if (r >= 0).any() else np.zeros(width) for r in slot])
    want_x = xv + N.rms(s, eps) * gpv
    assert rel(down(xd, F32, x.shape), want_x) < 1e-5
    assert rel(down(out, dt, x.shape), N.rms(want_x, eps) * gnv) < (1e-5 if dt == F32 else 6e-3)


GLA = [(2, 20, 24, 5, 8.0), (3, 64, 64, 16, 16.0), (1, 7, 9, 3, 1.0), (2, 128, 256, 16, 4.0), (2, 32, 96, 8, 0.5), (1, 160, 264, 24, 16.0), (4, 48, 80, 4, 2.0)]


@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("H,D,V,rank,tau", GLA)
def test_gated_linear_attention(dev, dt, H, D, V, rank, tau):
    """Two prompts, then portions of one to ninety rows and decoding, in slots whose states held something else before; strong
    and weak decays side by side."""
    rng = np.random.default_rng(D + V)
    max_seq, slots, eps = 300, 3, 1e-5
    L = {2: 200, 0: 150}
    total = {s: {"q": rng.standard_normal((n, H, D)), "k": rng.standard_normal((n, H, D)), "v": rng.standard_normal((n, H, V)), "g": rng.standard_normal((n, H, V)),
                 "a1": rng.standard_normal((n, rank))} for s, n in L.items()}
    a2, bias, norm = rng.standard_normal((H * D, rank)), rng.uniform(-9, 9, H * D), 1 + 0.2 * rng.standard_normal(V)
    ld = 2 * H * D + 2 * H * V + 8
    ld += -ld % 8
    row = {s: np.zeros((n, ld)) for s, n in L.items()}
    for s, x in total.items():
        n = L[s]
        row[s][:, :2 * H * D + 2 * H * V] = np.concatenate([x[k].reshape(n, -1) for k in ("q", "k", "v", "g")], 1)
        row[s] = up(dev, row[s], dt)[1]
    want = {}
    for s, n in L.items():
        r = row[s]
        q, k = r[:, :H * D].reshape(n, H, D) * 0.3, r[:, H * D:2 * H * D].reshape(n, H, D)
        v, g = r[:, 2 * H * D:2 * H * D + H * V].reshape(n, H, V), r[:, 2 * H * D + H * V:2 * H * D + 2 * H * V].reshape(n, H, V)
        z = total[s]["a1"].astype(np.float32).astype(np.float64) @ a2.astype(np.float32).T.astype(np.float64) + bias
        al = N.decay(z, tau).reshape(n, H, D)
        o = np.stack([N.gla(q[:, h], k[:, h], v[:, h], al[:, h], np.zeros((D, V)))[0] for h in range(H)], 1)
        want[s] = (N.rms(o, eps) * norm) * g * N.sigmoid(g)
    (a2d, _), (bd, _), (nd, _) = up(dev, a2, F32), up(dev, bias, F32), up(dev, norm, F32)
    cfg = GlaConfig(H, D, V, rank, tau, 0.3, eps)
    es = 4 if dt == F32 else 2

    def run(state, plan):
        """plan: list of steps, a step = {slot: rows}"""
        at = {s: 0 for s in L}
        got = {s: [] for s in L}
        for step in plan:
            seqs = [(s, at[s], n) for s, n in step.items()]
            b = Batch(dev, seqs, max_seq)
            x = up(dev, np.concatenate([row[s][a:a + n] for s, a, n in seqs]), dt)[0]
            a1 = up(dev, np.concatenate([total[s]["a1"][a:a + n] for s, a, n in seqs]), F32)[0]
            out = dev.alloc(b.rows * H * V, dt)
            off = lambda n: C.c_void_p(x.ptr + n * es)
            dev._check(dev._L.tq_gla(dev._ctx, C.byref(cfg), dt, off(0), off(H * D), off(2 * H * D), off(2 * H * D + H * V), ld, ptr(a1), rank, ptr(a2d), ptr(bd), ptr(nd),
                                     ptr(state), max_seq, slots * max_seq, ptr(b.rows_d), ptr(b.pos_d), ptr(b.crow_d), len(seqs), b.rows, b.max_q, ptr(out), H * V))
            o = down(out, dt, (b.rows, H, V))
            for i, (s, a, n) in enumerate(seqs):
                got[s].append(o[b.first[i]:b.first[i + 1]])
                at[s] += n
        return {s: np.concatenate(g) for s, g in got.items()}

    state = up(dev, rng.standard_normal((slots, H, D, V)) * 100, F32)[0]      # leftovers
    plans = [[{2: 200, 0: 150}], [{0: 1, 2: 64}, {2: 65, 0: 63}, {2: 1, 0: 1}, {0: 85, 2: 70}],
             [{2: 90, 0: 2}, {0: 2}, {0: 140, 2: 40}] + [{0: 1, 2: 1}] * 6 + [{2: 1}] * 4 + [{2: 60}],
             [{0: 10, 2: 16}, {0: 17, 2: 2}, {0: 33, 2: 31}, {0: 90, 2: 151}]]
    for i, plan in enumerate(plans):
        got = run(state, plan)
        for s in L:
            size = lambda x: np.sqrt(np.mean(x * x, axis=(1, 2)))
            err = size(got[s] - want[s]) / (size(want[s]) + np.sqrt(np.mean(want[s] ** 2)))
            assert err.max() < (1e-5 if dt == F32 else 6e-3), (i, s, int(err.argmax()), err.max())


@pytest.mark.parametrize("rows,experts,top,chunk", [(1, 1, 1, 8), (3, 5, 5, 2), (40, 12, 3, 8), (700, 33, 4, 64), (1500, 300, 2, 16), (5000, 7, 1, 256)])
@pytest.mark.parametrize("score,renorm", [(0, 0), (1, 1)])
def test_routing(dev, rows, experts, top, chunk, score, renorm):
    rng = np.random.default_rng(rows)
    z = rng.standard_normal((rows, experts)).astype(np.float32) * 3
    z[0] = 1.5                                            # equal scores: the lower indices
    pairs = rows * top
    mj = min(pairs, experts + pairs // chunk)
    e, w, slot, srow, jobs, nj = (dev.alloc(n, t) for n, t in ((pairs, I32), (pairs, F32), (pairs, I32), (pairs, I32), (4 * mj, I32), (1, I32)))
    for _ in range(2):                                    # (the counters are clean again after a launch)
        dev._check(dev._L.tq_route(dev._ctx, ptr(dev.upload(z.reshape(-1), F32)), rows, experts, top, score, renorm, chunk, ptr(e), ptr(w), ptr(slot), ptr(srow),
                                   ptr(jobs), ptr(nj)))
        ge, gw, gs, gr = e.to_vec().reshape(rows, top), w.to_vec().reshape(rows, top), slot.to_vec(), srow.to_vec()
        p = N.sigmoid(z) if score == 0 else np.exp(z - z.max(1, keepdims=True)) / np.exp(z - z.max(1, keepdims=True)).sum(1, keepdims=True)
        order = np.argsort(-z, axis=1, kind="stable")[:, :top]
        assert np.array_equal(ge, order)
        want = np.take_along_axis(p, order, 1)
        assert np.allclose(gw, want / want.sum(1, keepdims=True) if renorm else want, rtol=2e-5)
        assert np.array_equal(np.sort(gs), np.arange(pairs)) and np.array_equal(gr[gs], np.arange(pairs) // top)
        g = jobs.to_vec().reshape(-1, 4)[:int(nj.to_vec()[0])]
        owner = np.empty(pairs, np.int64)
        owner[gs] = ge.reshape(-1)
        seen = np.zeros(pairs, int)
        for ex, first, n, _ in g:
            assert 0 < n <= chunk and (owner[first:first + n] == ex).all()
            seen[first:first + n] += 1
        assert (seen == 1).all()


@pytest.mark.parametrize("dt,chunk", [(BF16, 3), (BF16, 8), (BF16, 16), (BF16, 48), (BF16, 256), (F32, 64)])
@pytest.mark.parametrize("cols,feat", [(72, 24), (96, 96), (130, 200), (1024, 40)])
@pytest.mark.parametrize("glu", [False, True])
def test_grouped_linear(dev, dt, chunk, cols, feat, glu):
    """Experts with no rows, few and many; row numbers, row factors, gate / up halves."""
    rng = np.random.default_rng(cols + feat)
    L, E = dev._L, 5
    counts = [0, 1, 37, 2, 300]
    group = 2 * pad8(feat) if glu else (feat + 15) // 16 * 16
    h = C.c_void_p()
    dev._check(L.tq_dweight_create(dev._ctx, E * group, cols, dt, C.byref(h)))
    ws = []
    for e in range(E):
        parts = [rng.standard_normal((feat, cols)) * cols ** -0.5 * 2 for _ in range(2 if glu else 1)]
        vals = [bf16_round(p.astype(np.float32))[1].astype(np.float32) for p in parts]
        ws.append([v.astype(np.float64) for v in vals])
        for i, v in enumerate(vals):
            v = np.ascontiguousarray(v)
            dev._check(L.tq_dweight_put(dev._ctx, h, C.c_void_p(v.ctypes.data), F32, feat, cols, e * group, 0, i + 1 if glu else 0))
    rows = sum(counts)
    jobs, first = [], 0
    for e, n in enumerate(counts):
        jobs += [(e, first + i, min(chunk, n - i), 0) for i in range(0, n, chunk)]
        first += n
    jobs = [jobs[i] for i in rng.permutation(len(jobs))]
    listed = dt == F32 or chunk <= 8
    src = rng.integers(0, 50, rows) if listed else np.arange(rows)
    ldx = (cols + 7) // 8 * 8 + 8
    x, xv = up(dev, rng.standard_normal((50 if listed else rows, ldx)), dt)
    scale = rng.uniform(0.2, 1.5, rows).astype(np.float32)
    width = group // 2 if glu else group
    ldy = width + 4
    y = dev.alloc(rows * ldy, F32)
    jd, nd = ints(dev, jobs), ints(dev, [len(jobs)])
    dev._check(L.tq_dlinear_grouped(dev._ctx, h, ptr(x), ldx, rows, ptr(jd), ptr(nd), len(jobs) + 3, chunk, group,
                                    ptr(ints(dev, src)) if listed else None, ptr(dev.upload(scale, F32)), 1.1, 1.702 if glu else 0.0, ptr(y), F32, ldy))
    got = down(y, F32, (rows, ldy))[:, :feat]
    owner = np.repeat(np.arange(E), counts)
    for r in range(rows):
        p = [m @ xv[src[r], :cols] * scale[r] for m in ws[owner[r]]]
        want = N.clamped_glu(p[0], p[1], 1.1) if glu else p[0]
        assert np.abs(got[r] - want).max() < 3e-5 * (1 + np.abs(want).max()), r
    L.tq_dweight_free(dev._ctx, h)


def test_bad_arguments_are_refused(dev):
    import tang_b200 as tb

    L, x = dev._L, dev.alloc(4096, F32)
    one = ints(dev, [0])
    with pytest.raises(tb.TangqError, match="multiple of kv_heads"):
        dev._check(L.tq_window_attention(dev._ctx, C.byref(AttnConfig(3, 2, 8, 8, 4, 1.0, 1.0, 0.0)), F32, ptr(x), 24, None, 0, ptr(x), ptr(x), 4, None, ptr(one),
                                         ptr(one), 1, 1, 1, 1, ptr(x), 24))
    with pytest.raises(tb.TangqError, match="rotated dimensions"):
        dev._check(L.tq_qk_norm_rope(dev._ctx, F32, 1, 1, 8, ptr(x), 8, ptr(x), ptr(x), 4, ptr(x), ptr(x), 3, ptr(x), 1.0, 1e-5, ptr(one), ptr(one), 1))
    with pytest.raises(tb.TangqError, match="experts"):
        dev._check(L.tq_route(dev._ctx, ptr(x), 1, 4, 5, 0, 0, 8, ptr(x), ptr(x), ptr(x), ptr(x), ptr(x), ptr(x)))
    with pytest.raises(tb.TangqError, match="bad sizes"):
        dev._check(L.tq_gla(dev._ctx, C.byref(GlaConfig(1, 8, 8, 0, 1.0, 1.0, 1e-5)), F32, ptr(x), ptr(x), ptr(x), ptr(x), 8, ptr(x), 1, ptr(x), ptr(x), ptr(x), ptr(x), 4, 4,
                            None, ptr(one), ptr(one), 1, 1, 1, ptr(x), 8))
