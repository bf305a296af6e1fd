"""Differential attention (windowed, first tokens kept) against the plain numpy implementation, on its own caches."""
import ctypes as C

import numpy as np
import pytest

import tofazen_oracle as T
from util import bf16_round

pytestmark = pytest.mark.gpu

EPS = 1e-5


@pytest.fixture(scope="module")
def dev():
    import tang_b200

    d = tang_b200.QuantComputeDevice(0)
    yield d
    d.close()


class _Cfg(C.Structure):
    _fields_ = [(n, C.c_uint32) for n in ("heads", "kv_heads", "dim", "vdim", "window", "keep_first")] + [
        (n, C.c_float) for n in ("scale", "lam", "out_scale", "eps")]


class Case:
    """Sequences with keys and values at every position of their slot; queries for the last n_q positions of each."""

    def __init__(self, rng, H, G, D, V, window, keep, seqs, max_seq=320, lam=0.6, diff=0.35, scale=None, spread=1.0):
        self.H, self.G, self.D, self.V, self.window, self.keep, self.max_seq = H, G, D, V, window, keep, max_seq
        self.lam, self.diff, self.scale = lam, diff, D ** -0.5 if scale is None else scale
        self.seqs = seqs                                       # (start, n_q)
        self.slots = list(rng.permutation(len(seqs) + 2)[:len(seqs)])
        r = lambda *s: bf16_round((rng.standard_normal(s) * spread).astype(np.float32))[1]
        self.k = [r(s + n, G, 2, D) for s, n in seqs]
        self.v = [r(s + n, G, V) for s, n in seqs]
        self.q = [r(n, H, 2, D) for _, n in seqs]

    def want(self, b, rows=None):
        start, n = self.seqs[b]
        rows = range(n) if rows is None else rows
        return np.concatenate([T.diff_attention(self.q[b][i:i + 1].astype(np.float64), self.k[b][:start + i + 1].astype(np.float64),
                                                self.v[b][:start + i + 1].astype(np.float64), start + i, self.scale, self.window, self.keep,
                                                self.lam, self.diff, EPS) for i in rows])

    def run(self, dev, dtype, poison=True):
        """All sequences in one call.  Cache rows that no query may see hold NaN (behind the last position, other slots)."""
        import tang_b200 as tb

        up8 = lambda n: (n + 7) // 8 * 8
        dp, vp, n_slots = up8(self.D), up8(self.V), len(self.seqs) + 2
        kc = np.full((n_slots, self.max_seq, self.G, 2, dp), np.nan if poison else 0, np.float32)
        vc = np.full((n_slots, self.max_seq, self.G, vp), np.nan if poison else 0, np.float32)
        counts = [n for _, n in self.seqs]
        row_pos, cache_row = [], []
        for b, (start, n) in enumerate(self.seqs):
            s = self.slots[b]
            kc[s, :start + n], vc[s, :start + n] = 0, 0
            kc[s, :start + n, :, :, :self.D], vc[s, :start + n, :, :self.V] = self.k[b], self.v[b]
            row_pos += range(start, start + n)
            cache_row += range(s * self.max_seq + start, s * self.max_seq + start + n)
        q = np.concatenate([x.reshape(x.shape[0], -1) for x in self.q])
        up = (lambda a: dev.upload(bf16_round(np.ascontiguousarray(a))[0], tb.BF16)) if dtype == tb.BF16 else dev.upload
        qb, kb, vb = up(q), up(kc), up(vc)
        i32 = lambda a: dev.upload(np.asarray(a, np.int32), tb.I32)
        cu, rp, cr = i32(np.cumsum([0] + counts)), i32(row_pos), i32(cache_row)
        R, ldo = len(row_pos), self.H * self.V + 3
        out = dev.alloc(R * ldo, dtype)
        dev.memset(out)
        cfg = _Cfg(self.H, self.G, self.D, self.V, self.window, self.keep, self.scale, self.lam, 1 - self.diff, EPS)
        one = max(counts) == 1
        dev._check(dev._L.tq_diff_attention(dev._ctx, C.byref(cfg), dtype, C.c_void_p(qb.ptr), q.shape[1], C.c_void_p(kb.ptr), C.c_void_p(vb.ptr),
                                            n_slots * self.max_seq, C.c_void_p(0 if one else cu.ptr), C.c_void_p(rp.ptr), C.c_void_p(cr.ptr),
                                            len(counts), R, max(counts), max(s + n for s, n in self.seqs), C.c_void_p(out.ptr), ldo))
        dev.sync()
        o = out.to_vec()
        o = (o if dtype == tb.F32 else (o.astype(np.uint32) << 16).view(np.float32)).reshape(R, ldo)
        assert np.all(o[:, self.H * self.V:] == 0)
        return np.split(o[:, :self.H * self.V].reshape(R, self.H, self.V), np.cumsum(counts)[:-1])


def check(dev, case, rows=None):
    import tang_b200 as tb

    for dtype, tol in ((tb.F32, 2e-5), (tb.BF16, 6e-3)):
        got = case.run(dev, dtype)
        for b in range(len(case.seqs)):
            want = case.want(b, rows)
            g = got[b] if rows is None else got[b][list(rows)]
            err = np.abs(g - want).max() / np.sqrt(np.mean(want ** 2))
            # bf16: the result's own rounding (2^-9 of values up to a few rms) plus 2^-17 of the weights
            assert err < tol * (1 if dtype == tb.F32 else max(1.0, np.abs(want).max() / np.sqrt(np.mean(want ** 2)))), (dtype, b, err)


# heads, kv heads, dim, vdim, window, keep_first
SHAPES = [(4, 2, 16, 32, 20, 3), (6, 2, 40, 24, 64, 0), (3, 3, 7, 9, 5, 2), (8, 1, 33, 50, 65, 66), (12, 1, 24, 104, 1, 1), (2, 1, 64, 128, 1000, 0),
          (2, 2, 120, 184, 31, 130), (1, 1, 200, 256, 100, 4), (20, 1, 16, 16, 63, 5), (2, 1, 260, 48, 40, 3)]


@pytest.mark.parametrize("shape", SHAPES)
def test_prompts(dev, shape):
    rng = np.random.default_rng(sum(shape))
    check(dev, Case(rng, *shape, seqs=[(0, 70), (0, 1), (0, 33)]))


@pytest.mark.parametrize("shape", SHAPES)
def test_one_query_per_sequence(dev, shape):
    rng = np.random.default_rng(sum(shape) + 1)
    check(dev, Case(rng, *shape, seqs=[(0, 1), (63, 1), (64, 1), (129, 1), (300, 1), (5, 1)]))


@pytest.mark.parametrize("shape", SHAPES[:7])
def test_portions_behind_a_cached_prefix(dev, shape):
    rng = np.random.default_rng(sum(shape) + 2)
    check(dev, Case(rng, *shape, seqs=[(100, 2), (63, 2), (0, 2), (127, 18), (200, 1), (31, 65)]))


def _stand_out(case, b, i, j, score, head=0, mp=0):
    """Makes the score of query i (index in the chunk) with key position j about `score` in one map of one head, all other
    keys' scores small, and the value of key j large: whether key j is seen decides the result."""
    g = head // (case.H // case.G)
    q = case.q[b][i, head, mp]
    case.k[b][:, g, mp] *= 0.05
    case.k[b][j, g, mp] = q / np.dot(q, q) * score / case.scale
    for x in (case.k[b],):
        x[:] = bf16_round(x)[1]
    case.v[b][j, g] = bf16_round((10 * np.sign(case.v[b][j, g])).astype(np.float32))[1]


@pytest.mark.parametrize("window,keep", [(40, 3), (64, 0), (65, 4), (1, 1), (128, 70), (17, 64)])
@pytest.mark.parametrize("start,n_q", [(0, 200), (199, 1), (150, 50)])
def test_window_and_kept_edges(dev, window, keep, start, n_q):
    """Key just inside / just outside the window, last kept / first dropped token, key on both sides of a 64-key tile."""
    rng = np.random.default_rng(window * 1000 + keep)
    pos = 199
    keys = {pos - window + 1, pos - window, 0, keep - 1, keep, 63, 64, 127, 128, pos, pos - 1}
    for n, j in enumerate(sorted(k for k in keys if 0 <= k <= pos)):
        case = Case(rng, 4, 2, 24, 40, window, keep, seqs=[(start, n_q)], max_seq=200)
        i = pos - start
        head, mp = n % 4, n % 2
        plain = case.want(0, [i])
        _stand_out(case, 0, i, j, 12.0, head, mp)
        seen = T.visible(pos, j, window, keep)
        moved = np.abs(case.want(0, [i])[0, head] - plain[0, head]).max() > 0.2
        assert seen == moved or not seen           # (the planted key decides the head's result when it is seen)
        check(dev, case, rows=[i])


def test_far_key_among_many(dev):
    """One key of 2000 stands out, at several distances, under a window that covers all of them."""
    rng = np.random.default_rng(77)
    for j in (0, 1, 700, 1023, 1024, 1999):
        case = Case(rng, 2, 1, 32, 64, 5000, 0, seqs=[(1999, 1), (1990, 10)], max_seq=2000)
        _stand_out(case, 0, 0, j, 14.0, 0, 0)
        _stand_out(case, 1, 9, min(j, 1999), 14.0, 1, 1)
        import tang_b200 as tb

        for dtype, tol in ((tb.F32, 3e-5), (tb.BF16, 1.5e-2)):
            got = case.run(dev, dtype)
            assert np.abs(got[0] - case.want(0)).max() < tol * 3
            assert np.abs(got[1][9:] - case.want(1, [9])).max() < tol * 3


def test_a_query_far_from_the_scores_of_others(dev):
    """Large scores (softmax close to one key) and a balance above one: no overflow, no lost difference."""
    rng = np.random.default_rng(5)
    check(dev, Case(rng, 4, 2, 32, 48, 50, 2, seqs=[(0, 66), (70, 1)], lam=1.7, scale=1.5, spread=1.0))


def test_result_does_not_depend_on_slots_or_batch(dev):
    import tang_b200 as tb

    rng = np.random.default_rng(9)
    case = Case(rng, 6, 2, 24, 40, 37, 2, seqs=[(90, 1), (3, 1), (200, 1)])
    together = case.run(dev, tb.BF16)
    for b in range(3):
        single = Case(np.random.default_rng(1), 6, 2, 24, 40, 37, 2, seqs=[case.seqs[b]])
        single.k, single.v, single.q = [case.k[b]], [case.v[b]], [case.q[b]]
        assert np.abs(single.run(dev, tb.BF16)[0] - together[b]).max() < 2e-2


def test_bad_arguments_are_refused(dev):
    import tang_b200 as tb

    p = dev.alloc(4096, tb.F32)
    ptr = C.c_void_p(p.ptr)
    for H, G, D, window in ((3, 2, 16, 4), (4, 2, 16, 0), (4, 2, 0, 4)):
        cfg = _Cfg(H, G, D, 16, window, 0, 1.0, 1.0, 1.0, EPS)
        st = dev._L.tq_diff_attention(dev._ctx, C.byref(cfg), tb.F32, ptr, 64, ptr, ptr, 8, C.c_void_p(0), ptr, ptr, 1, 1, 1, 1, ptr, 64)
        assert st == tb._lib.TQ_EINVAL
