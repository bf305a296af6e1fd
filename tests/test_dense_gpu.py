"""Dense linear layers and the small Tofazen operators against plain numpy."""
import ctypes as C

import numpy as np
import pytest

import tofazen_oracle as T
from util import bf16_round, rel_err

pytestmark = pytest.mark.gpu


@pytest.fixture(scope="module")
def dev():
    import tang_b200

    d = tang_b200.QuantComputeDevice(0)
    yield d
    d.close()


class Dense:
    def __init__(self, dev, rows, cols, dtype):
        self.dev, self.rows, self.cols = dev, rows, cols
        h = C.c_void_p()
        dev._check(dev._L.tq_dweight_create(dev._ctx, rows, cols, dtype, C.byref(h)))
        self.h = h

    def put(self, w, row0=0, col0=0, interleave=0):
        from tang_b200 import F32

        w = np.ascontiguousarray(w, np.float32)
        self.dev._check(self.dev._L.tq_dweight_put(self.dev._ctx, self.h, C.c_void_p(w.ctypes.data), F32, *w.shape, row0, col0, interleave))
        return self

    def __call__(self, x, m, y_dtype, ldx=0):
        y = self.dev.alloc(m * self.rows, y_dtype)
        self.dev._check(self.dev._L.tq_dlinear(self.dev._ctx, self.h, C.c_void_p(x.ptr), ldx, m, C.c_void_p(y.ptr), y_dtype, 0))
        self.dev.sync()
        out = y.to_vec().reshape(m, self.rows)
        return out if y_dtype == 0 else (out.astype(np.uint32) << 16).view(np.float32)

    def free(self):
        self.dev._L.tq_dweight_free(self.dev._ctx, self.h)


# rows x cols: below one tile, ragged in both, several tiles, K that splits
SHAPES = [(1, 8), (24, 40), (130, 72), (257, 200), (384, 1000), (1100, 328), (160, 4104)]
# activation rows: the GEMV's limits, the first of the tensor-core kernel, tile borders
ROWS = [1, 2, 3, 7, 8, 9, 16, 17, 100, 255, 257, 700]


@pytest.mark.parametrize("shape", SHAPES)
def test_dlinear_bf16(dev, shape):
    import tang_b200 as tb

    rows, cols = shape
    rng = np.random.default_rng(rows)
    w = bf16_round(rng.standard_normal(shape).astype(np.float32))[1]
    lin = Dense(dev, rows, cols, tb.BF16).put(w)
    for m in ROWS:
        bits, x = bf16_round(rng.standard_normal((m, cols)).astype(np.float32))
        want = x.astype(np.float64) @ w.T.astype(np.float64)
        xb = dev.upload(bits, tb.BF16)
        assert rel_err(lin(xb, m, tb.F32), want, 1.0) < 1e-3, m
        assert rel_err(lin(xb, m, tb.BF16), want, 1.0) < 5e-3, m
    lin.free()


def test_dlinear_bf16_strided_activations(dev):
    """Few rows on both sides of what the GEMV keeps in shared memory, a ragged last k chunk, a row stride with garbage
    behind the columns."""
    import tang_b200 as tb

    rng = np.random.default_rng(4)
    rows, cols, ld = 48, 9000, 9216
    w = bf16_round(rng.standard_normal((rows, cols)).astype(np.float32))[1]
    lin = Dense(dev, rows, cols, tb.BF16).put(w)
    for m in (1, 5, 8):
        bits, x = bf16_round(rng.standard_normal((m, ld)).astype(np.float32))
        bits[:, cols:] = 0x7FC0                      # not a number
        got = lin(dev.upload(bits, tb.BF16), m, tb.F32, ldx=ld)
        assert rel_err(got, x[:, :cols].astype(np.float64) @ w.T.astype(np.float64), 1.0) < 1e-3
    lin.free()


@pytest.mark.parametrize("shape", SHAPES[:6])
def test_dlinear_f32_is_f32(dev, shape):
    import tang_b200 as tb

    rows, cols = shape
    rng = np.random.default_rng(rows + 1)
    w = rng.standard_normal(shape).astype(np.float32)
    lin = Dense(dev, rows, cols, tb.F32).put(w)
    for m in (1, 5, 64, 65, 300):
        x = rng.standard_normal((m, cols)).astype(np.float32)
        want = x.astype(np.float64) @ w.T.astype(np.float64)
        assert rel_err(lin(dev.upload(x), m, tb.F32), want, 1.0) < 1e-5   # (f32 sums of up to 1000 terms; tf32 gives 1e-3)
    lin.free()


def test_dweight_blocks_and_gate_up_order(dev):
    import tang_b200 as tb

    rng = np.random.default_rng(8)
    a, b = (rng.standard_normal((13, 21)).astype(np.float32) for _ in range(2))
    lin = Dense(dev, 48, 30, tb.F32).put(a, 0, 1, 1).put(b, 0, 1, 2)
    p, rp, cp = C.c_void_p(), C.c_size_t(), C.c_size_t()
    dev._check(dev._L.tq_dweight_data(lin.h, C.byref(p), C.byref(rp), C.byref(cp)))
    got = tb.Buffer(dev, p.value, rp.value * cp.value, tb.F32, owns=False).to_vec().reshape(rp.value, cp.value)
    want = np.zeros_like(got)
    for i in range(13):
        want[i // 8 * 16 + i % 8, 1:22] = a[i]
        want[i // 8 * 16 + 8 + i % 8, 1:22] = b[i]
    assert np.array_equal(got, want)
    for bad in (lambda: lin.put(a, 40, 0), lambda: lin.put(a, 0, cp.value - 20), lambda: lin.put(a, 8, 0, 1), lambda: lin.put(a, 32, 0, 2)):
        with pytest.raises(tb.TangqError):
            bad()
    lin.free()


@pytest.mark.parametrize("limit,alpha", [(1.25, 1.702), (7.0, 0.5)])
def test_clamped_glu(dev, limit, alpha):
    import tang_b200 as tb

    rng = np.random.default_rng(3)
    g = np.concatenate([rng.standard_normal(1000) * 4, [limit, -limit, 1e4, -1e4, 0.0]]).astype(np.float32)
    u = np.concatenate([rng.standard_normal(1000) * 4, [-limit, limit, -1e4, 1e4, -1.0]]).astype(np.float32)
    gb, ub, y = dev.upload(g), dev.upload(u), dev.alloc(g.size)
    dev._check(dev._L.tq_clamped_glu(dev._ctx, C.c_void_p(gb.ptr), C.c_void_p(ub.ptr), tb.F32, g.size, limit, alpha, C.c_void_p(y.ptr), tb.F32))
    g64, u64 = np.minimum(g.astype(np.float64), limit), np.clip(u.astype(np.float64), -limit, limit)
    with np.errstate(over="ignore"):
        want = g64 / (1 + np.exp(-alpha * g64)) * (u64 + 1)
        assert alpha != 1.702 or np.array_equal(want, T.clamped_glu(g.astype(np.float64), u.astype(np.float64), limit))
    assert np.abs(y.to_vec() - want).max() < 1e-5


def test_embedding_pos(dev):
    import tang_b200 as tb

    rng = np.random.default_rng(6)
    vocab, dim, n_pos, max_seq, n_slots = 50, 37, 40, 32, 5
    (tbits, table), (pbits, pos) = (bf16_round(rng.standard_normal((n, dim)).astype(np.float32)) for n in (vocab, n_pos))
    counts, starts, slots = [3, 1, 0, 7, 2], [0, 31, 4, 25, 9], [4, 0, 3, 1, 2]
    cu = np.cumsum([0] + counts)
    ids = rng.integers(0, vocab, cu[-1])
    i32 = lambda a: dev.upload(np.asarray(a, np.int32), tb.I32)
    tb_, pb_ = dev.upload(tbits, tb.BF16), dev.upload(pbits, tb.BF16)

    def run(ids, cu, starts, slots, rows):
        out, rp, cr = dev.alloc(rows * dim), dev.alloc(rows, tb.I32), dev.alloc(rows, tb.I32)
        keep = [i32(ids), None if cu is None else i32(cu), i32(starts), None if slots is None else i32(slots)]
        ptr = [C.c_void_p(b.ptr if b else 0) for b in keep]
        dev._check(dev._L.tq_embedding_pos(dev._ctx, C.c_void_p(tb_.ptr), C.c_void_p(pb_.ptr), tb.BF16, *ptr, len(starts), rows, dim, vocab, n_pos,
                                           max_seq, n_slots, C.c_void_p(out.ptr), C.c_void_p(rp.ptr), C.c_void_p(cr.ptr)))
        return out.to_vec().reshape(rows, dim), rp.to_vec(), cr.to_vec()

    x, rp, cr = run(ids, cu, starts, slots, cu[-1])
    dev.sync()
    for b, n in enumerate(counts):
        if n:
            want = T.embed(ids[cu[b]:cu[b + 1]], starts[b], table, pos)
            assert np.array_equal(x[cu[b]:cu[b + 1]], want.astype(np.float32))
            assert rp[cu[b]:cu[b + 1]].tolist() == list(range(starts[b], starts[b] + n))
            assert cr[cu[b]:cu[b + 1]].tolist() == [slots[b] * max_seq + p for p in range(starts[b], starts[b] + n)]
    x, rp, cr = run([1, 2], None, [3, 5], None, 2)
    dev.sync()
    assert rp.tolist() == [3, 5] and cr.tolist() == [3, max_seq + 5]
    # a position behind the cache, a slot that does not exist: no cache row, and the next sync says so
    for starts_, slots_ in (([32, 0], [0, 1]), ([0, 0], [5, 1]), ([-1, 0], [0, 1])):
        _, _, cr = run([1, 2], None, starts_, slots_, 2)
        assert cr.tolist() == [-1, max_seq]
        with pytest.raises(tb.TangqError, match="position"):
            dev.sync()
    dev.sync()
