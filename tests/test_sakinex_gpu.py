"""The Sakinex family on the device, whole model: loading, prompts, portions, decoding, ragged batches, slots and states used again,
generation and the trace runner, against the numpy implementation in 32-bit and in bf16."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import sakinex_oracle as X
from sakinex_util import CONFIGS, TOL, config, layer, moe, reference, row_errors, save, views, weights
from util import bf16_round

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


@pytest.fixture(scope="module")
def dev():
    import tang_b200

    d = tang_b200.QuantComputeDevice(0)
    yield d
    d.close()


@pytest.fixture(scope="module")
def refs():
    """Logits of one prompt per configuration, computed once."""
    out = {}
    for name, cfg in CONFIGS.items():
        w = weights(cfg, 3)
        tokens = [int(t) for t in np.random.default_rng(12).integers(0, cfg["vocab"], 150)]
        out[name] = (cfg, w, tokens, reference(cfg, w, tokens))
    return out


def make(dev, cfg, w, dtype, **kw):
    import tang_b200 as tb

    return tb.SakinexModel.from_tensors(dev, cfg, views(w), tb.F32 if dtype == "f32" else tb.BF16, **kw)


def engine(model, **kw):
    from tang_b200 import Engine

    return Engine(model, **kw)


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_prompt_portions_and_decoding(dev, refs, name, dtype):
    cfg, w, tokens, want = refs[name]
    model = make(dev, cfg, w, dtype, max_slots=6, max_seq=160)
    e = engine(model)
    n = len(tokens)
    cuts = {"whole": [n], "portions": [30, 60, n], "twos": list(range(2, n, 2)) + [n], "chunks": [64, 128, n], "around": [63, 65, 127, 130, n],
            "mixed": [1, 3, 40, 41, 43, n], "decode": [100] + list(range(101, n + 1)), "single": list(range(1, n + 1))}
    for label, ends in cuts.items():
        got, a = [], 0
        for b in ends:
            got.append(e.step([(label, tokens[a:b], range(b - a))]))
            a = b
        e.close(label)
        err = row_errors(np.concatenate(got), want)
        assert err.max() < TOL[dtype], (label, int(err.argmax()), err.max())
    model.destroy()


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("name", ["mixed", "aligned"])
def test_stream_after_every_run(dev, refs, name, dtype):
    """In a prompt, and in the decode step behind it; what is added ahead of a pass is not part of the run before."""
    import tang_b200 as tb

    cfg, w, tokens, _ = refs[name]
    model = make(dev, cfg, w, dtype, max_slots=1, max_seq=160)
    trace = []
    m = X.Sakinex(cfg, w)
    m.forward(tokens[:80], m.new_state(), trace)
    buf, e = dev.alloc(len(trace) * 79 * cfg["width"], tb.F32), engine(model)
    model.trace(buf)
    for part, rows in ((tokens[:79], slice(0, 79)), (tokens[79:80], slice(79, 80))):
        e.step([(0, part, [])])
        got = buf.to_vec()[:len(trace) * len(part) * cfg["width"]].reshape(len(trace), len(part), -1)
        for i, (g, x) in enumerate(zip(got, trace)):
            assert row_errors(g, x[rows]).max() < TOL[dtype], (i, rows)
    model.trace(None)
    model.destroy()


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("name", ["mixed", "odd", "aligned"])
def test_ragged_batches_equal_each_alone_and_slots_are_reused(dev, refs, name, dtype):
    """Unequal prompts start together, others join while they decode, some end early; freed slots (caches, pooled rows and states) serve
    new requests."""
    cfg, w, _, _ = refs[name]
    rng = np.random.default_rng(3)
    model = make(dev, cfg, w, dtype, max_slots=5, max_seq=100)
    e = engine(model, max_rows=70)
    lengths = {"a": 1, "b": 70, "c": 24, "d": 96, "e": 2, "f": 65, "g": 33, "h": 1}
    toks = {r: [int(t) for t in rng.integers(0, cfg["vocab"], n)] for r, n in lengths.items()}
    want = {r: reference(cfg, w, t) for r, t in toks.items()}
    at = {r: 0 for r in toks}
    got = {r: [] for r in toks}

    def step(counts):
        entries = [(r, toks[r][at[r]:at[r] + n], range(n)) for r, n in counts.items()]
        out, k = e.step(entries), 0
        for r, n in counts.items():
            got[r].append(out[k:k + n])
            k += n
            at[r] += n
            if at[r] == lengths[r]:
                e.close(r)

    step({"a": 1, "b": 66, "c": 20, "d": 90})         # (cut in portions of at most 70 rows)
    for _ in range(4):
        step({"d": 1, "b": 1, "c": 1})
    step({"e": 2, "d": 1})                            # e takes a freed slot
    step({"f": 40, "d": 1, "g": 30, "h": 1})
    step({"f": 25, "g": 3})
    assert all(at[r] == lengths[r] for r in toks) and len(e.pool.free) == 5
    for r in toks:
        assert row_errors(np.concatenate(got[r]), want[r]).max() < TOL[dtype], r
    model.destroy()


@pytest.mark.parametrize("name,rows", [("mixed", 1), ("mixed", 5), ("aligned", 2), ("aligned", 8), ("aligned", 9), ("odd", 24), ("aligned", 40), ("mixed", 70)])
def test_decode_batches(dev, refs, name, rows):
    """Decode steps on both sides of the GEMV's row limits, every sequence at its own position."""
    cfg, w, tokens, want = refs[name]
    model = make(dev, cfg, w, "bf16", max_slots=rows, max_seq=100)
    e = engine(model)
    lens = [1 + (7 * i) % 80 for i in range(rows)]
    e.step([(i, tokens[:n], []) for i, n in enumerate(lens)])
    for k in range(3):
        got = e.step([(i, [tokens[n + k]], [0]) for i, n in enumerate(lens)])
        assert row_errors(got, want[[n + k for n in lens]]).max() < TOL["bf16"]
    model.destroy()


def test_large_prompt_batch(dev, refs):
    """Enough rows for many jobs per expert, row tiles of the widest size and several rows per thread of the convolutions."""
    cfg, w, tokens, want = refs["aligned"]
    model = make(dev, cfg, w, "bf16", max_slots=40, max_seq=160)
    e = engine(model)
    got = e.step([(i, tokens[:150 - i], [149 - i, 3]) for i in range(40)])
    assert row_errors(got, np.concatenate([want[[149 - i, 3]] for i in range(40)])).max() < TOL["bf16"]
    got = e.step([(i, tokens[150 - i:151 - i], [0]) for i in range(1, 40)])       # the states that it left
    assert row_errors(got, want[[150 - i for i in range(1, 40)]]).max() < TOL["bf16"]
    model.destroy()


def _planted(window, pool, n, j, i, dim=16):
    """A one-layer model in which the token at position i looks for what the token at position j left, and no convolution smears it;
    token ids carry the match, so that the same weights serve any pair of positions."""
    cfg = config([layer(2, 1, dim, 24, window, pool, 16, rot=4, scale=4.0, left=1.0, right=0.2)], width=64, vocab=40, taps=2, mult=1.0)
    w = weights(cfg, 21)
    rng = np.random.default_rng(22)
    w["embed"][:, :2] = 0
    w["embed"][38], w["embed"][39] = 0, 0
    w["embed"][38, 0], w["embed"][39, 1] = 8.0, 8.0
    w["l0.norm1"][:] = 1
    w["l0.canon1"][:] = [0, 0.25]
    left = lambda name: w["l0.mix.left." + name]
    for name in ("q", "k", "v"):
        left(name + ".conv")[:] = 0
        left(name + ".conv")[:, -1] = 1
    d = dim - 1                                       # not a rotated dimension
    left("q")[:, 0] *= 0.05
    left("q")[d::dim, 0] = 2.0
    left("k")[d] = 0
    left("k")[:, 1] *= 0.05
    left("k")[d, 1] = 2.0
    left("v")[:, 1] = rng.standard_normal(len(left("v"))) * 3
    tokens = rng.integers(0, 38, n)
    tokens[i], tokens[j] = 38, 39
    return cfg, {k: bf16_round(np.asarray(v, np.float32))[1] for k, v in w.items()}, [int(t) for t in tokens]


@pytest.mark.parametrize("window,pool", [(40, 4), (64, 16), (65, 5), (130, 2), (7, 64), (1, 3)])
def test_edges_of_window_and_blocks_show_in_prompts_and_in_decoding(dev, window, pool):
    n, i = 190, 177
    blocks = len(X.seen_blocks(i, window, pool))
    near = {i - window + 1, i - window, i - window - 1, i - 1, 0, 1, 63, 64, 127, 128}
    near |= {blocks * pool - 1, blocks * pool, blocks * pool + pool - 1, (blocks - 1) * pool, pool - 1, pool}      # the last block seen, the first one not seen
    for j in sorted({p for p in near if 0 <= p < i}):
        cfg, w, tokens = _planted(window, pool, n, j, i)
        want = reference(cfg, w, tokens[:i + 1])[i]
        if i - j < window or j // pool < blocks:      # (of a block's key only a share stands out)
            blind = list(tokens)
            blind[j] = 0
            assert row_errors(reference(cfg, w, blind[:i + 1])[i][None], want[None])[0] > 0.1, j
        for dtype in ("f32", "bf16"):
            model = make(dev, cfg, w, dtype, max_slots=3, max_seq=n)
            e = engine(model)
            whole = e.step([("whole", tokens[:i + 1], [i])])
            e.step([("decoded", tokens[:i - 3], [])])
            for p in range(i - 3, i):
                e.step([("decoded", [tokens[p]], [])])
            one = e.step([("decoded", [tokens[i]], [0])])
            for a in range(0, i - 1, 40):
                e.step([("cut", tokens[a:min(a + 40, i - 1)], [])])
            two = e.step([("cut", tokens[i - 1:i + 1], [1])])
            for got in (whole, one, two):
                assert row_errors(got, want[None]).max() < TOL[dtype], (j, dtype)
            model.destroy()


def test_the_recurrence_reaches_far_back(dev):
    """Gates that are almost shut keep what the first tokens left; the same slot then starts from nothing."""
    cfg = config([layer(1, 1, 8, 8, 4, 2, 48, left=0.1, right=2.0), layer(2, 1, 8, 8, 4, 2, 24, right=1.0)], width=40, vocab=30, loop=(0, 1, 2), mult=1.0)
    w = weights(cfg, 17)
    w["l0.mix.right.z.b"][:] = -8
    w["l1.mix.right.z.b"][::2] = -8
    rng = np.random.default_rng(18)
    tokens = [int(t) for t in rng.integers(0, 30, 300)]
    other = [(t + 7) % 30 for t in tokens[:2]] + tokens[2:]
    want, changed = reference(cfg, w, tokens), reference(cfg, w, other)
    for dtype in ("f32", "bf16"):
        assert row_errors(changed[-1:], want[-1:])[0] > 5 * TOL["f32"]
        model = make(dev, cfg, w, dtype, max_slots=1, max_seq=300)
        e = engine(model)
        for toks, ref in ((tokens, want), (other, changed)):
            got = np.concatenate([e.step([(0, toks[:257], range(257))])] + [e.step([(0, [t], [0])]) for t in toks[257:]])
            assert row_errors(got, ref).max() < TOL[dtype]
            e.close(0)
        model.destroy()


def test_long_decoding_crosses_windows_blocks_and_tiles(dev):
    cfg = config([layer(4, 2, 24, 16, 21, 4, 24, moe(3, 1, 24, 16)), layer(2, 1, 16, 32, 100, 16, 32, moe(4, 2, 24)), layer(4, 4, 8, 8, 3, 1, 20)], loop=(1, 3, 2))
    w = weights(cfg, 31)
    tokens = [int(t) for t in np.random.default_rng(32).integers(0, cfg["vocab"], 270)]
    want = reference(cfg, w, tokens)
    for dtype in ("f32", "bf16"):
        model = make(dev, cfg, w, dtype, max_slots=1, max_seq=270)
        e = engine(model)
        got = [e.step([(0, tokens[:5], range(5))])] + [e.step([(0, [t], [0])]) for t in tokens[5:]]
        assert row_errors(np.concatenate(got), want).max() < TOL[dtype]
        model.destroy()


@pytest.mark.parametrize("layers,width,vocab,taps,loop", [
    ([layer(1, 1, 2, 1, 1, 1, 1, moe(1, 1, 1, 1), conv=1, rot=2), layer(1, 1, 1, 2, 2, 3, 2, moe(2, 2, 3), rot=0)], 12, 5, 1, (0, 1, 3)),
    ([layer(33, 1, 8, 8, 9, 2, 16, None, scaling=(1.0, 32, 4.0, 1.0)), layer(1, 1, 16, 16, 200, 4, 40, moe(16, 6, 8, 20))], 40, 1000, 2, None),
    ([layer(3, 1, 8, 8, 3, 200, 200, moe(4, 4, 130, 5), conv=9, rot=2), layer(130, 2, 8, 9, 9, 6, 8, None, rot=4)], 136, 30, 8, (1, 2, 4))])
def test_other_sizes(dev, layers, width, vocab, taps, loop):
    cfg = config(layers, width=width, vocab=vocab, taps=taps, loop=loop)
    w = weights(cfg, 8)
    tokens = [int(t) for t in np.random.default_rng(9).integers(0, vocab, 70)]
    want = reference(cfg, w, tokens)
    for dtype in ("f32", "bf16"):
        model = make(dev, cfg, w, dtype, max_slots=2, max_seq=70)
        e = engine(model)
        a = e.step([(0, tokens, range(70))])
        b = np.concatenate([e.step([(1, tokens[:30], range(30))])] + [e.step([(1, [t], [0])]) for t in tokens[30:]])
        for got in (a, b):
            assert row_errors(got, want).max() < TOL[dtype] * 1.5
        model.destroy()


def test_parts_that_are_not_there(dev):
    """No window, no blocks, no convolution on the heads, no rotation, no shared expert, no loop."""
    cfg = config([layer(4, 2, 16, 24, 1000, 0, 32, moe(3, 2, 24), conv=0), layer(2, 1, 24, 8, 9, 0, 16, rot=0)])
    del cfg["layers"][0]["mixer"]["left"]["mask"], cfg["layers"][1]["mixer"]["left"]["mask"]["pool"], cfg["layers"][1]["mixer"]["left"]["rot"]
    plain = json.loads(json.dumps(cfg))
    for l in plain["layers"]:                          # what they mean: a window over everything, blocks longer than the prompt, no pair that turns
        l["mixer"]["left"].setdefault("mask", {"size": 1000})["pool"] = 1000
        l["mixer"]["left"].setdefault("rot", {"dims": 0, "base": 10.0})
    w = weights(plain, 13)
    tokens = [int(t) for t in np.random.default_rng(14).integers(0, cfg["vocab"], 90)]
    want = reference(plain, w, tokens)
    for dtype in ("f32", "bf16"):
        model = make(dev, cfg, w, dtype, max_slots=1, max_seq=90)
        e = engine(model)
        got = np.concatenate([e.step([(0, tokens[:60], range(60))])] + [e.step([(0, [t], [0])]) for t in tokens[60:]])
        assert row_errors(got, want).max() < TOL[dtype]
        model.destroy()


def test_long_rows_split_over_k(dev):
    """Wide enough that the router's and the mixers' products are split over k."""
    cfg = config([layer(2, 1, 16, 16, 20, 4, 600, moe(20, 3, 40, 200)), layer(2, 2, 16, 32, 30, 6, 700)], width=1100, vocab=50)
    w = weights(cfg, 41)
    tokens = [int(t) for t in np.random.default_rng(42).integers(0, 50, 90)]
    model = make(dev, cfg, w, "bf16", max_slots=1, max_seq=90)
    assert row_errors(engine(model).step([(0, tokens, range(90))]), reference(cfg, w, tokens)).max() < TOL["bf16"]
    model.destroy()


def greedy(cfg, w, prompt, n):
    m = X.Sakinex(cfg, w)
    st = m.new_state()
    lg, out, gaps = m.forward(prompt, st)[-1], [], []
    for _ in range(n):
        top = np.sort(lg)[-2:]
        gaps.append((top[1] - top[0]) / np.sqrt(np.mean(lg ** 2)))
        out.append(int(lg.argmax()))
        lg = m.forward(out[-1:], st)[0]
    return out, gaps


def test_greedy_generation(dev, refs):
    """``generate`` (one ragged prefill, then the replayed graph) gives the numpy model's tokens, for prompts of unequal
    lengths, one of a single token."""
    cfg, w, tokens, _ = refs["mixed"]
    prompts = [tokens[:1], tokens[5:40], tokens[2:90], tokens[10:13]]
    model = make(dev, cfg, w, "f32", max_slots=4, max_seq=128)
    out = model.generate_greedy(prompts, 24)
    for b, p in enumerate(prompts):
        want, gaps = greedy(cfg, w, p, 24)
        assert min(gaps) > 2e-5
        assert out[b].tolist() == want
    assert np.array_equal(model.generate_greedy(prompts[1:3], 24), out[1:3])      # slots used again
    m16 = make(dev, cfg, w, "bf16", max_slots=4, max_seq=128)
    out16 = m16.generate_greedy(prompts, 24)
    for b, p in enumerate(prompts):
        seq = list(p) + out16[b].tolist()
        lg = reference(cfg, w, seq)[len(p) - 1:-1]
        short = lg.max(1) - lg[np.arange(24), out16[b]]
        assert short.max() < 0.1 * np.sqrt(np.mean(lg ** 2))
    model.destroy()
    m16.destroy()


def test_sampling_with_penalty_sees_each_prompt(dev, refs, orc):
    """Unequal prompts through temperature / top-k / top-p / repetition penalty: the draws equal the sampler's restatement
    on the device's own logits, stepped by hand."""
    import tang_b200 as tb

    cfg, w, tokens, _ = refs["mixed"]
    prompts = [tokens[:3], tokens[20:61]]
    vals = (25.0, 20, 0.9, 1.4)
    model = make(dev, cfg, w, "bf16", max_slots=2, max_seq=64)
    out = model.generate(prompts, 8, tb.SamplerConfig(*vals), seed=5)
    e = engine(model)
    for b, p in enumerate(prompts):
        seq, state = list(p), 5
        # the same cut as ``generate``: all but the last token, then one by one
        e.step([(b, p[:-1], [])])
        lg = e.step([(b, p[-1:], [0])])[0]
        for t in out[b]:
            draw, state = orc.sampler_sample(lg.astype(np.float64), orc.SamplerConfig(*vals), state, past=seq)
            assert draw == t
            seq.append(draw)
            lg = e.step([(b, [draw], [0])])[0]
    model.destroy()


def test_bad_models_and_steps_are_refused(dev, refs):
    import tang_b200 as tb

    cfg, w, tokens, _ = refs["mixed"]
    for gone in ("l1.mix.left.k.conv", "l0.mlp.e4.up", "l2.canon1", "l0.mlp.router.b", "l0.mlp.shared.sg", "l3.mix.right.x.b", "head"):
        v = views(w)
        del v[gone]
        with pytest.raises(tb.SafetensorsError, match=gone):
            tb.SakinexModel.from_tensors(dev, cfg, v)
    for name, shape in (("l0.mlp.e1.up", (24, 71)), ("l1.mix.left.o", (72, 25)), ("l0.canon2", (72, 4)), ("l2.mix.left.q.conv", (64, 3)), ("l3.mix.right.z.b", (25,)),
                        ("l0.mlp.shared.sg", (2, 72))):
        v = views(w)
        v[name] = tb.TensorView("BF16", shape, np.zeros(int(np.prod(shape)), np.uint16))
        with pytest.raises(tb.TangqError, match="must be"):
            tb.SakinexModel.from_tensors(dev, cfg, v)
    for change, what in ((lambda c: c["layers"][0]["mlp"]["router"].update(top=9), "experts"), (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=7), "rotation"),
                         (lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=4), "multiple")):
        bad = json.loads(json.dumps(cfg))
        change(bad)
        with pytest.raises(tb.TangqError, match=what):
            tb.SakinexModel.from_tensors(dev, bad, views(w))
    model = make(dev, cfg, w, "bf16", max_slots=2, max_seq=32)
    e = engine(model)
    with pytest.raises(tb.TangqError, match="positions"):
        e.step([(0, tokens[:33], [])])
    # a position behind the cache that only the device sees is skipped and reported, and the model goes on
    lg = dev.alloc(2 * cfg["vocab"])
    tok, pos = dev.upload(np.array([1, 2], np.int32), tb.I32), dev.upload(np.array([32, 0], np.int32), tb.I32)
    model.decode(tok, pos, 2, 32, lg)
    with pytest.raises(tb.TangqError, match="position"):
        dev.sync()
    assert row_errors(e.step([(0, tokens[:20], range(20))]), reference(cfg, w, tokens[:20])).max() < TOL["bf16"]
    model.destroy()


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_command_line(dev, refs, tmp_path, dtype):
    cfg, w, tokens, want = refs["odd"]
    save(tmp_path, cfg, w)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": tokens[:40], "want": [39, 0]}, {"id": "y", "tokens": tokens[:3], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": tokens[40:41], "want": []}, {"id": "y", "tokens": tokens[3:4], "want": []}], "end": ["y"]},
             {"step": 2, "entries": [{"id": "x", "tokens": tokens[41:42], "want": [0]}], "end": ["x"]},
             {"step": 3, "entries": [{"id": "y", "tokens": tokens[:9], "want": [8]}], "end": ["y"]}]
    text = "\n".join(json.dumps(s) for s in steps) + "\n"
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", dtype, "--out", str(tmp_path), "--max-tokens", "64"],
                       input=text, capture_output=True, text=True)
    assert r.returncode == 0, r.stderr
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
    tol = TOL["f32" if dtype == "float32" else "bf16"]
    for step, rows in ((0, [39, 0]), (2, [41]), (3, [8])):
        got = np.fromfile(tmp_path / f"{step}.f32", "<f4").reshape(len(rows), cfg["vocab"])
        assert row_errors(got, want[rows]).max() < tol
    assert not (tmp_path / "1.f32").exists()
    if dtype == "float32":
        r = subprocess.run([sys.executable, "-m", "tang_b200", "generate", "--model", str(tmp_path), "--prompt", ",".join(map(str, tokens[:7])),
                            "--prompt", str(tokens[0]), "--max-new", "6", "--dtype", dtype], capture_output=True, text=True, cwd=ROOT)
        assert r.returncode == 0, r.stderr
        lines = [[int(x) for x in l.split(",")] for l in r.stdout.split()]
        assert lines == [greedy(cfg, w, tokens[:7], 6)[0], greedy(cfg, w, tokens[:1], 6)[0]]
