"""The Tofazen family on the device, whole model: loading, prompts, portions, decoding, ragged batches, slots used again,
generation and the trace runner, against the numpy implementation in 32-bit and in bf16."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import tofazen_oracle as T
from tofazen_util import CONFIGS, TOL, config, layer, reference, row_errors, save, views, weights

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
        w = weights(cfg, 11)
        tokens = list(np.random.default_rng(12).integers(0, cfg["vocab"], 90))
        out[name] = (cfg, w, tokens, reference(cfg, w, tokens))
    return out


def make(dev, cfg, w, dtype, **kw):
    import tang_b200 as tb

    return tb.TofazenModel.from_tensors(dev, cfg, views(w), tb.F32 if dtype == "f32" else tb.BF16, **kw)


def engine(model, **kw):
    from tang_b200 import Engine

    return Engine(model, **kw)


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_prompt_portions_and_decoding(dev, refs, name, dtype):
    cfg, w, tokens, want = refs[name]
    model = make(dev, cfg, w, dtype, max_slots=6, max_seq=128)
    e = engine(model)
    n = len(tokens)
    cuts = {"whole": [n], "portions": [30, 60, n], "twos": list(range(2, n, 2)) + [n], "mixed": [1, 3, 40, 41, 43, n],
            "decode": [66] + list(range(67, n + 1)), "single": list(range(1, n + 1))}
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
def test_stream_after_every_layer(dev, refs, dtype):
    import tang_b200 as tb

    cfg, w, tokens, _ = refs["mixed"]
    model = make(dev, cfg, w, dtype, max_slots=1)
    trace = []
    m = T.Tofazen(cfg, w)
    m.forward(tokens[:29], m.new_state(), trace)
    buf = dev.alloc(len(trace) * 29 * cfg["width"], tb.F32)
    model.trace(buf)
    engine(model).step([(0, tokens[:29], [])])
    for i, (g, x) in enumerate(zip(buf.to_vec().reshape(len(trace), 29, -1), trace)):
        assert row_errors(g, x).max() < TOL[dtype], i
    model.trace(None)
    model.destroy()


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_ragged_batches_equal_each_alone_and_slots_are_reused(dev, refs, dtype):
    """Unequal prompts start together, others join while they decode, some end early; freed slots serve new requests."""
    cfg, w, _, _ = refs["mixed"]
    rng = np.random.default_rng(3)
    model = make(dev, cfg, w, dtype, max_slots=5, max_seq=96)
    e = engine(model, max_rows=50)
    lengths = {"a": 1, "b": 70, "c": 24, "d": 96, "e": 2, "f": 65, "g": 33}
    toks = {r: list(rng.integers(0, cfg["vocab"], n)) for r, n in lengths.items()}
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

    step({"a": 1, "b": 66, "c": 20, "d": 90})         # (cut in portions of at most 50 rows)
    for _ in range(4):
        step({"d": 1, "b": 1, "c": 1})
    step({"e": 2, "d": 1})                            # e takes a freed slot
    step({"f": 40, "d": 1, "g": 30})
    step({"f": 25, "g": 3})
    assert all(at[r] == lengths[r] for r in toks) and len(e.pool.free) == 5
    for r in toks:
        assert row_errors(np.concatenate(got[r]), want[r]).max() < TOL[dtype], r
    model.destroy()


@pytest.mark.parametrize("rows", [1, 2, 5, 8, 9, 24, 40])
def test_decode_batches(dev, refs, rows):
    """Decode steps on both sides of the GEMV's row limit, every sequence at its own position."""
    cfg, w, tokens, want = refs["wide_group"]
    model = make(dev, cfg, w, "bf16", max_slots=rows, max_seq=100)
    e = engine(model)
    lens = [1 + (7 * i) % 80 for i in range(rows)]
    e.step([(i, tokens[:n], []) for i, n in enumerate(lens)])
    for k in range(3):
        got = e.step([(i, [tokens[n + k]], [0]) for i, n in enumerate(lens)])
        assert row_errors(got, want[[n + k for n in lens]]).max() < TOL["bf16"]
    model.destroy()


def _planted(window, keep, n, j, i, strength=9.0):
    """A one-layer model whose query at the token of position i matches the key of position j's token alone: token ids
    carry the match, so the same weights serve any pair of positions."""
    cfg = config([layer(2, 1, 16, 24, window, keep, ff=None, diff=0.2, scale=1.0)], width=64, vocab=40, max_positions=n + 8)
    w = weights(cfg, 21)
    rng = np.random.default_rng(22)
    w["pos"] = w["pos"] * 0.02
    ask, tell = np.zeros(64), np.zeros(64)
    ask[0], tell[1] = 8.0, 8.0                        # after the norm about 8 (the row's rms is 1)
    w["embed"][:, :2] = 0
    w["embed"][38], w["embed"][39] = ask, tell
    w["l0.norm1"][:] = 1
    w["l0.mix.q"][:] *= 0.05
    w["l0.mix.k"][:] *= 0.05
    w["l0.mix.q"][0, 0] = strength / 8                # map 1 of head 0
    w["l0.mix.k"][0, 1] = 1 / 8 * 2
    w["l0.mix.v"][:, 1] = rng.standard_normal(24)
    tokens = rng.integers(0, 38, n)
    tokens[i], tokens[j] = 38, 39
    from util import bf16_round

    return cfg, {k: bf16_round(np.asarray(v, np.float32))[1] for k, v in w.items()}, [int(t) for t in tokens]


@pytest.mark.parametrize("window,keep", [(40, 3), (64, 0), (65, 1), (130, 66)])
def test_edges_show_in_prompts_and_in_decoding(dev, window, keep):
    """The asking token's key sits just inside / outside the window, among the last kept / first dropped tokens, at tile
    borders and far away; the logits tell whether it was seen, in a whole prompt and when the asking token is decoded."""
    n, i = 180, 170
    places = sorted({p for p in (i - window + 1, i - window, i - window - 1, keep - 1, keep, 0, 63, 64, 127, 128, i - 1) if 0 <= p < i})
    for j in places:
        cfg, w, tokens = _planted(window, keep, n, j, i)
        want = reference(cfg, w, tokens[:i + 1])[i]
        blind = list(tokens)
        blind[j] = 0
        moved = np.abs(reference(cfg, w, blind[:i + 1])[i] - want).max() / np.sqrt(np.mean(want ** 2))
        if T.visible(i, j, window, keep):
            assert moved > 0.3, (j, moved)
        for dtype in ("f32", "bf16"):
            model = make(dev, cfg, w, dtype, max_slots=2)
            e = engine(model)
            whole = e.step([("whole", tokens, [i])])
            e.step([("decoded", tokens[:i - 3], [])])
            for p in range(i - 3, i):
                e.step([("decoded", [tokens[p]], [])])
            one = e.step([("decoded", [tokens[i]], [0])])
            for got in (whole, one):
                assert row_errors(got, want[None]).max() < TOL[dtype], (j, dtype)
            model.destroy()


@pytest.mark.parametrize("ff", [5, 24, 130])
def test_long_rows_split_over_k(dev, ff):
    """Wide enough that the tcgen05 GEMM splits k over CTAs, with tiles of few features: projections, GLU and residual."""
    cfg = config([layer(2, 1, 8, 16, 20, 1, ff=ff), layer(2, 2, 4, 8, 9, 0, ff=ff)], width=1100)
    w = weights(cfg, 41)
    tokens = list(np.random.default_rng(42).integers(0, cfg["vocab"], 45))
    model = make(dev, cfg, w, "bf16", max_slots=1)
    assert row_errors(engine(model).step([(0, tokens, range(45))]), reference(cfg, w, tokens)).max() < TOL["bf16"]
    model.destroy()


def test_long_decoding_crosses_windows_and_tiles(dev):
    cfg = config([layer(4, 2, 24, 32, 21, 2, ff=48), layer(4, 2, 24, 32, 100, 0, ff=48, kv_from=0)], max_positions=300)
    w = weights(cfg, 31, sharp=2.0)
    tokens = list(np.random.default_rng(32).integers(0, cfg["vocab"], 270))
    want = reference(cfg, w, tokens)
    for dtype in ("f32", "bf16"):
        model = make(dev, cfg, w, dtype, max_slots=1)
        e = engine(model)
        got = [e.step([(0, tokens[:5], range(5))])] + [e.step([(0, [t], [0])]) for t in tokens[5:]]
        assert row_errors(np.concatenate(got), want).max() < TOL[dtype] * (1 if dtype == "f32" else 1.5)
        model.destroy()


def greedy(cfg, w, prompt, n):
    m = T.Tofazen(cfg, w)
    st = m.new_state()
    lg, out, gaps = m.forward(prompt, st)[-1], [], []
    for _ in range(n):
        top = np.sort(lg)[-2:]
        gaps.append(top[1] - top[0])
        out.append(int(lg.argmax()))
        lg = m.forward(out[-1:], st)[0]
    return out, gaps


def test_greedy_generation(dev, refs):
    """``generate`` (one ragged prefill, then the replayed graph) gives the numpy model's tokens, for prompts of unequal
    lengths, one of a single token."""
    cfg, w, tokens, _ = refs["mixed"]
    prompts = [tokens[:1], tokens[5:40], tokens[2:90], tokens[10:13]]
    model = make(dev, cfg, w, "f32", max_slots=4)
    out = model.generate_greedy(prompts, 24)
    for b, p in enumerate(prompts):
        want, gaps = greedy(cfg, w, p, 24)
        assert min(gaps) > 1e-4
        assert out[b].tolist() == want
    assert np.array_equal(model.generate_greedy(prompts[1:3], 24), out[1:3])      # slots used again
    # bf16: every token is the maximum of the numpy logits up to the error of the format
    m16 = make(dev, cfg, w, "bf16", max_slots=4)
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
    vals = (0.8, 20, 0.9, 1.4)
    model = make(dev, cfg, w, "bf16", max_slots=2)
    out = model.generate(prompts, 8, tb.SamplerConfig(*vals), seed=5)
    e = engine(model)
    for b, p in enumerate(prompts):
        seq, state = list(p), 5
        lg = e.step([(b, p, [len(p) - 1])])[0]
        for t in out[b]:
            draw, state = orc.sampler_sample(lg.astype(np.float64), orc.SamplerConfig(*vals), state, past=seq)
            assert draw == t
            seq.append(draw)
            lg = e.step([(b, [draw], [0])])[0]
    model.destroy()


def test_bad_models_and_steps_are_refused(dev, refs):
    import tang_b200 as tb

    cfg, w, tokens, _ = refs["mixed"]
    v = views(w)
    del v["l1.mix.q"]
    with pytest.raises(tb.SafetensorsError, match="l1.mix.q"):
        tb.TofazenModel.from_tensors(dev, cfg, v)
    v = views(w)
    v["l0.mlp.up"] = tb.TensorView("BF16", (88, 71), np.zeros(88 * 71, np.uint16))
    with pytest.raises(tb.TangqError, match="must be"):
        tb.TofazenModel.from_tensors(dev, cfg, v)
    for kv in (1, 5, 3):                               # a layer without keys of its own, none such, itself
        bad = json.loads(json.dumps(cfg))
        bad["layers"][3]["mixer"]["kv_from"] = kv
        with pytest.raises(tb.TangqError, match="kv_from"):
            tb.TofazenModel.from_tensors(dev, bad, views(w))
    bad = json.loads(json.dumps(cfg))
    bad["layers"][1]["mixer"]["dim"] = 24
    with pytest.raises(tb.TangqError, match="shape"):
        tb.TofazenModel.from_tensors(dev, bad, views(w))
    model = make(dev, cfg, w, "bf16", max_slots=2, max_seq=32)
    e = engine(model)
    with pytest.raises(tb.TangqError, match="positions"):
        e.step([(0, tokens[:33], [])])
    # a position behind the cache that only the device sees is skipped and reported, and the model goes on
    lg = dev.alloc(2 * cfg["vocab"])
    model.decode(dev.upload(np.array([1, 2], np.int32), tb.I32), dev.upload(np.array([32, 0], np.int32), tb.I32), 2, 32, lg)
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
    tokens = [int(t) for t in tokens]
    text = "\n".join(json.dumps(s, default=int) for s in steps) + "\n"
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
