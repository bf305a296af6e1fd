"""The Dotanex family on the device, whole model: loading, prompts, portions, decoding, ragged batches, slots and states used
again, generation and the trace runner, against the numpy implementation in 32-bit and in bf16."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import dotanex_oracle as X
from dotanex_util import CONFIGS, TOL, again, attn, config, dense, latent, lightning, moe, reference, row_errors, save, views, weights
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

    return tb.DotanexModel.from_tensors(dev, cfg, views(w), tb.F32 if dtype == "f32" else tb.BF16, **kw)


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
def test_stream_after_every_layer(dev, refs, name, dtype):
    import tang_b200 as tb

    cfg, w, tokens, _ = refs[name]
    model = make(dev, cfg, w, dtype, max_slots=1, max_seq=160)
    trace = []
    m = X.Dotanex(cfg, w)
    m.forward(tokens[:79], m.new_state(), trace)
    buf = dev.alloc(len(trace) * 79 * cfg["width"], tb.F32)
    model.trace(buf)
    engine(model).step([(0, tokens[:79], [])])
    for i, (g, x) in enumerate(zip(buf.to_vec().reshape(len(trace), 79, -1), trace)):
        assert row_errors(g, x).max() < TOL[dtype], i
    model.trace(None)
    model.destroy()


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("name", ["mixed", "aligned"])
def test_ragged_batches_equal_each_alone_and_slots_are_reused(dev, refs, name, dtype):
    """Unequal prompts start together, others join while they decode, some end early; freed slots (caches and states) serve new
    requests."""
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
    """Enough rows for many jobs per expert and for row tiles of the widest size."""
    cfg, w, tokens, want = refs["aligned"]
    model = make(dev, cfg, w, "bf16", max_slots=20, max_seq=160)
    got = engine(model).step([(i, tokens[:150 - i], [149 - i, 3]) for i in range(20)])
    assert row_errors(got, np.concatenate([want[[149 - i, 3]] for i in range(20)])).max() < TOL["bf16"]
    model.destroy()


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_expansion_in_parts(dev, refs, dtype):
    """Keys and values of the latent layers expanded for one or a few sequences at a time, among sequences that bring one row."""
    cfg, w, tokens, want = refs["mixed"]
    for expand_bytes in (1, 200_000):
        model = make(dev, cfg, w, dtype, max_slots=6, max_seq=120, expand_bytes=expand_bytes)
        e = engine(model)
        at, got = {r: 0 for r in range(6)}, {r: [] for r in range(6)}
        for counts in ((70, 1, 33, 5, 64, 1), (1, 40, 2, 1, 9, 30), (3, 1, 1, 60, 20, 1)):
            out, k = e.step([(r, tokens[at[r]:at[r] + n], range(n)) for r, n in enumerate(counts)]), 0
            for r, n in enumerate(counts):
                got[r].append(out[k:k + n])
                k, at[r] = k + n, at[r] + n
        for r in range(6):
            assert row_errors(np.concatenate(got[r]), want[:at[r]]).max() < TOL[dtype], (expand_bytes, r)
        model.destroy()


def _planted(mixer, n, j, i):
    """A one-layer model in which the token at position i looks for what the token at position j left; token ids carry the
    match, so that the same weights serve any pair of positions."""
    cfg = config([mixer], width=64, vocab=40)
    w = weights(cfg, 21)
    rng = np.random.default_rng(22)
    m = mixer["mixer"]
    w["embed"][:, :2] = 0
    w["embed"][38], w["embed"][39] = 0, 0
    w["embed"][38, 0], w["embed"][39, 1] = 8.0, 8.0
    w["l0.norm1"][:] = 1
    w["l0.hc1.out"][:] = 2.0
    mix = lambda name: w["l0.mix." + name]
    d = m["dim"] - 1                                  # not a rotated dimension
    if mixer["type"] == "latent_attention":
        D, R = m["dim"], m["rot_dim"]
        for name in ("dq", "dkv", "uq", "uk"):
            mix(name)[:] *= 0.05
        mix("dq")[0], mix("dkv")[0] = 0, 0
        mix("dq")[0, 0], mix("dkv")[0, 1] = 2.0, 2.0
        for h in range(m["heads"]):
            mix("uq")[h * (D + R) + d, 0] = 2.0
            mix("uk")[h * D + d] = 0
            mix("uk")[h * D + d, 0] = 2.0
    else:
        for name in [x for x in ("q", "k", "v") if f"l0.mix.{x}" in w]:
            mix(name)[:] *= 0.05
        mix("q")[d, 0] = 2.0
        mix("k")[:, 1] += rng.standard_normal(len(mix("k"))) * 0.1
        mix("k")[d, :] = 0
        mix("k")[d, 1] = 2.0
        if "l0.mix.v" in w:
            mix("v")[:, 1] = rng.standard_normal(len(mix("v"))) * 3
    tokens = rng.integers(0, 38, n)
    tokens[i], tokens[j] = 38, 39
    return cfg, {k: bf16_round(np.asarray(v, np.float32))[1] for k, v in w.items()}, [int(t) for t in tokens]


def _check_planted(dev, cfg, w, tokens, i, j, seen):
    want = reference(cfg, w, tokens[:i + 1])[i]
    blind = list(tokens)
    blind[j] = 0
    moved = row_errors(reference(cfg, w, blind[:i + 1])[i][None], want[None])[0]
    assert not seen or moved > 0.2, (j, moved)
    for dtype in ("f32", "bf16"):
        model = make(dev, cfg, w, dtype, max_slots=3, max_seq=len(tokens))
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


@pytest.mark.parametrize("window", [40, 64, 65, 130])
def test_window_edges_show_in_prompts_and_in_decoding(dev, window):
    n, i = 180, 170
    mixer = attn(2, 1, 16, window, rot=4, scale=1.0)
    for j in sorted({p for p in (i - window + 1, i - window, i - window - 1, 0, 63, 64, 127, 128, i - 1) if 0 <= p < i}):
        cfg, w, tokens = _planted(mixer, n, j, i)
        _check_planted(dev, cfg, w, tokens, i, j, X.visible(i, j, window))


@pytest.mark.parametrize("heads,kv_rank", [(2, 24), (20, 300)])
def test_latents_are_found_anywhere(dev, heads, kv_rank):
    """The first tokens, both sides of the decode kernel's tiles, the neighbour."""
    n, i = 330, 320
    for j in (0, 1, 63, 64, 191, 192, 318, 319):
        cfg, w, tokens = _planted(latent(heads, 12, 4, 10, 16, kv_rank, scale=0.3), n, j, i)
        _check_planted(dev, cfg, w, tokens, i, j, True)


@pytest.mark.parametrize("dim,vdim", [(20, 24), (64, 64)])
def test_a_state_reaches_far_back(dev, dim, vdim):
    n, i = 200, 190
    for j in (0, 15, 16, 63, 64, 127, 128, 188):
        cfg, w, tokens = _planted(lightning(2, dim, vdim, decay=[1.0, 0.999]), n, j, i)
        _check_planted(dev, cfg, w, tokens, i, j, True)


def test_a_sink_takes_its_share(dev):
    """One head whose sink outweighs every key, one whose sink is far below: the first leaves the stream almost alone."""
    cfg = config([attn(2, 1, 16, 30)], width=64, vocab=40)
    w = weights(cfg, 23)
    tokens = [int(t) for t in np.random.default_rng(24).integers(0, 40, 90)]
    plain = reference(cfg, w, tokens)
    for sinks, least in (([30.0, -30.0], 0.1), ([3.0, 4.0], 0.03)):
        w["l0.mix.sink"] = bf16_round(np.array(sinks, np.float32))[1]
        want = reference(cfg, w, tokens)
        assert row_errors(want, plain).mean() > least
        for dtype in ("f32", "bf16"):
            model = make(dev, cfg, w, dtype, max_slots=1, max_seq=90)
            e = engine(model)
            got = np.concatenate([e.step([(0, tokens[:50], range(50))])] + [e.step([(0, [t], [0])]) for t in tokens[50:]])
            assert row_errors(got, want).max() < TOL[dtype]
            model.destroy()


def test_long_decoding_crosses_windows_tiles_and_chunks(dev):
    cfg = config([attn(4, 2, 24, 21, moe(3, 1, 1, 24, 16)), lightning(2, 32, 32, moe(4, 2, 2, 24, 40)), latent(4, 16, 8, 16, 24, 40, dense(40)), attn(4, 2, 24, 100)])
    w = weights(cfg, 31)
    tokens = [int(t) for t in np.random.default_rng(32).integers(0, cfg["vocab"], 270)]
    want = reference(cfg, w, tokens)
    for dtype in ("f32", "bf16"):
        model = make(dev, cfg, w, dtype, max_slots=1, max_seq=270)
        e = engine(model)
        got = [e.step([(0, tokens[:5], range(5))])] + [e.step([(0, [t], [0])]) for t in tokens[5:]]
        assert row_errors(np.concatenate(got), want).max() < TOL[dtype]
        model.destroy()


@pytest.mark.parametrize("layers,width,vocab,streams", [
    ([attn(1, 1, 2, 1, moe(1, 0, 1, 1, 1), rot=2), lightning(1, 1, 1, moe(2, 1, 2, 3, 2)), latent(1, 1, 2, 1, 1, 1, dense(1))], 8, 5, 2),
    ([lightning(1, 16, 16, None), lightning(1, 8, 40, moe(16, 8, 6, 8, 20)), latent(33, 8, 4, 8, 16, 16, None, scaling=(1.0, 32, 4.0, 1.0))], 40, 1000, 7),
    ([attn(3, 1, 8, 3, moe(4, 2, 4, 130, 5), rot=8, scaling=(1.0, 1.0, 4.0, 32)), attn(130, 2, 8, 9, None, rot=2), latent(2, 200, 64, 200, 24, 512)], 136, 30, 1)])
def test_other_sizes(dev, layers, width, vocab, streams):
    cfg = config(layers, width=width, vocab=vocab, streams=streams)
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


def test_long_rows_split_over_k(dev):
    """Wide enough that the router's and the mixers' products are split over k."""
    cfg = config([attn(2, 1, 16, 20, moe(20, 4, 3, 40, 200)), lightning(2, 16, 32, moe(3, 1, 1, 24, 24)), latent(2, 16, 8, 16, 600, 24, dense(700))], width=1100, vocab=50)
    w = weights(cfg, 41)
    tokens = [int(t) for t in np.random.default_rng(42).integers(0, 50, 90)]
    model = make(dev, cfg, w, "bf16", max_slots=1, max_seq=90)
    assert row_errors(engine(model).step([(0, tokens, range(90))]), reference(cfg, w, tokens)).max() < TOL["bf16"]
    model.destroy()


def greedy(cfg, w, prompt, n):
    m = X.Dotanex(cfg, w)
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
    for gone in ("l1.mix.dq.norm", "l0.mlp.e4.up", "l2.hc1.mix", "l0.mlp.correction", "l0.mlp.shared.down", "head"):
        v = views(w)
        del v[gone]
        with pytest.raises(tb.SafetensorsError, match=gone):
            tb.DotanexModel.from_tensors(dev, cfg, v)
    for name, shape in (("l0.mlp.e1.up", (24, 71)), ("l1.mix.uk", (36, 27)), ("l0.mix.q.norm", (19,)), ("l1.hc2.mix", (3, 2)), ("l2.mix.norm", (119,))):
        v = views(w)
        v[name] = tb.TensorView("BF16", shape, np.zeros(int(np.prod(shape)), np.uint16))
        with pytest.raises(tb.TangqError, match="must be"):
            tb.DotanexModel.from_tensors(dev, cfg, v)
    bad = json.loads(json.dumps(cfg))
    bad["layers"][0]["mlp"]["router"]["top"] = bad["layers"][7]["mlp"]["router"]["top"] = 9
    with pytest.raises(tb.TangqError, match="experts"):
        tb.DotanexModel.from_tensors(dev, bad, views(w))
    bad = json.loads(json.dumps(cfg))
    bad["layers"][0]["mixer"]["rot"]["dims"] = bad["layers"][7]["mixer"]["rot"]["dims"] = 7
    with pytest.raises(tb.TangqError, match="rotation"):
        tb.DotanexModel.from_tensors(dev, bad, views(w))
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
