"""Host side of the Tofazen family, without a GPU: configuration, tensor list, batching, slots, command line, and the
numpy implementation's own consistency (prompt in one piece against token by token)."""
import math
import os
import subprocess
import sys

import numpy as np
import pytest

import tofazen_oracle as T
from tofazen_util import CONFIGS, config, layer, reference, save, weights

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def test_numpy_model_does_not_depend_on_the_cut():
    cfg = CONFIGS["mixed"]
    w = weights(cfg, 1)
    tokens = list(np.random.default_rng(2).integers(0, cfg["vocab"], 41))
    whole = reference(cfg, w, tokens)
    m = T.Tofazen(cfg, w)
    st = m.new_state()
    cut = np.concatenate([m.forward(tokens[a:b], st) for a, b in ((0, 1), (1, 3), (3, 20), (20, 41))])
    assert np.abs(whole - cut).max() < 1e-12


def test_numpy_mask_and_glu():
    assert [j for j in range(12) if T.visible(9, j, 3, 2)] == [0, 1, 7, 8, 9]
    assert [j for j in range(12) if T.visible(2, j, 1, 0)] == [2]
    assert T.clamped_glu(np.array([50.0]), np.array([-50.0]), 2.0)[0] == pytest.approx(2.0 / (1 + math.exp(-1.702 * 2)) * -1.0)


def test_config_reads_every_field():
    from tang_b200 import TofazenConfig, registry

    c = TofazenConfig.from_dict(CONFIGS["mixed"])
    assert (c.width, c.vocab, c.max_positions, c.eps, c.residual_mult) == (72, 101, 400, 1e-5, 0.9)
    a, b = c.layers[0], c.layers[1]
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.window, a.keep_first, a.ff, a.limit, a.kv_from, a.diff) == (6, 2, 20, 40, 17, 3, 88, 1.5, None, 0.4)
    assert (b.kv_from, b.window, b.keep_first, b.diff) == (0, 33, 0, 0.1) and c.layers[2].ff == 0 and c.layers[3].scale == 0.4
    assert registry.resolve(CONFIGS["mixed"])[0] is TofazenConfig
    # one cached row: layers 0 and 2 project keys and values, head sizes padded to 8 values
    assert c.cache_bytes_per_token(1) == 2 * (2 * (2 * 24 + 40) + 3 * (2 * 24 + 16))


def test_config_rejects_what_it_does_not_know():
    from tang_b200 import TofazenConfig, registry
    from tang_b200.tofazen import ConfigError

    with pytest.raises(registry.UnknownArchitecture):
        registry.resolve({"architecture": "Nothing"})
    bad = config([layer(2, 1, 8, 8, 4, 0, ff=8)])
    bad["layers"][0]["type"] = "recurrent"
    with pytest.raises(ConfigError, match="recurrent"):
        TofazenConfig.from_dict(bad)
    bad = config([layer(2, 1, 8, 8, 4, 0, ff=8)])
    bad["layers"][0]["mlp"]["kind"] = "routed"
    with pytest.raises(ConfigError, match="routed"):
        TofazenConfig.from_dict(bad)
    bad = config([layer(2, 1, 8, 8, 4, 0)])
    del bad["residual_mult"]
    with pytest.raises(ConfigError, match="residual_mult"):
        TofazenConfig.from_dict(bad)


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_tensor_names_are_the_checkpoints(name):
    from tang_b200 import TofazenConfig
    from tang_b200.tofazen import tensor_names

    cfg = CONFIGS[name]
    names = [n for n, _, _ in tensor_names(TofazenConfig.from_dict(cfg))]
    assert len(names) == len(set(names))
    assert set(names) == {n for n in weights(cfg, 0) if n.split(".")[-1] not in ("lq1", "lk1", "lq2", "lk2")}


def test_map_balance():
    from tang_b200 import TofazenConfig
    from tang_b200.tofazen import map_balance

    cfg = CONFIGS["odd"]
    w = weights(cfg, 3)
    v = [w[f"l0.mix.{n}"] for n in ("lq1", "lk1", "lq2", "lk2")]
    assert map_balance(TofazenConfig.from_dict(cfg).layers[0], *v) == pytest.approx(T.lam(*(x.astype(np.float64) for x in v), 0.4), rel=1e-12)


@pytest.mark.parametrize("max_rows", [1, 2, 3, 7, 100])
def test_portions_cover_every_token_once_in_order(max_rows):
    from tang_b200.engine import portions

    lengths = [5, 1, 12, 2]
    seen = [0] * len(lengths)
    for batch in portions(lengths, max_rows):
        assert 0 < sum(n for _, _, n in batch) <= max_rows and len({s for s, _, _ in batch}) == len(batch)
        for s, at, n in batch:
            assert at == seen[s] and n > 0
            seen[s] += n
    assert seen == lengths


def test_slot_pool_reuses_slots():
    from tang_b200 import TangqError
    from tang_b200.engine import SlotPool

    p = SlotPool(2)
    a, b = p.open("a"), p.open("b")
    assert {a, b} == {0, 1}
    with pytest.raises(TangqError):
        p.open("c")
    with pytest.raises(TangqError):
        p.open("a")
    p.length["a"] = 9
    p.close("a")
    assert p.open("c") == a and p.length["c"] == 0


class _FakeDevice:
    """Records what a step is given; 'device memory' is a numpy array per buffer."""

    def __init__(self):
        self.mem = {}

    def alloc(self, n, dtype):
        from tang_b200 import Buffer

        ptr = (len(self.mem) + 1) << 32
        self.mem[ptr] = np.zeros(n, np.int32 if dtype == 5 else np.float32)
        return Buffer(self, ptr, n, dtype, owns=False)

    def _at(self, buf):
        base = max(p for p in self.mem if p <= buf.ptr)
        off = (buf.ptr - base) // 4
        return self.mem[base][off:off + buf.n]

    def upload_into(self, buf, data):
        self._at(buf)[:len(data)] = data

    def download(self, buf):
        return self._at(buf).copy()

    def sync(self):
        pass


class _FakeModel:
    """Logits of a row: [token, position, slot]."""

    max_slots, max_seq = 3, 64

    class cfg:
        vocab = 3

    def __init__(self):
        self.dev, self.steps = _FakeDevice(), []

    def step(self, tok, rows, seq_rows, starts, slots, n_seqs, max_q, max_len, logit_rows, n_logits, logits):
        g = lambda b: self.dev._at(b)
        cu = np.arange(n_seqs + 1) if seq_rows is None else g(seq_rows)
        per_row = [(g(tok)[r], g(starts)[b] + r - cu[b], g(slots)[b]) for b in range(n_seqs) for r in range(cu[b], cu[b + 1])]
        assert len(per_row) == rows and max(p for _, p, _ in per_row) < max_len and max(np.diff(cu)) == max_q
        self.steps.append(rows)
        if n_logits:
            g(logits)[:n_logits * 3] = np.concatenate([per_row[r] for r in g(logit_rows)])


@pytest.mark.parametrize("max_rows", [2, 5, 64])
def test_engine_returns_wanted_rows_in_the_callers_order(max_rows):
    from tang_b200 import Engine

    m = _FakeModel()
    e = Engine(m, max_rows=max_rows)
    got = e.step([("a", [2, 1, 0, 2, 1], [4, 0]), ("b", [1], []), ("c", [0, 2, 2], [1, 2])])
    sa, sc = e.pool.slot["a"], e.pool.slot["c"]
    assert got.tolist() == [[1, 4, sa], [2, 0, sa], [2, 1, sc], [2, 2, sc]]
    assert all(s <= max_rows for s in m.steps) and sum(m.steps) == 9
    got = e.step([("c", [1], [0]), ("a", [0], [0])])
    assert got.tolist() == [[1, 3, sc], [0, 5, sa]]
    sb = e.pool.slot["b"]
    e.close("b")
    assert e.step([("d", [1, 1], [1])]).tolist() == [[1, 1, sb]]
    assert e.step([("d", [0], [])]).shape == (0, 3)


def test_engine_rejects_bad_steps():
    from tang_b200 import Engine, TangqError

    e = Engine(_FakeModel())
    for bad in ([("a", [3], [0])], [("a", [], [])], [("a", [1], [1])], [("a", [1], []), ("a", [1], [])], [("a", [1] * 65, [])]):
        with pytest.raises(TangqError):
            e.step(bad)
    assert not e.pool.slot


def test_checkpoint_round_trip(tmp_path):
    from tang_b200 import read_safetensors, registry

    cfg = CONFIGS["odd"]
    w = weights(cfg, 5)
    save(tmp_path, cfg, w)
    assert registry.read_config(str(tmp_path)) == cfg
    t = read_safetensors(tmp_path / "model.safetensors")
    assert all(np.array_equal(t[k].to_f32().reshape(v.shape), v) for k, v in w.items())


def test_command_line_help_and_no_gpu(tmp_path):
    import torch

    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--help"], capture_output=True, text=True)
    assert r.returncode == 0 and "--max-tokens" in r.stdout
    r = subprocess.run([sys.executable, "-m", "tang_b200"], capture_output=True, text=True, cwd=ROOT)
    assert r.returncode == 2 and "generate" in r.stderr
    if torch.cuda.is_available():
        pytest.skip("a GPU is present")
    from tang_b200 import _build

    _build.build_library()
    save(tmp_path, CONFIGS["odd"], weights(CONFIGS["odd"], 5))
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", "bfloat16", "--out", str(tmp_path),
                        "--max-tokens", "64"], input="", capture_output=True, text=True)
    assert r.returncode not in (0, 3) and "no CPU fallback" in r.stderr
