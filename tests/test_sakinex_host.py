"""Host side of the Sakinex family, without a GPU: configuration, runs of layers, tensor list, slots, and the numpy implementation's
own consistency (prompt in one piece against token by token, hand-computed cases)."""
import json
import math

import numpy as np
import pytest

import sakinex_oracle as X
from sakinex_util import CONFIGS, config, layer, moe, reference, save, weights


@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_numpy_model_does_not_depend_on_the_cut(name):
    cfg = CONFIGS[name]
    w = weights(cfg, 3)
    tokens = list(np.random.default_rng(2).integers(0, cfg["vocab"], 41))
    whole = reference(cfg, w, tokens)
    m = X.Sakinex(cfg, w)
    st = m.new_state()
    cut = np.concatenate([m.forward(tokens[a:b], st) for a, b in ((0, 1), (1, 3), (3, 20), (20, 41))])
    assert np.abs(whole - cut).max() < 1e-10


def test_a_loop_equals_its_layers_written_out():
    """A pass beyond the first equals further layers with copies of the weights that start with the embedding output added."""
    layers = [layer(2, 1, 8, 6, 5, 2, 12, moe(3, 2, 10, 6)), layer(2, 2, 8, 4, 9, 3, 8)]
    looped = config(layers, width=40, vocab=30, loop=(0, 2, 2))
    w = weights(looped, 5)
    copied = {**w, **{f"l{int(k[1]) + 2}{k[2:]}": v for k, v in w.items() if k[0] == "l" and k[1].isdigit()}}
    tokens = list(np.random.default_rng(6).integers(0, 30, 25))
    out = X.Sakinex(config(layers * 2, width=40, vocab=30), copied)
    out.runs = [(0, False), (1, False), (2, True), (3, False)]
    assert np.array_equal(reference(looped, w, tokens), out.forward(tokens, out.new_state()))
    assert np.abs(reference(looped, w, tokens) - reference(config(layers * 2, width=40, vocab=30), copied, tokens)).max() > 0.1


def test_numpy_mechanisms_by_hand():
    assert X.seen_tokens(9, 3) == [7, 8, 9] and X.seen_tokens(1, 3) == [0, 1]
    # blocks of 4 before a window of 3 at position 9: the window starts at 7, so it has passed 0..3 and still touches 4..7
    assert X.seen_blocks(9, 3, 4) == [0] and X.seen_blocks(10, 3, 4) == [0, 1] and X.seen_blocks(6, 3, 4) == [0] and X.seen_blocks(5, 3, 4) == []
    assert X.seen_blocks(2, 1, 1) == [0, 1]
    q, k, v = np.array([2.0]), np.array([[1.0], [3.0], [0.5]]), np.array([[1.0], [2.0], [5.0]])
    e = np.exp([0.5 * 2 * 2.0, 0.5 * 2 * 0.5])         # the block's mean key, then the token in the window
    assert X.one_query(q, k, v, 2, 0.5, 1, 2)[0] == pytest.approx((e[0] * 1.5 + e[1] * 5.0) / e.sum())
    y, last = X.conv(np.array([[1.0], [2.0], [3.0]]), np.array([[0.5, 10.0]]), np.array([[4.0]]))
    assert y[:, 0] == pytest.approx([12.0, 20.5, 31.0]) and last[0, 0] == 3.0
    y, last = X.conv(np.array([[1.0]]), np.array([[7.0, 0.5, 10.0]]), np.array([[4.0], [6.0]]))
    assert y[0, 0] == pytest.approx(7 * 4 + 3 + 10) and last[:, 0].tolist() == [6.0, 1.0]
    s, S = X.min_gru(np.array([[0.0], [math.log(3)]]), np.array([[2.0], [-math.log(4)]]), np.array([1.0]))
    assert s[:, 0] == pytest.approx([0.5 + 0.5 * 2.5, 0.25 * 1.75 + 0.75 * 0.2]) and S[0] == s[1, 0]
    e, p = X.choose(np.log(np.array([0.5, 0.1, 0.3, 0.1])), 2)
    assert e == [0, 2] and p == pytest.approx([0.5 / 0.8, 0.3 / 0.8])
    assert X.gated(np.array([1.0]), np.array([3.0]))[0] == pytest.approx(3.0 / (1 + math.exp(-1)))
    assert X.rotate(np.array([1.0, 2.0, 0.0, 0.0, 7.0]), 1, np.array([1.0, 0.1]), 2.0) == pytest.approx(
        [2 * math.cos(1), 4 * math.cos(0.1), 2 * math.sin(1), 4 * math.sin(0.1), 7.0])
    assert X.Sakinex(config([None] * 5, loop=(1, 3, 3)), {}).runs == [(0, False), (1, False), (2, False), (1, True), (2, False), (1, True), (2, False), (3, False), (4, False)]


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_expert_choices_of_the_test_models_are_not_close_calls(name, monkeypatch):
    cfg, gaps, choose = CONFIGS[name], [], X.choose

    def watch(z, top):
        e, p = choose(z, top)
        gaps.extend(z[e[-1]] - z[x] for x in range(len(z)) if x not in e)
        return e, p

    monkeypatch.setattr(X, "choose", watch)
    tokens = np.random.default_rng(12).integers(0, cfg["vocab"], 150)
    reference(cfg, weights(cfg, 3), tokens)
    assert min(gaps) > 0.1


def test_the_two_restatements_of_yarn_agree():
    import dotanex_oracle as D

    for dims, base, scaling in ((8, 10000.0, None), (64, 500000.0, (8.0, 512, 32.0, 1.0)), (10, 50.0, (2.0, 4096, 4.0, 2.0))):
        rot = {"dims": dims, "base": base, "scaling": None if scaling is None else dict(zip(("factor", "original", "fast", "slow"), scaling))}
        assert np.allclose(X.frequencies(rot)[0], D.yarn_frequencies(rot)[0]) and X.frequencies(rot)[1] == pytest.approx(D.yarn_frequencies(rot)[1])


def test_config_reads_every_field():
    from tang_b200 import SakinexConfig, registry
    from tang_b200.sakinex import Run

    c = SakinexConfig.from_dict(CONFIGS["mixed"])
    assert (c.width, c.vocab, c.eps, c.residual_mult, c.taps, len(c.layers), c.loop) == (72, 101, 1e-5, 0.6, 3, 4, (1, 3, 3))
    a, b, l, last = c.layers
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.window, a.pool, a.state_width, a.taps, a.scale, a.left_scale, a.right_scale) == (
        6, 2, 20, 24, 17, 4, 50, 3, 1.5 * 20 ** -0.5, 0.7, 1.2)
    assert (a.rot.dims, a.rot.base, a.rot.factor, a.rot.original, a.rot.fast, a.rot.slow) == (20, 10000.0, 4.0, 64, 16.0, 1.0)
    assert (a.mlp.experts, a.mlp.top, a.mlp.ff, a.mlp.shared_ff) == (5, 2, 24, 40) and b.mlp.shared_ff == 0 and l.mlp.experts == 0
    assert last.rot.factor == 0 and last.rot.dims == 20 and l.rot.dims == 8
    assert c.runs() == [Run(0, -1, False), Run(1, -1, False), Run(2, -1, False), Run(1, 1, True), Run(2, 2, False), Run(1, 1, True), Run(2, 2, False), Run(3, -1, False)]
    assert [(r.layer, r.add_embedding) for r in c.runs()] == X.Sakinex(CONFIGS["mixed"], {}).runs
    assert registry.resolve(CONFIGS["mixed"])[0] is SakinexConfig
    # caches of eight runs with their pooled rows; states of the recurrences and of the convolutions
    rows = 2 * 48 * 1.25 + 3 * 3 * 32 * (17 / 16) + 3 * 56 * 1.125 + 2 * 48 * (4 / 3)
    assert rows * 2 <= c.cache_bytes_per_token(1) <= rows * 2 + 2
    heads = [128 + 48 + 48, 80 + 80 + 32, 64 + 16 + 48, 128 + 48 + 48]
    assert c.state_bytes(1) == 4 * (50 + 3 * 36 + 3 * 64 + 24) + 2 * (2 * heads[0] + 3 * 2 * heads[1] + 3 * 3 * heads[2] + heads[3] + 2 * 72 * (2 + 6 + 3 + 2))
    assert c.bytes_per_slot(0, 10) == 10 * c.cache_bytes_per_token(0) + c.state_bytes(0)


def test_parts_of_a_model_may_be_absent():
    from tang_b200 import SakinexConfig
    from tang_b200.sakinex import tensor_names
    from tang_b200.stepmodel import NO_WINDOW

    c = json.loads(json.dumps(config([layer(2, 1, 8, 6, 5, 2, 12, moe(3, 2, 10, 6)), layer(2, 2, 8, 4, 9, 3, 8)])))
    left = c["layers"][1]["mixer"]["left"]
    del left["conv"], left["mask"], left["rot"]
    c["layers"][0]["mlp"]["shared"] = None
    cfg = SakinexConfig.from_dict(c)
    l = cfg.layers[1]
    assert (l.window, l.pool, l.taps, l.rot.dims) == (NO_WINDOW, 0, 0, 0) and cfg.layers[0].mlp.shared_ff == 0 and len(cfg.runs()) == 2
    names = [n for n, _, _, _ in tensor_names(cfg)]
    assert not any("shared" in n or n.startswith(("l1.mlp", "l1.norm2", "l1.canon2", "l1.mix.left.q.conv")) for n in names) and "l0.mix.left.q.conv" in names


def test_config_rejects_what_it_does_not_know():
    from tang_b200 import SakinexConfig
    from tang_b200.stepmodel import ConfigError

    def broken(change):
        c = json.loads(json.dumps(CONFIGS["mixed"]))
        change(c)
        return c

    for change, what in ((lambda c: c["layers"][2].update(type="scan"), "scan"), (lambda c: c["layers"][1]["mlp"].update(kind="dense"), "dense"),
                         (lambda c: c["loop"].update(stop=5), "loop"), (lambda c: c["loop"].update(times=0), "loop"), (lambda c: c["canon"].update(taps=0), "taps"),
                         (lambda c: c["layers"][0]["mixer"]["left"].pop("vdim"), "vdim"), (lambda c: c["layers"][0]["mixer"].pop("right_scale"), "right_scale"),
                         (lambda c: c.pop("residual_mult"), "residual_mult"), (lambda c: c.pop("norm"), "norm"),
                         (lambda c: c["layers"][0]["mixer"]["left"]["rot"]["scaling"].update(factor=0), "stretched")):
        with pytest.raises(ConfigError, match=what):
            SakinexConfig.from_dict(broken(change))


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_tensor_names_are_the_checkpoints(name):
    from tang_b200 import SakinexConfig
    from tang_b200.sakinex import tensor_names

    names = [n for n, _, _, _ in tensor_names(SakinexConfig.from_dict(CONFIGS[name]))]
    assert len(names) == len(set(names)) and set(names) == set(weights(CONFIGS[name], 0))


def test_slots_follow_the_cache_budget(tmp_path, monkeypatch):
    """Without a largest position the default holds, and slots are cut to the budget, states included."""
    from tang_b200 import SakinexConfig, registry

    cfg = CONFIGS["odd"]
    w = weights(cfg, 5)
    save(tmp_path, cfg, w)
    got = {}

    class Fake:
        @classmethod
        def from_tensors(cls, dev, config, tensors, dtype, max_slots, max_seq):
            got.update(slots=max_slots, seq=max_seq, names=set(tensors))

    monkeypatch.setitem(registry.ARCHITECTURES, "Sakinex", (SakinexConfig, Fake))
    registry.load_model(None, str(tmp_path))
    assert got["seq"] == registry.DEFAULT_MAX_SEQ and got["slots"] == 64 and got["names"] == set(w)
    per = SakinexConfig.from_dict(cfg).bytes_per_slot(1, 100)
    registry.load_model(None, str(tmp_path), max_seq=100, cache_budget=5 * per + 1)
    assert got["seq"] == 100 and got["slots"] == 5
