"""Host side of the Dotanex family, without a GPU: configuration, tensor list, slots, frequencies, and the numpy
implementation's own consistency (prompt in one piece against token by token, hand-computed cases)."""
import ctypes as C
import json
import math

import numpy as np
import pytest

import dotanex_oracle as X
from dotanex_util import CONFIGS, again, attn, config, dense, latent, lightning, moe, reference, save, weights


def test_numpy_model_does_not_depend_on_the_cut():
    cfg = CONFIGS["mixed"]
    w = weights(cfg, 3)
    tokens = list(np.random.default_rng(2).integers(0, cfg["vocab"], 41))
    whole = reference(cfg, w, tokens)
    m = X.Dotanex(cfg, w)
    st = m.new_state()
    cut = np.concatenate([m.forward(tokens[a:b], st) for a, b in ((0, 1), (1, 3), (3, 20), (20, 41))])
    assert np.abs(whole - cut).max() < 1e-10


def test_shared_weights_keep_states_of_their_own():
    """A layer that repeats another's weights equals a layer with a copy of them."""
    layers = [latent(2, 8, 4, 6, 10, 12, dense(20)), lightning(2, 8, 8, dense(16)), attn(2, 1, 8, 5, None)]
    twice = config(layers + [again(layers, j) for j in range(3)], width=40, vocab=30)
    w = weights(twice, 5)
    copied = {**w, **{f"l{int(k[1]) + 3}{k[2:]}": v for k, v in w.items() if k[0] == "l" and k[1].isdigit()}}
    tokens = list(np.random.default_rng(6).integers(0, 30, 25))
    assert np.array_equal(reference(twice, w, tokens), reference(config(layers * 2, width=40, vocab=30), copied, tokens))


def test_numpy_mechanisms_by_hand():
    assert [j for j in range(12) if X.visible(9, j, 3)] == [7, 8, 9] and X.visible(9, 0, None) and not X.visible(3, 4, None)
    # one key beside a sink: weight e^s / (e^sink + e^s)
    q, k, v = np.array([2.0, 0.0]), np.array([[3.0, 1.0]]), np.array([[5.0]])
    assert X.one_query(q, k, v, 0, 0.5, 1, 1.0)[0] == pytest.approx(5.0 * math.exp(3) / (math.exp(1) + math.exp(3)))
    assert X.one_query(q, k, v, 0, 0.5, None, None)[0] == 5.0
    o, S = X.lightning(np.array([[1.0, 1.0], [1.0, 2.0]]), np.array([[1.0, 2.0], [0.5, 0.0]]), np.array([[3.0], [4.0]]), 0.5, np.zeros((2, 1)))
    assert o[0, 0] == pytest.approx(9.0) and S[:, 0] == pytest.approx([0.5 * 3 + 0.5 * 4, 0.5 * 6]) and o[1, 0] == pytest.approx(3.5 + 6.0)
    # the correction brings expert 3 in; its weight is its own score all the same
    z = np.log(np.array([0.5, 0.3, 0.15, 0.05]))
    e, s = X.choose(z, np.array([0.0, 0.0, 0.0, 1.0]), 2)
    assert e == [3, 0] and s == pytest.approx([0.05 / 0.55, 0.5 / 0.55])
    assert X.clamped_gated(np.array([50.0]), np.array([-50.0]), 2.0)[0] == pytest.approx(2.0 / (1 + math.exp(-1.702 * 2)) * -1.0)
    assert X.gated(np.array([1.0]), np.array([3.0]))[0] == pytest.approx(3.0 / (1 + math.exp(-1)))
    assert X.rotate_halves(np.array([1.0, 2.0, 0.0, 0.0, 7.0]), 1, np.array([1.0, 0.1])) == pytest.approx([math.cos(1), 2 * math.cos(0.1), math.sin(1), 2 * math.sin(0.1), 7.0])
    assert X.rotate_neighbours(np.array([1.0, 0.0, 2.0, 0.0, 7.0]), 1, np.array([1.0, 0.1]), 2.0) == pytest.approx(
        [2 * math.cos(1), 2 * math.sin(1), 4 * math.cos(0.1), 4 * math.sin(0.1), 7.0])
    xs = np.array([[[1.0]], [[10.0]]])
    assert X.write_streams(xs, np.array([[1.0, 2.0], [3.0, 4.0]]), np.array([0.5, -1.0]), np.array([[100.0]])).reshape(-1) == pytest.approx([1 + 30 + 50, 2 + 40 - 100])
    assert X.read_streams(xs, np.array([2.0, 0.5]))[0, 0] == pytest.approx(7.0)
    f, _ = X.banded_frequencies({"dims": 6, "base": 1000.0, "scaling": {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 100.0}})
    wave = 2 * math.pi * 10
    s = (100 / wave - 1) / 3
    assert f == pytest.approx([1.0, (1 - s) * 0.1 / 4 + s * 0.1, 0.01 / 4])


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_expert_choices_of_the_test_models_are_not_close_calls(name, monkeypatch):
    cfg, gaps, choose = CONFIGS[name], [], X.choose

    def watch(z, correction, top):
        e, s = choose(z, correction, top)
        rest = [x for x in range(len(z)) if x not in e and correction[x] == correction[e[-1]]]
        gaps.extend(z[e[-1]] - z[x] for x in rest)
        return e, s

    monkeypatch.setattr(X, "choose", watch)
    reference(cfg, weights(cfg, 3), np.random.default_rng(12).integers(0, cfg["vocab"], 150))
    assert min(gaps) > 0.1


def test_config_reads_every_field():
    from tang_b200 import DotanexConfig, registry
    from tang_b200.dotanex import ATTENTION, DENSE, LATENT, LIGHTNING, MOE, NONE

    c = DotanexConfig.from_dict(CONFIGS["mixed"])
    assert (c.width, c.vocab, c.eps, c.streams, len(c.layers)) == (72, 101, 1e-5, 3, 10)
    a, l, g, last = c.layers[0], c.layers[1], c.layers[2], c.layers[8]
    assert (a.kind, a.heads, a.kv_heads, a.dim, a.vdim, a.window, a.scale, a.weights_of) == (ATTENTION, 6, 2, 20, 20, 17, 20 ** -0.5, -1)
    assert (a.rot.dims, a.rot.base, a.rot.factor, a.rot.low, a.rot.high, a.rot.original) == (8, 10000.0, 4.0, 1.0, 3.0, 64)
    assert (a.mlp.kind, a.mlp.experts, a.mlp.identity, a.mlp.top, a.mlp.ff, a.mlp.limit, a.mlp.shared_ff, a.mlp.shared_limit) == (MOE, 5, 3, 2, 24, 1.3, 40, 0.9)
    assert (l.kind, l.heads, l.dim, l.rot_dim, l.vdim, l.q_rank, l.kv_rank, l.mlp.kind, l.mlp.ff) == (LATENT, 3, 12, 8, 20, 24, 28, DENSE, 50)
    assert (l.rot.dims, l.rot.factor, l.rot.original, l.rot.fast, l.rot.slow) == (8, 4.0, 64, 16.0, 1.0)
    assert (g.kind, g.heads, g.dim, g.vdim, g.decay) == (LIGHTNING, 3, 20, 40, (1 - 0.6, 1 - 0.6 ** 2, 1 - 0.6 ** 3))
    assert c.layers[4].mlp.kind == NONE and last.rot.factor == 0 and last.rot.dims == 20
    assert [x.weights_of for x in c.layers] == [-1, -1, -1, -1, -1, 1, -1, 0, -1, 2]
    assert registry.resolve(CONFIGS["mixed"])[0] is DotanexConfig
    # keys and values of four attention layers (one of them repeated), latents and rotated parts of three, states of three
    assert c.cache_bytes_per_token(1) == 2 * (2 * (2 * 24 + 3 * 24 + 2 * 24 + 2 * 24) + 2 * (32 + 16) + 48 + 16)
    assert c.state_bytes() == 4 * (2 * 3 * 20 * 40 + 2 * 24 * 16)
    assert c.bytes_per_slot(0, 10) == 10 * 2 * c.cache_bytes_per_token(1) + c.state_bytes()


def test_parts_of_a_layer_may_be_absent():
    from tang_b200 import DotanexConfig
    from tang_b200.dotanex import tensor_names
    from tang_b200.stepmodel import NO_WINDOW

    c = json.loads(json.dumps(config([attn(2, 1, 8, 5, moe(2, 0, 1, 4, 4)), latent(1, 4, 2, 4, 4, 4)])))
    del c["layers"][0]["mixer"]["mask"], c["layers"][0]["mixer"]["rot"], c["layers"][0]["mlp"]["shared"], c["layers"][0]["mlp"]["router"]["identity"]
    l = DotanexConfig.from_dict(c).layers[0]
    assert l.window == NO_WINDOW and l.rot.dims == 0 and l.mlp.shared_ff == 0 and l.mlp.identity == 0
    names = [n for n, _, _, _ in tensor_names(DotanexConfig.from_dict(c))]
    assert not any("shared" in n or n.startswith("l1.hc2") for n in names) and "l0.mlp.correction" in names


def test_config_rejects_what_it_does_not_know():
    from tang_b200 import DotanexConfig
    from tang_b200.stepmodel import ConfigError

    def broken(change):
        c = json.loads(json.dumps(CONFIGS["mixed"]))
        change(c)
        return c

    for change, what in ((lambda c: c["layers"][2].update(type="scan"), "scan"), (lambda c: c["layers"][1]["mlp"].update(kind="sparse"), "sparse"),
                         (lambda c: c["layers"][0]["mixer"].update(vdim=21), "vdim"), (lambda c: c["layers"][6]["mixer"]["decay"].append(0.5), "decays"),
                         (lambda c: c["layers"][3]["mixer"].update(rot_dim=8), "rot_dim"), (lambda c: c["layers"][1]["mixer"].pop("q_rank"), "q_rank"),
                         (lambda c: c["layers"][5]["mixer"].update(heads=4), "weights_of"), (lambda c: c["layers"][5].update(weights_of=7), "weights_of"),
                         (lambda c: c["layers"][5].update(weights_of=10), "weights_of"), (lambda c: c.pop("streams"), "streams"), (lambda c: c.pop("norm"), "norm")):
        with pytest.raises(ConfigError, match=what):
            DotanexConfig.from_dict(broken(change))


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_tensor_names_are_the_checkpoints(name):
    from tang_b200 import DotanexConfig
    from tang_b200.dotanex import tensor_names

    names = [n for n, _, _, _ in tensor_names(DotanexConfig.from_dict(CONFIGS[name]))]
    assert len(names) == len(set(names)) and set(names) == set(weights(CONFIGS[name], 0))


@pytest.mark.parametrize("dims,base,scaling", [(8, 10000.0, None), (64, 500000.0, (8.0, 1.0, 4.0, 8192)), (10, 50.0, (2.0, 0.5, 2.0, 40)), (2, 1000.0, (3.0, 1.0, 2.0, 5)),
                                               (128, 10000.0, (1.0, 1.0, 32.0, 2048))])
def test_banded_frequencies(dims, base, scaling):
    from tang_b200 import _build, load

    _build.build_library()
    f = (C.c_float * (dims // 2))()
    factor, low, high, original = scaling or (0.0, 0.0, 0.0, 0.0)
    assert load().tq_banded_frequencies(dims, base, factor, low, high, original, f) == 0
    sc = None if scaling is None else {"factor": factor, "low": low, "high": high, "original": original}
    assert np.allclose(np.array(f[:]), X.banded_frequencies({"dims": dims, "base": base, "scaling": sc})[0], rtol=1e-6)
    assert load().tq_banded_frequencies(3, base, 0.0, 0.0, 0.0, 0.0, f) != 0 and load().tq_banded_frequencies(4, base, 2.0, 3.0, 3.0, 10.0, f) != 0


@pytest.mark.parametrize("dims,base,scaling", [(8, 10000.0, None), (64, 500000.0, (8.0, 512, 32.0, 1.0)), (10, 50.0, (2.0, 4096, 4.0, 2.0))])
def test_the_two_restatements_of_yarn_agree(dims, base, scaling):
    import numuzen_oracle as N

    rot = {"dims": dims, "base": base, "scaling": None if scaling is None else dict(zip(("factor", "original", "fast", "slow"), scaling))}
    assert np.allclose(X.yarn_frequencies(rot)[0], N.frequencies(rot)[0]) and X.yarn_frequencies(rot)[1] == pytest.approx(N.frequencies(rot)[1])


def test_slots_follow_the_cache_budget(tmp_path, monkeypatch):
    """Without a largest position the default holds, and slots are cut to the budget, states included."""
    from tang_b200 import DotanexConfig, registry

    cfg = CONFIGS["odd"]
    w = weights(cfg, 5)
    save(tmp_path, cfg, w)
    got = {}

    class Fake:
        @classmethod
        def from_tensors(cls, dev, config, tensors, dtype, max_slots, max_seq):
            got.update(slots=max_slots, seq=max_seq, names=set(tensors))

    monkeypatch.setitem(registry.ARCHITECTURES, "Dotanex", (DotanexConfig, Fake))
    registry.load_model(None, str(tmp_path))
    assert got["seq"] == registry.DEFAULT_MAX_SEQ and got["slots"] == 64 and got["names"] == set(w)
    per = DotanexConfig.from_dict(cfg).bytes_per_slot(1, 100)
    registry.load_model(None, str(tmp_path), max_seq=100, cache_budget=5 * per + 1)
    assert got["seq"] == 100 and got["slots"] == 5
