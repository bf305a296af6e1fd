"""Host side of the Numuzen family, without a GPU: configuration, tensor list, slots, frequencies, and the numpy
implementation's own consistency (prompt in one piece against token by token, hand-computed cases)."""
import ctypes as C
import json
import math

import numpy as np
import pytest

import numuzen_oracle as N
from numuzen_util import CONFIGS, RANKS, attn, config, gla, moe, reference, save, weights


def test_numpy_model_does_not_depend_on_the_cut():
    cfg = CONFIGS["mixed"]
    w = weights(cfg, 3, RANKS["mixed"])
    tokens = list(np.random.default_rng(2).integers(0, cfg["vocab"], 41))
    whole = reference(cfg, w, tokens)
    m = N.Numuzen(cfg, w)
    st = m.new_state()
    cut = np.concatenate([m.forward(tokens[a:b], st) for a, b in ((0, 1), (1, 3), (3, 20), (20, 41))])
    assert np.abs(whole - cut).max() < 1e-10


def test_numpy_mechanisms_by_hand():
    assert [j for j in range(12) if N.visible(9, j, 3)] == [7, 8, 9]
    # one key: weight e^s / (1 + e^s) beside the sink, the score capped
    q, k, v = np.array([2.0, 0.0]), np.array([[3.0, 1.0]]), np.array([[5.0]])
    s = 4.0 * math.tanh(6.0 * 0.5 / 4.0)
    assert N.one_query(q, k, v, 0, 0.5, 4.0, 1)[0] == pytest.approx(5.0 * math.exp(s) / (1 + math.exp(s)))
    # two steps of the recurrence: the decay acts on the key channels
    o, S = N.gla(np.array([[1.0, 1.0], [1.0, 2.0]]), np.array([[1.0, 2.0], [0.5, 0.0]]), np.array([[3.0], [4.0]]), np.array([[0.1, 0.1], [0.5, 0.25]]),
                 np.zeros((2, 1)))
    assert o[0, 0] == pytest.approx(9.0) and S[:, 0] == pytest.approx([0.5 * 3 + 0.5 * 4, 0.25 * 6]) and o[1, 0] == pytest.approx(3.5 + 3.0)
    assert N.decay(np.array([0.0]), 2.0)[0] == pytest.approx(math.sqrt(0.5))
    e, s = N.choose(np.array([0.1, 2.0, 2.0, -1.0]), 3)
    assert e == [1, 2, 0] and s[0] == pytest.approx(1 / (1 + math.exp(-2.0)))
    assert N.clamped_glu(np.array([50.0]), np.array([-50.0]), 2.0)[0] == pytest.approx(2.0 / (1 + math.exp(-1.702 * 2)) * -1.0)
    assert N.norm(np.array([3.0, 4.0]), np.array([0.0, 1.0]), 0.0) == pytest.approx([3 / math.sqrt(12.5), 8 / math.sqrt(12.5)])
    x = N.rotate(np.array([[1.0, 2.0, 0.0, 0.0, 7.0]]), 1, {"dims": 4, "base": 100.0, "scaling": None})
    assert x[0] == pytest.approx([math.cos(1), 2 * math.cos(0.1), math.sin(1), 2 * math.sin(0.1), 7.0])


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_expert_choices_of_the_test_models_are_not_close_calls(name, monkeypatch):
    cfg, gaps, choose = CONFIGS[name], [], N.choose

    def watch(z, top):
        s = np.sort(z)[::-1]
        if top < len(z):
            gaps.append(s[top - 1] - s[top])
        return choose(z, top)

    monkeypatch.setattr(N, "choose", watch)
    reference(cfg, weights(cfg, 3, RANKS[name]), np.random.default_rng(12).integers(0, cfg["vocab"], 150))
    assert min(gaps) > 0.1


def test_config_reads_every_field():
    from tang_b200 import NumuzenConfig, registry
    from tang_b200.numuzen import ATTENTION, GLA

    c = NumuzenConfig.from_dict(CONFIGS["mixed"])
    assert (c.width, c.vocab, c.eps, len(c.layers)) == (72, 101, 1e-5, 5)
    a, g, n, last = c.layers[0], c.layers[1], c.layers[2], c.layers[4]
    assert (a.kind, a.heads, a.kv_heads, a.dim, a.vdim, a.window, a.softcap, a.scale) == (ATTENTION, 6, 2, 20, 20, 17, 20.0, 20 ** -0.5)
    assert (a.rot.dims, a.rot.base, a.rot.factor, a.rot.original, a.rot.fast, a.rot.slow) == (8, 10000.0, 4.0, 64, 16.0, 1.0)
    assert (a.experts.count, a.experts.top, a.experts.ff, a.experts.limit) == (5, 2, 24, 1.3)
    assert (g.kind, g.heads, g.dim, g.vdim, g.tau, g.scale) == (GLA, 3, 20, 40, 12.0, 20 ** -0.5)
    assert n.experts is None and last.rot.factor == 0 and last.rot.dims == 20
    assert registry.resolve(CONFIGS["mixed"])[0] is NumuzenConfig
    # keys and values of three attention layers, head sizes padded to 8 values; f32 states of two recurrent ones
    assert c.cache_bytes_per_token(1) == 2 * 2 * (2 * 24 + 3 * 24 + 2 * 24)
    assert c.state_bytes() == 4 * (3 * 20 * 40 + 2 * 24 * 16)
    assert c.bytes_per_slot(0, 10) == 10 * 2 * c.cache_bytes_per_token(1) + c.state_bytes()


def test_config_rejects_what_it_does_not_know():
    from tang_b200 import NumuzenConfig
    from tang_b200.stepmodel import ConfigError

    def broken(change):
        c = json.loads(json.dumps(CONFIGS["mixed"]))
        change(c)
        return c

    for change, what in ((lambda c: c["layers"][1].update(type="scan"), "scan"), (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "dense"),
                         (lambda c: c["layers"][0]["mixer"].update(vdim=21), "vdim"), (lambda c: c["layers"][0]["mixer"].pop("softcap"), "softcap"),
                         (lambda c: c["layers"][1]["mixer"].pop("tau"), "tau"), (lambda c: c.pop("norm"), "norm")):
        with pytest.raises(ConfigError, match=what):
            NumuzenConfig.from_dict(broken(change))


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_tensor_names_are_the_checkpoints(name):
    from tang_b200 import NumuzenConfig
    from tang_b200.numuzen import tensor_names

    names = [n for n, _, _, _ in tensor_names(NumuzenConfig.from_dict(CONFIGS[name]))]
    assert len(names) == len(set(names)) and set(names) == set(weights(CONFIGS[name], 0, RANKS[name]))


@pytest.mark.parametrize("dims,base,scaling", [(8, 10000.0, None), (64, 500000.0, (8.0, 512, 32.0, 1.0)), (10, 50.0, (2.0, 4096, 4.0, 2.0)), (2, 1000.0, (3.0, 9, 1.0, 0.5)),
                                               (128, 10000.0, (1.0, 2048, 32.0, 1.0))])
def test_frequencies(dims, base, scaling):
    from tang_b200 import _build, load

    _build.build_library()
    f, mult = (C.c_float * (dims // 2))(), C.c_float()
    factor, original, fast, slow = scaling or (0.0, 0.0, 0.0, 0.0)
    assert load().tq_yarn_frequencies(dims, base, factor, original, fast, slow, f, C.byref(mult)) == 0
    sc = None if scaling is None else {"factor": factor, "original": original, "fast": fast, "slow": slow}
    want, want_mult = N.frequencies({"dims": dims, "base": base, "scaling": sc})
    assert np.allclose(np.array(f[:]), want, rtol=1e-6) and mult.value == pytest.approx(want_mult, rel=1e-6)
    assert load().tq_yarn_frequencies(3, base, 0.0, 0.0, 0.0, 0.0, f, C.byref(mult)) != 0


def test_slots_follow_the_cache_budget(tmp_path, monkeypatch):
    """Without a largest position the default holds, and slots are cut to the budget, states included."""
    from tang_b200 import NumuzenConfig, registry

    cfg = CONFIGS["odd"]
    w = weights(cfg, 5, RANKS["odd"])
    save(tmp_path, cfg, w)
    got = {}

    class Fake:
        @classmethod
        def from_tensors(cls, dev, config, tensors, dtype, max_slots, max_seq):
            got.update(slots=max_slots, seq=max_seq, names=set(tensors))

    monkeypatch.setitem(registry.ARCHITECTURES, "Numuzen", (NumuzenConfig, Fake))
    registry.load_model(None, str(tmp_path))
    assert got["seq"] == registry.DEFAULT_MAX_SEQ and got["slots"] == 64 and got["names"] == set(w)
    per = NumuzenConfig.from_dict(cfg).bytes_per_slot(1, 100)
    registry.load_model(None, str(tmp_path), max_seq=100, cache_budget=5 * per + 1)
    assert got["seq"] == 100 and got["slots"] == 5


def test_other_shapes_are_only_a_configuration():
    from tang_b200 import NumuzenConfig

    c = NumuzenConfig.from_dict(config([gla(1, 1, 1, moe(1, 1, 1)), attn(1, 1, 2, 1, rot=2)], width=1, vocab=2))
    assert c.layers[0].experts.count == 1 and c.layers[1].window == 1
