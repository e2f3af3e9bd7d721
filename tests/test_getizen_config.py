"""Getizen on the CPU: the configuration reader, the tensor list, what each stop of the schedule keeps in the cache, pages
of chunks, and the plain implementation's own properties (mechanisms restated a second way)."""
import copy

import numpy as np
import pytest

from getizen_helpers import CONFIGS, GET_A, GET_B, config, layer, left, parallel, retention
from plain import getizen_plain as G


def _cfg(raw):
    from stratum_b200.config import find_architecture
    return find_architecture(raw).config_class.from_dict(raw)


def _model(raw):
    from stratum_b200.config import find_architecture
    from stratum_b200.engine.model import Model
    return Model(find_architecture(raw).describe_model(_cfg(raw)), None)


def test_configuration_round_trip_and_registry():
    from stratum_b200.config import find_architecture
    from stratum_b200.config.getizen import GetizenConfig
    assert find_architecture({"architecture": "Getizen"}).config_class is GetizenConfig
    for raw in CONFIGS.values():
        cfg = _cfg(raw)
        assert GetizenConfig.from_dict(cfg.to_dict()) == cfg
        assert [la.kind for la in cfg.layers] == [e["type"] for e in raw["layers"]]
    a = _cfg(GET_A)
    assert a.layers[0].mixer.left.chunk == 50 and a.layers[0].mixer.left.rot.scaling.original == 64
    assert a.layers[0].mixer.right.conv == 3 and a.layers[1].mixer.decay == (0.75, 0.9375, 1.0 - 2.0 ** -6)
    assert (a.alpha, a.norm_groups, a.layers[1].mlp.limit, a.layers[2].mlp) == (1.7, 3, 0.9, None)
    assert _cfg(GET_B).layers[2].mixer.left.chunk == 0 and _cfg(GET_B).layers[2].mixer.left.scale == -0.4


def test_what_a_file_does_not_mention_does_not_exist():
    raw = copy.deepcopy(GET_A)
    del raw["layers"][0]["mixer"]["left"]["rot"]
    del raw["layers"][0]["mixer"]["left"]["mask"]
    del raw["layers"][2]["mixer"]["left"]["rot"]["scaling"]
    del raw["layers"][1]["mixer"]["rot"]
    raw["layers"][1]["mlp"] = None
    del raw["norm"]["groups"]
    cfg = _cfg(raw)
    assert type(cfg).from_dict(cfg.to_dict()) == cfg
    model = _model(raw)
    pair = model.layers[0].part("mixer")
    assert pair.mixers[0].position is None and pair.mixers[0].chunk == 0
    assert model.layers[2].part("mixer").mixers[0].position.scaling is None
    assert model.layers[1].part("mixer").position is None and model.layers[1].part("feed_forward") is None
    assert "l1.norm2" not in model.tensors() and model.layers[0].part("mixer_norm").groups == 1


def test_configuration_problems_are_listed_together():
    from stratum_b200.config import ConfigError
    raw = copy.deepcopy(GET_A)
    del raw["vocab"]
    raw["norm"]["groups"] = 7                                # of 72
    raw["layers"][0]["mixer"]["left"]["kv_heads"] = 3        # 4 heads on 3 kv heads
    raw["layers"][0]["mixer"]["right"]["blocks"] = 7         # of 60 channels
    raw["layers"][1]["mixer"]["decay"] = [0.5]               # for 3 heads
    raw["layers"][2]["type"] = "convolution"
    raw["layers"][3]["mixer"]["rot"]["dims"] = 21
    with pytest.raises(ConfigError) as e:
        _cfg(raw)
    for piece in ("vocab", "groups=7", "kv_heads=3", "blocks=7", "1 numbers for 3 heads", "convolution", "dims=21"):
        assert piece in str(e.value), piece


def test_tensors_of_the_model():
    t = _model(GET_A).tensors()
    shape = lambda n: tuple(t[n].shape)                                                          # noqa: E731
    assert shape("embed") == (211, 72) and shape("embed.norm") == shape("final.norm") == (72,) and "head" not in t
    p = "l0.mix.left."
    assert (shape(p + "q"), shape(p + "k"), shape(p + "v"), shape(p + "g"), shape(p + "o")) == \
        ((96, 72), (48, 72), (32, 72), (64, 72), (72, 64))
    assert shape(p + "q.norm") == (96,) and shape(p + "k.norm") == (48,) and shape(p + "temp") == (4,)
    p = "l0.mix.right."
    assert shape(p + "y") == shape(p + "x") == (60, 72) and shape(p + "conv") == (60, 3) and shape(p + "o") == (72, 60)
    assert shape(p + "ra") == shape(p + "ri") == (5, 12, 12) and shape(p + "ra.b") == (5, 12) and shape(p + "lam") == (60,)
    assert shape("l0.mix.left.out") == shape("l0.mix.right.out") == (72,)
    assert shape("l1.mix.v") == (60, 72) and shape("l1.mix.q") == (36, 72) and "l1.mix.norm" not in t
    assert "l2.norm2" not in t and shape("l1.mlp.gate") == (80, 72)
    # a file may carry the norm of a feed-forward that is not there
    from stratum_b200.config import find_architecture
    assert "l2.norm2".endswith(find_architecture("Getizen").ignored_tensor_suffixes)


def test_what_the_stops_keep():
    """A layer of two mixers owns keys and values that live in chunks and a block of state; layers that keep the same
    share a group of the cache."""
    import torch
    from stratum_b200.cache import KVSpec, SequenceCache, StateSpec
    raw = config([layer("parallel", parallel()), layer("retention", retention()), layer("parallel", parallel())])
    specs = _model(raw).cache_specs()
    kv, st = specs[0]
    assert isinstance(kv, KVSpec) and (kv.n_kv_heads, kv.head_dim, kv.v_heads, kv.v_dim, kv.chunk) == (2, 24, 2, 16, 50)
    assert isinstance(st, StateSpec) and st.shape == (60 * 4,) and specs[1] == StateSpec((3 * 12 * 20,))
    c = SequenceCache(specs, 512, 3, torch.float32, "cpu")
    assert len(c.groups) == 3 and c.layer_places == {0: ((0, 0), (1, 0)), 1: ((2, 0),), 2: ((0, 1), (1, 1))}
    v = c.layer_view(2, True, {0: torch.zeros(1, 1, dtype=torch.int32)})
    assert v.k is None and v.parts[0].k.shape == (8, 2, 64, 24) and v.parts[0].v.shape == (8, 2, 64, 16)
    assert v.parts[1].state.shape == (4, 240) and v.parts[0].writes and v.parts[0].block_table is not None
    assert v.parts[1].state.data_ptr() == c.groups[1].state[1].data_ptr()
    assert c.layer_view(1, False, {}).state.shape == (4, 720)


@pytest.mark.parametrize("chunk", [1, 5, 50, 63, 64, 65, 130, 200])
@pytest.mark.parametrize("step", [1, 2, 37, 64, 129])
def test_pages_of_chunks(chunk, step):
    """A sequence keeps exactly the pages that its next position's chunk has begun; the others are free again."""
    from stratum_b200.cache import PagePool, SequencePages
    pool = PagePool(16)
    sp = SequencePages(pool, chunk=chunk)
    while sp.length + step <= 600:
        sp.reserve(step)
        for p in range((sp.length - sp.length % chunk) // 64, (sp.length + step - 1) // 64 + 1):
            assert sp.table[p] >= 0                                   # what the step reads or writes is there
        sp.advance(step)
        start = sp.length - sp.length % chunk
        held = [i for i, p in enumerate(sp.table) if p >= 0]
        assert held == list(range(start // 64, (sp.length + 63) // 64)), (sp.length, held)
        assert pool.free_pages == 16 - len(held)
        pool.check()
    sp.release()
    assert pool.free_pages == 16


def test_rescaled_frequencies():
    from stratum_b200.parts.rope import precise_frequencies
    for sc in ({"factor": 6.0, "low": 0.8, "high": 5.0, "original": 700}, {"factor": 0.5, "low": 2.0, "high": 3.0, "original": 40},
               {"factor": 3.0, "low": 2.0, "high": 2.0, "original": 100}):
        rot = {"base": 20000.0, "dims": 48, "scaling": sc}
        got, mag = precise_frequencies(48, 20000.0, {"kind": "llama3", "factor": sc["factor"], "low_freq_factor": sc["low"],
                                                     "high_freq_factor": sc["high"], "original_max_position": sc["original"]})
        want = G.frequencies(rot)
        assert mag == 1.0 and np.allclose(got, want, rtol=2e-7, atol=0)
        plain = G.frequencies({"base": 20000.0, "dims": 48})
        assert np.isclose(want[0], plain[0]) and np.isclose(want[-1], plain[-1] / sc["factor"])     # kept, and scaled


# ------------------------------------------------------------------------------------------ the plain implementation
def test_plain_chunks():
    m = G.visible(13, 5)
    assert m[7].nonzero()[0].tolist() == [5, 6, 7] and m[5].nonzero()[0].tolist() == [5] and m[4].sum() == 5
    assert G.visible(6, None)[5].all() and G.visible(6, 0).sum() == 21


def test_plain_group_norm_is_the_plain_norm_part_by_part():
    rng = np.random.default_rng(0)
    x, g = rng.standard_normal((4, 12)), rng.uniform(0.5, 1.5, 12)
    y = G.group_norm(x, g, 1e-5, 3)
    for p in range(3):
        s = slice(4 * p, 4 * p + 4)
        assert np.allclose(y[:, s], G.rms_norm(x[:, s], g[s], 1e-5))
    assert np.allclose(G.group_norm(x, g, 1e-5, 1), G.rms_norm(x, g, 1e-5))


def test_plain_retention_is_the_sum_over_earlier_tokens():
    """o_t = sum_s decay^(t - s) (q_t . k_s) v_s, before the head's norm and the gate."""
    rng = np.random.default_rng(1)
    m = retention(heads=2, dim=6, vdim=4, rot=4, decay=[0.9, 0.6])
    T, width = 9, 10
    h = rng.standard_normal((T, width))
    w = {k: rng.standard_normal(s) for k, s in (("q", (12, width)), ("k", (12, width)), ("v", (8, width)), ("g", (8, width)))}
    w["o"] = np.eye(8)
    got = G.retention(m, 1e-5, w, h, "")
    q, k = (G.rotate((h @ w[n].T).reshape(T, 2, 6), m["rot"]) for n in ("q", "k"))
    v = (h @ w["v"].T).reshape(T, 2, 4)
    o = np.zeros((T, 2, 4))
    for t in range(T):
        for s in range(t + 1):
            for j in range(2):
                o[t, j] += m["decay"][j] ** (t - s) * (q[t, j] @ k[s, j]) / np.sqrt(6) * v[s, j]
    g = h @ w["g"].T
    want = (o / np.sqrt((o ** 2).mean(-1, keepdims=True) + 1e-5)).reshape(T, 8) * g / (1 + np.exp(-g))
    assert np.allclose(got, want)


def test_plain_recurrence_forgets_by_its_gates():
    """The weight of a token's input in a later state is the product of the decays in between."""
    rng = np.random.default_rng(2)
    T, width, blocks = 7, 6, 2
    u = rng.standard_normal((T, width))
    w = {"ra": rng.standard_normal((2, 3, 3)), "ri": rng.standard_normal((2, 3, 3)), "ra.b": rng.standard_normal((2, 3)),
         "ri.b": rng.standard_normal((2, 3)), "lam": rng.standard_normal(width)}
    S = G.linear_recurrence(u, blocks, w, "")
    gate = lambda m, t: np.concatenate([1 / (1 + np.exp(-(w[m][b] @ u[t, 3 * b:3 * b + 3] + w[m + ".b"][b]))) for b in range(2)])  # noqa: E731
    a = np.stack([np.exp(-8 * gate("ra", t) * np.log1p(np.exp(w["lam"]))) for t in range(T)])
    want = sum(np.prod(a[s + 1:], axis=0) * np.sqrt(1 - a[s] ** 2) * gate("ri", s) * u[s] for s in range(T))
    assert np.allclose(S[-1], want)


def test_plain_convolution_and_clamped_gate():
    x = np.arange(8, dtype=float).reshape(4, 2)
    w, b = np.array([[0.5, 1.0, 2.0], [1.0, 0.0, -1.0]]), np.array([0.1, -0.2])
    y = G.causal_conv(x, w, b)
    assert np.isclose(y[0, 0], 0.1) and np.isclose(y[3, 0], 0.1 + 0.5 * x[1, 0] + x[2, 0] + 2 * x[3, 0])
    assert np.isclose(y[1, 1], -0.2 - x[1, 1]) and np.isclose(y[2, 1], -0.2 + x[0, 1] - x[2, 1])
    W = {"gate": np.array([[1.0], [1.0], [1.0]]), "up": np.array([[-5.0], [0.5], [9.0]]), "down": np.eye(3)}
    for h in (-2.0, 0.3, 4.0):
        y = G.feed_forward({"limit": 1.5}, W, np.array([[h]]), "")[0]
        g = min(h, 1.5)
        want = [g / (1 + np.exp(-1.702 * g)) * (np.clip(v * h, -1.5, 1.5) + 1) for v in (-5.0, 0.5, 9.0)]
        assert np.allclose(y, want)


def test_plain_prefix_of_a_sequence_is_the_sequence_of_the_prefix():
    from getizen_helpers import lively
    import torch
    from stratum_b200.weights.random_init import random_tensors
    from stratum_b200.engine.model import expected_tensors
    for raw in (GET_A, GET_B):
        t = random_tensors(expected_tensors(_cfg(raw)), 3, 0.05, torch.float32)
        lively(t)
        w = {n: v.double().numpy() for n, v in t.items()}
        toks = np.random.default_rng(0).integers(0, raw["vocab"], 60).tolist()
        whole = G.forward(raw, w, toks)
        assert np.isfinite(whole).all()
        for n in (1, 2, 33, 50):
            assert np.allclose(G.forward(raw, w, toks[:n]), whole[:n], rtol=1e-9, atol=1e-9)
