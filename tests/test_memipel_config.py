"""Memipel on the CPU: the configuration reader, the tensor list, what each stop of the schedule keeps in the cache, and the
plain implementation's own properties (mechanisms restated a second way)."""
import copy
import math

import numpy as np
import pytest

from memipel_helpers import CONFIGS, MEM_A, MEM_B, attention, config, latent, layer, lightning, moe
from plain import memipel_plain as M


def _cfg(raw):
    from stratum_b200.config import find_architecture
    return find_architecture(raw).config_class.from_dict(raw)


def _model(raw):
    from stratum_b200.config import find_architecture
    from stratum_b200.engine.model import Model
    return Model(find_architecture(raw).describe_model(_cfg(raw)), None)


def test_configuration_round_trip_and_registry():
    from stratum_b200.config import find_architecture
    from stratum_b200.config.memipel import MemipelConfig
    assert find_architecture({"architecture": "Memipel"}).config_class is MemipelConfig
    for raw in CONFIGS.values():
        cfg = _cfg(raw)
        assert MemipelConfig.from_dict(cfg.to_dict()) == cfg
        assert [la.kind for la in cfg.layers] == [e["type"] for e in raw["layers"]]
    a = _cfg(MEM_A)
    assert (a.layers[2].mixer.conv, a.layers[2].mixer.window, a.layers[1].mixer.v_mix) == (3, 50, False)
    assert (a.layers[3].mixer.q_rank, a.layers[3].mixer.kv_rank, a.layers[3].mlp) == (28, 36, None)
    assert a.layers[0].mixer.decay == (0.5, 0.9375, 1.0 - 2.0 ** -7)
    f = a.layers[0].mlp
    assert (f.experts, f.top, f.groups, f.keep, f.expert.limit, f.shared.ff, f.shared.limit) == (6, 2, 3, 2, 1.1, 36, 0.7)
    assert a.layers[2].mlp.shared is None and a.layers[4].mixer.window == 0


def test_what_a_file_does_not_mention_does_not_exist():
    raw = copy.deepcopy(MEM_A)
    m = raw["layers"][2]["mixer"]
    for key in ("conv", "v_mix", "mask"):
        del m[key]
    del raw["layers"][3]["mixer"]["mask"]
    del raw["layers"][0]["mlp"]["router"]["groups"]
    del raw["layers"][0]["mlp"]["shared"]
    cfg = _cfg(raw)
    assert type(cfg).from_dict(cfg.to_dict()) == cfg
    model = _model(raw)
    part = model.layers[2].part("mixer")
    assert (part.taps, part.window, part.value_mix) == (0, 0, None)
    assert model.layers[3].part("mixer").window == 0 and model.layers[3].part("feed_forward") is None
    f = model.layers[0].part("feed_forward")
    assert (f.n_groups, f.keep, f.shared_ff) == (1, 1, 0)
    t = model.tensors()
    assert "l2.mix.vmix" not in t and "l2.mix.q.conv" not in t and "l0.mlp.shared.up" not in t
    assert model.layers[4].part("mixer").value_mix == "first"       # now the first layer that mixes lends


def test_configuration_problems_are_listed_together():
    from stratum_b200.config import ConfigError
    raw = copy.deepcopy(MEM_A)
    del raw["vocab"]
    raw["layers"][0]["mixer"]["decay"] = [0.5]               # for 3 heads
    raw["layers"][0]["mlp"]["router"]["groups"]["count"] = 4 # of 6 experts
    raw["layers"][1]["mixer"]["kv_heads"] = 3                # 4 heads on 3 kv heads
    raw["layers"][2]["mlp"]["router"]["top"] = 5             # of 4 that can be chosen
    del raw["layers"][3]["mixer"]["q_rank"]
    raw["layers"][4]["mixer"]["vdim"] = 20                   # 20 values mixed with 32
    raw["layers"][5]["type"] = "convolution"
    with pytest.raises(ConfigError) as e:
        _cfg(raw)
    for piece in ("vocab", "1 numbers for 3 heads", "groups.count=4", "kv_heads=3", "top=5", "q_rank", "mixes its 20 values",
                  "convolution"):
        assert piece in str(e.value), piece


def test_tensors_of_the_model():
    t = _model(MEM_A).tensors()
    shape = lambda n: tuple(t[n].shape)                                                          # noqa: E731
    assert shape("embed") == (211, 72) and shape("final.norm") == (72,) and "head" not in t
    p = "l2.mix."
    assert (shape(p + "q"), shape(p + "k"), shape(p + "v"), shape(p + "o")) == ((96, 72), (48, 72), (32, 72), (72, 64))
    assert (shape(p + "q.b"), shape(p + "k.b"), shape(p + "v.b"), shape(p + "o.b")) == ((96,), (48,), (32,), (72,))
    assert (shape(p + "q.conv"), shape(p + "k.conv"), shape(p + "v.conv"), shape(p + "vmix")) == ((96, 3), (48, 3), (32, 3), ())
    assert "l1.mix.vmix" not in t and shape("l4.mix.vmix") == ()
    p = "l3.mix."
    assert (shape(p + "dq"), shape(p + "dq.norm"), shape(p + "uq"), shape(p + "dkv"), shape(p + "dkv.norm")) == \
        ((28, 72), (28,), (60, 28), (36, 72), (36,))
    assert (shape(p + "uk"), shape(p + "uv"), shape(p + "sink"), shape(p + "o")) == ((60, 36), (36, 36), (3,), (72, 36))
    p = "l0.mix."
    assert (shape(p + "q"), shape(p + "v"), shape(p + "g"), shape(p + "norm"), shape(p + "o")) == \
        ((36, 72), (60, 72), (60, 72), (60,), (72, 60))
    assert shape("l0.mlp.router") == (6, 72) and shape("l0.mlp.e5.gate") == (20, 72) and shape("l0.mlp.shared.down") == (72, 36)
    assert shape("l1.mlp.up") == (96, 72) and shape("l1.mlp.down") == (72, 96) and "l1.norm2" not in t
    assert "l0.mlp.router.b" not in t and "l0.mlp.correction" not in t


def test_what_the_stops_keep():
    """A layer behind a convolution owns windowed keys and values and a block of inputs; one tap or none needs no block;
    latent attention keeps the latent alone, lightning attention a state."""
    import torch
    from stratum_b200.cache import KVSpec, SequenceCache, StateSpec
    specs = _model(MEM_A).cache_specs()
    kv, st = specs[2]
    assert isinstance(kv, KVSpec) and (kv.n_kv_heads, kv.head_dim, kv.v_heads, kv.v_dim, kv.window) == (2, 24, 2, 16, 50)
    assert st == StateSpec((2 * (96 + 48 + 32),)) and specs[0] == StateSpec((3 * 12 * 20,))
    assert (specs[3].n_kv_heads, specs[3].head_dim, specs[3].v_heads, specs[3].window) == (1, 36, 0, 45)
    b = _model(MEM_B).cache_specs()
    assert isinstance(b[2], KVSpec) and isinstance(b[4], KVSpec) and isinstance(b[0], tuple)
    c = SequenceCache(specs, 512, 3, torch.float32, "cpu")
    v = c.layer_view(2, True, {})
    assert v.parts[0].k.shape == (8, 2, 64, 24) and v.parts[0].v.shape == (8, 2, 64, 16) and v.parts[1].state.shape == (4, 352)


def test_who_lends_values_and_who_mixes():
    mixes = lambda raw: [la.part("mixer").value_mix for la in _model(raw).layers if la.spec.parts["mixer"].kind == "conv_attention"]  # noqa: E731
    assert mixes(MEM_A) == [None, "first", "mix"] and mixes(MEM_B) == ["first", "mix", "mix"]
    assert mixes(config([layer("attention", attention())])) == ["first"]


# ------------------------------------------------------------------------------------------ the oracle, restated
def test_plain_attention_by_loops():
    rng = np.random.default_rng(0)
    m = attention(heads=4, kv=2, dim=3, vdim=2, conv=3, size=4, scale=0.7)
    T, width = 11, 5
    h = rng.standard_normal((T, width))
    W = {"q": (12, width), "k": (6, width), "v": (4, width), "o": (width, 8)}
    W = {n: rng.standard_normal(s) for n, s in W.items()}
    W.update({n + ".b": rng.standard_normal(W[n].shape[0]) for n in ("q", "k", "v", "o")})
    W.update({n + ".conv": rng.standard_normal((W[n].shape[0], 3)) for n in ("q", "k", "v")})
    W["vmix"] = np.array(0.3)
    first = rng.standard_normal((T, 4))
    y = {}
    for n in ("q", "k", "v"):
        u = h @ W[n].T + W[n + ".b"]
        y[n] = np.zeros_like(u)
        for t in range(T):
            for j in range(3):
                if t - 2 + j >= 0:
                    y[n][t] += W[n + ".conv"][:, j] * u[t - 2 + j]
    y["v"] = 0.7 * y["v"] + 0.3 * first
    out = np.zeros((T, 8))
    for t in range(T):
        for a in range(4):
            g, num, den = a // 2, np.zeros(2), 0.0
            for s in range(max(0, t - 3), t + 1):
                e = math.exp(0.7 * y["q"][t, 3 * a:3 * a + 3] @ y["k"][s, 3 * g:3 * g + 3] - 4.0 ** -(a + 1) * (t - s))
                num, den = num + e * y["v"][s, 2 * g:2 * g + 2], den + e
            out[t, 2 * a:2 * a + 2] = num / den
    assert np.allclose(M.attention(m, W, h, "", first), out @ W["o"].T + W["o.b"])


def test_plain_latent_attention_by_loops():
    rng = np.random.default_rng(1)
    m = latent(heads=2, dim=3, vdim=4, q_rank=5, kv_rank=6, scale=0.6, size=3)
    T, width = 8, 7
    W = {n: rng.standard_normal(s) for n, s in {"dq": (5, width), "dq.norm": (5,), "uq": (6, 5), "dkv": (6, width), "dkv.norm": (6,),
                                                "uk": (6, 6), "uv": (8, 6), "sink": (2,), "o": (width, 8)}.items()}
    h, out = rng.standard_normal((T, width)), np.zeros((T, 8))
    norm = lambda x, w: x / np.sqrt((x * x).mean() + 0.01) * w                                   # noqa: E731
    q = [W["uq"] @ norm(W["dq"] @ x, W["dq.norm"]) for x in h]
    c = [norm(W["dkv"] @ x, W["dkv.norm"]) for x in h]
    for t in range(T):
        for a in range(2):
            num, den = np.zeros(4), math.exp(W["sink"][a])
            for s in range(max(0, t - 2), t + 1):
                e = math.exp(0.6 * q[t][3 * a:3 * a + 3] @ (W["uk"] @ c[s])[3 * a:3 * a + 3])
                num, den = num + e * (W["uv"] @ c[s])[4 * a:4 * a + 4], den + e
            out[t, 4 * a:4 * a + 4] = num / den
    assert np.allclose(M.latent_attention(m, 0.01, W, h, ""), out @ W["o"].T)


def test_plain_lightning_as_a_sum_over_the_past():
    rng = np.random.default_rng(2)
    m = lightning(heads=2, dim=3, vdim=4, decay=[0.7, 0.95])
    T, width = 9, 10
    h = rng.standard_normal((T, width))
    W = {k: rng.standard_normal(s) for k, s in (("q", (6, width)), ("k", (6, width)), ("v", (8, width)), ("g", (8, width)))}
    W["o"], W["norm"] = np.eye(8), rng.standard_normal(8)
    act = lambda z: z / (1 + np.exp(-z))                                                         # noqa: E731
    q, k, v = act(h @ W["q"].T), act(h @ W["k"].T), act(h @ W["v"].T)
    o = np.zeros((T, 8))
    for t in range(T):
        for s in range(t + 1):
            for a in range(2):
                o[t, 4 * a:4 * a + 4] += m["decay"][a] ** (t - s) * (q[t, 3 * a:3 * a + 3] @ k[s, 3 * a:3 * a + 3]) * v[s, 4 * a:4 * a + 4]
    want = o / np.sqrt((o ** 2).mean(-1, keepdims=True) + 1e-5) * W["norm"] / (1 + np.exp(-h @ W["g"].T))
    assert np.allclose(M.lightning(m, 1e-5, W, h, ""), want)


def test_plain_routing():
    """The group of the largest score stays although the other group's two best sum to more; the chosen scores are not
    renormalised; with one group all experts can be chosen."""
    z = np.log(np.array([[0.40, 0.01, 0.02, 0.03, 0.30, 0.24]]))
    w = M.route(z, 2, 2, 1)
    assert np.allclose(w, [[0.40, 0, 0.02, 0, 0, 0]])
    assert np.allclose(M.route(z, 2), [[0.40, 0, 0, 0, 0.30, 0]])
    assert np.allclose(M.route(z, 3, 2, 2), [[0.40, 0, 0, 0, 0.30, 0.24]])
    assert np.isclose(M.route_margin(z, 2, 2, 1), min(math.log(0.40 / 0.30), math.log(0.02 / 0.01)))


def test_plain_dense_and_expert():
    W = {"up": np.eye(3), "down": np.eye(3)}
    z = np.array([[-1.0, 0.2, 2.0]])
    assert np.allclose(M.dense(W, z, ""), [[v * 0.5 * math.erfc(-v / math.sqrt(2)) for v in z[0]]])
    W = {"gate": np.array([[1.0], [1.0], [1.0]]), "up": np.array([[-5.0], [0.5], [9.0]]), "down": np.eye(3)}
    for h in (-2.0, 0.3, 4.0):
        g = min(h, 1.5)
        want = [g / (1 + np.exp(-1.702 * g)) * (np.clip(v * h, -1.5, 1.5) + 1) for v in (-5.0, 0.5, 9.0)]
        assert np.allclose(M.clamped_expert(W, np.array([[h]]), "", 1.5)[0], want)


def test_plain_sublayers_side_by_side_on_one_norm():
    """A layer's two sublayers add up: the stream after a layer is the stream after the mixer alone plus the feed-forward of
    the same normed rows."""
    from memipel_helpers import lively
    import torch
    from stratum_b200.weights.random_init import random_tensors
    from stratum_b200.engine.model import expected_tensors
    raw = config([layer("lightning", lightning(), moe())])
    bare = config([layer("lightning", lightning())])
    t = random_tensors(expected_tensors(_cfg(raw)), 3, 0.05, torch.float32)
    lively(t)
    w = {n: v.double().numpy() for n, v in t.items()}
    toks, a, b = [5, 3, 99], [], []
    M.forward(raw, w, toks, a)
    M.forward(bare, w, toks, b)
    h = M.rms_norm(w["embed"][toks], 1 + w["l0.norm1"], 1e-5)
    assert np.allclose(a[0] - b[0], M.experts(raw["layers"][0]["mlp"], w, h, "l0.mlp."))


def test_plain_prefix_of_a_sequence_is_the_sequence_of_the_prefix():
    from memipel_helpers import lively
    import torch
    from stratum_b200.weights.random_init import random_tensors
    from stratum_b200.engine.model import expected_tensors
    for raw in (MEM_A, MEM_B):
        t = random_tensors(expected_tensors(_cfg(raw)), 3, 0.05, torch.float32)
        lively(t)
        w = {n: v.double().numpy() for n, v in t.items()}
        toks = np.random.default_rng(0).integers(0, raw["vocab"], 60).tolist()
        whole = M.forward(raw, w, toks)
        assert np.isfinite(whole).all()
        for n in (1, 2, 33, 50):
            assert np.allclose(M.forward(raw, w, toks[:n]), whole[:n], rtol=1e-9, atol=1e-9)
