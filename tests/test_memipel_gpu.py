"""Memipel on the GPU against the plain implementation: each kernel and each mechanism alone, whole prompts against
token-by-token decoding, prompts fed in portions, unequal batches, pages, slots and state rows used again, keys on either
side of every window's edge and on the pages' borders, the convolution's edge, states carried from the first token, the
values that one layer lends to the others, long decoding, generation through the entry point."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

from helpers import TOL
from plain import memipel_plain as M
from memipel_helpers import (MEM_A, MEM_MIX, assert_rows_close as assert_close, attention, clear_tokens, config, dense, latent,
                             layer, lightning, make, moe, plain_logits)

pytestmark = pytest.mark.gpu
DTYPES = ["float32", "bfloat16"]


def _td(dtype):
    return torch.float32 if dtype == "float32" else torch.bfloat16


def _engine(path, dtype, max_tokens=2048):
    from stratum_b200.engine import Engine, load_model
    model, _ = load_model(path, _td(dtype), "cuda")
    return Engine(model, max_tokens=max_tokens)


@pytest.fixture(scope="module", params=[(n, d) for n in ("A", "B", "TC", "BIG") for d in DTYPES],
                ids=lambda p: f"{p[0]}-{p[1]}")
def setup(request, tmp_path_factory):
    name, dtype = request.param
    path, cfg, w = make(str(tmp_path_factory.mktemp(f"mem{name}_{dtype}")), name, dtype, seed=len(name) + 1)
    return name, dtype, cfg, w, _engine(path, dtype), path


def _dev(a, dtype=torch.float32):
    return torch.from_numpy(np.ascontiguousarray(a)).to(dtype).cuda()


def _i32(a):
    return _dev(np.asarray(a), torch.int32)


def _tokens(rng, n, cfg):
    return [int(t) for t in rng.integers(0, cfg["vocab"], n)]


def _bf16(a):
    """The nearest bfloat16 values, as float64."""
    return torch.from_numpy(np.ascontiguousarray(a)).to(torch.bfloat16).double().numpy()


class _Step:
    """The fields of a step's description that a recurrent mixer's kernels read."""

    def __init__(self, n_new, before, slots):
        self.n_new = n_new
        self.token_pos = _i32(np.concatenate([np.arange(b, b + n) for b, n in zip(before, n_new)]))
        self.token_seq = _i32(np.concatenate([np.full(n, i if s >= 0 else -1) for i, (n, s) in enumerate(zip(n_new, slots))]))
        self.seq_start = _i32(np.concatenate([[0], np.cumsum(n_new)]))
        self.seq_slot = _i32([s if s >= 0 else 0 for s in slots])

    def runs(self, size):
        rows, r = [], 0
        for i, n in enumerate(self.n_new):
            rows += [(i, r + b, min(size, n - b)) for b in range(0, n, size)]
            r += n
        rows.append((-1, 0, 0))                              # a list of fixed length may hold entries without tokens
        return tuple(_i32(c) for c in zip(*rows))


# ------------------------------------------------------------------------------------------ kernels alone
@pytest.mark.parametrize("heads,kv,dim,vdim,taps", [(4, 2, 24, 16, 3), (3, 1, 18, 10, 6), (4, 2, 7, 5, 0), (2, 2, 15, 5, 1), (8, 1, 64, 64, 4),
                                                    (2, 1, 8, 20, 2), (6, 2, 12, 8, 12), (5, 5, 4, 4, 1), (4, 4, 128, 32, 4), (2, 1, 8, 8, 0)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_short_convolution_kernel(heads, kv, dim, vdim, taps, dtype):
    """Three sequences of unequal lengths in steps of many tokens, a few and one each, with a row of no sequence between
    them: convolved queries, the caches' rows, lent and mixed values, the inputs kept."""
    from stratum_b200 import kernels as K
    rng = np.random.default_rng(dim + taps)
    td = _td(dtype)
    r = _bf16 if dtype == "bfloat16" else (lambda a: a)
    nq, nk, nv = heads * dim, kv * dim, kv * vdim
    C = nq + nk + nv
    lens = (150, 40, 14)
    u = [rng.standard_normal((n, C)) for n in lens]
    first = [r(rng.standard_normal((n, nv))) for n in lens]
    cw, lam = rng.uniform(-0.8, 0.8, (C, taps)), 0.3
    y = [M.short_conv(x, cw) if taps else x for x in u]
    mixed = [(1 - lam) * a[:, nq + nk:] + lam * f for a, f in zip(y, first)]
    pages = [[5, 0, 7], [2, 0, 0], [3, 0, 0]]
    tables = _i32(pages)
    kc = torch.zeros(9, kv, 64, dim, dtype=td, device="cuda")
    vc = torch.zeros(9, kv, 64, vdim, dtype=td, device="cuda")
    state = torch.zeros(6, max(taps - 1, 0) * C + 4, device="cuda")
    state[5] = 7.0
    conv_w = _dev(cw.T) if taps else None
    slots, done, got, lent = [3, 0, 4], [0, 0, 0], [[], [], []], [[], [], []]
    pad = lambda n: (n + 7) // 8 * 8                                                             # noqa: E731
    for cut in ((120, 20, 2), (2, 5, 1), (1, 1, 1), (1, 1, 1), (9, 2, 3), (1, 1, 1), None, (1, 1, 1)):
        live = (0, 1, 2)
        at = list(done)
        if cut is None:                                      # the second row belongs to nobody
            cut, live, at[1] = (1, 1, 1), (0, 2), 0
        step = _Step(list(cut), at, [s if i in live else -1 for i, s in enumerate(slots)])
        rows = np.concatenate([u[i][at[i]:at[i] + cut[i]] for i in range(3)])
        T = rows.shape[0]
        p = torch.zeros(T, pad(C), device="cuda")
        p[:, :C] = _dev(rows)
        q = torch.full((T, pad(nq)), 3.0, dtype=td, device="cuda")
        fi = torch.zeros(T, pad(nv), dtype=td, device="cuda")
        fi[:, :nv] = _dev(np.concatenate([first[i][at[i]:at[i] + cut[i]] for i in range(3)]), td)
        fo = torch.zeros(T, pad(nv), dtype=td, device="cuda")
        runs = None if all(n == 1 for n in cut) else step.runs(max(8, taps - 1))
        before = state.clone()
        for writes in (False, True):                         # told not to write, it leaves caches and state alone
            K.short_conv(p[:, :C], conv_w, step, runs, state if taps > 1 else None, tables, q, kc, vc, heads, kv, dim, vdim, 64,
                         writes, _dev([lam]), fi, fo)
            assert writes or torch.equal(before, state)
        o, f, row = q[:, :nq].double().cpu().numpy(), fo[:, :nv].double().cpu().numpy(), 0
        for i in range(3):
            if i in live:
                got[i].append(o[row:row + cut[i]]); lent[i].append(f[row:row + cut[i]])
                done[i] += cut[i]
            row += cut[i]
    tol = 3e-6 if dtype == "float32" else 5e-3
    close = lambda a, b: np.max(np.abs(a - b)) <= tol * np.max(np.abs(b))                        # noqa: E731
    for i in range(3):
        n = done[i]
        assert close(np.concatenate(got[i]), y[i][:n, :nq]) and close(np.concatenate(lent[i]), mixed[i][:n]), i
        for t in range(n):
            page = pages[i][t // 64]
            assert close(kc[page, :, t % 64].double().cpu().numpy().reshape(-1), y[i][t, nq:nq + nk]), (i, t)
            assert close(vc[page, :, t % 64].double().cpu().numpy().reshape(-1), mixed[i][t]), (i, t)
        if taps > 1:
            kept = state[slots[i], :(taps - 1) * C].double().cpu().numpy().reshape(taps - 1, C)
            assert np.max(np.abs(kept - u[i][n - taps + 1:n])) <= 1e-6 * np.max(np.abs(kept))
    assert float(state[[1, 2]].abs().max()) == 0.0 and bool((state[5] == 7.0).all())
    assert float(state[:5, max(taps - 1, 0) * C:].abs().max()) == 0.0


@pytest.mark.parametrize("heads,dim,vdim", [(3, 12, 20), (2, 40, 8), (1, 9, 7), (4, 64, 32), (2, 130, 70), (1, 260, 8), (2, 128, 128),
                                            (2, 256, 36), (1, 208, 100), (3, 16, 4)])
@pytest.mark.parametrize("form", ["tokens", "chunks"])
@pytest.mark.parametrize("dtype", DTYPES)
def test_lightning_kernels(heads, dim, vdim, form, dtype):
    """Recurrence behind silu and the norm over all heads, on projections made here: two sequences of unequal lengths whose
    tokens come in four steps, in slots that lie apart; token by token, and in chunks where sizes allow."""
    from stratum_b200 import kernels as K
    if form == "chunks" and (dim % 16 or dim > 256):
        pytest.skip("sizes the chunked form does not take")
    rng = np.random.default_rng(dim + vdim)
    HD, HV = heads * dim, heads * vdim
    lens = (213, 11)
    proj = [rng.standard_normal((n, 2 * HD + 2 * HV)) * 1.5 for n in lens]
    decay, gain, eps = [0.999, 0.6, 0.97, 1.0][:heads], rng.uniform(0.5, 1.5, HV), 0.2
    want = []
    for p in proj:
        q, k, v = (M.silu(p[:, a:b]).reshape(len(p), heads, -1) for a, b in ((0, HD), (HD, 2 * HD), (2 * HD, 2 * HD + HV)))
        o = M.lightning_read(q, k, v, decay)[0].reshape(len(p), HV)
        want.append(M.rms_norm(o, gain, eps) * M.sigmoid(p[:, 2 * HD + HV:]))
    st = torch.zeros(6, HD * vdim + 4, device="cuda")
    slots, done, got = (4, 1), [0, 0], [[], []]
    for cut in ((lens[0] - 5, 7), (1, 1), (3, 2), (1, 1)):
        rows = np.concatenate([proj[i][done[i]:done[i] + cut[i]] for i in range(2)])
        T = rows.shape[0]
        seq = np.concatenate([np.full(cut[i], i) for i in range(2)])
        ld = (rows.shape[1] + 7) // 8 * 8
        pd = torch.zeros(T, ld, device="cuda")
        pd[:, :rows.shape[1]] = _dev(rows)
        g = K.GlaStep(pd, heads, dim, vdim, 0, 1.0, 1.0, eps, head_decay=_dev(decay), silu_qkv=True, norm_all=True)
        o_raw = torch.empty(T, HV, device="cuda")
        out = torch.empty(T, (HV + 7) // 8 * 8, dtype=_td(dtype), device="cuda")
        if form == "chunks":
            assert g.chunks_ok()
        g.recur(o_raw, st, _i32(seq), _i32([0, cut[0], T]), _i32(slots), True, chunked=form == "chunks")
        g.finish(_dev(gain), out)
        o = out[:, :HV].double().cpu().numpy()
        got[0].append(o[:cut[0]]); got[1].append(o[cut[0]:])
        done = [done[i] + cut[i] for i in range(2)]
    tol = 1e-4 if dtype == "float32" else 6e-3
    for i in range(2):
        o = np.concatenate(got[i])
        assert np.isfinite(o).all()
        assert np.max(np.abs(o - want[i])) <= tol * np.max(np.abs(want[i])), (i, np.max(np.abs(o - want[i])))
    assert float(st[0].abs().max()) == 0.0 and float(st[5].abs().max()) == 0.0            # rows of nobody stay clean
    assert float(st[:, HD * vdim:].abs().max()) == 0.0                                    # nothing beyond a state


@pytest.mark.parametrize("M_,N,K_,split", [(1, 192, 72, 40), (5, 320, 128, 96), (8, 64, 264, 8), (17, 1024, 256, 200), (64, 2048, 512, 1000),
                                           (100, 768, 1024, 384), (150, 512, 256, 1), (300, 4096, 192, 1504), (2100, 512, 128, 255)])
def test_two_limits_in_one_product(M_, N, K_, split):
    """Pairs of gate and up with one limit up to an output column and another from it on, through every kernel that serves
    such shapes."""
    from stratum_b200 import kernels as K
    from stratum_b200.parts.base import Runtime
    from stratum_b200.parts.linear import SWIGLU, Linear
    rng = np.random.default_rng(M_)
    x, w = _bf16(rng.standard_normal((M_, K_))), _bf16(rng.standard_normal((N, K_)) * 3 / np.sqrt(K_))
    s = x @ w.T
    limit = np.where(np.arange(N // 2) < split, 1.3, 0.5)
    g, up = np.minimum(s[:, 0::2], limit), np.clip(s[:, 1::2], -limit, limit)
    want = g * M.sigmoid(1.702 * g) * (up + 1)
    for dt, tol in ((torch.float32, 2e-5), (torch.bfloat16, 2e-2)):
        got = Linear(Runtime(dt, "cuda"), _dev(w, dt))(_dev(x, dt), mode=SWIGLU, act=K.ACT_CLAMPED_GATE, limit=(1.3, split, 0.5))
        assert np.max(np.abs(got.double().cpu().numpy() - want)) <= tol * np.max(np.abs(want))


@pytest.mark.parametrize("E,top,count,keep,width", [(6, 2, 3, 2, 72), (8, 3, 2, 1, 70), (5, 1, 1, 1, 33), (16, 4, 8, 4, 128), (64, 8, 8, 3, 256),
                                                    (12, 12, 4, 4, 64), (256, 8, 4, 2, 512)])
def test_routing_by_the_groups_largest_scores(E, top, count, keep, width):
    from stratum_b200 import kernels as K
    rng = np.random.default_rng(E)
    T = 40
    x, w = rng.standard_normal((T, width)), rng.standard_normal((E, width)) * 2 / np.sqrt(width)
    want = M.route(x @ w.T, top, count, keep)
    assert M.route_margin(x @ w.T, top, count, keep) > 1e-5
    if 1 < keep < count:                                     # the rule is told apart from the sum of a group's two largest
        s = np.exp(x @ w.T).reshape(T, count, -1)
        sums = np.sort(s, axis=-1)[:, :, -2:].sum(-1)
        assert any(set(np.argsort(-sums[t])[:keep]) != set(np.argsort(-s.max(-1)[t])[:keep]) for t in range(T))
    dense_ = torch.empty(T, E, device="cuda")
    chosen, weights = torch.empty(T, top, dtype=torch.int32, device="cuda"), torch.empty(T, top, device="cuda")
    K.moe_route(_dev(x), _dev(w), None, dense_, chosen, weights, top, count, keep, 1.0, softmax=True, renorm=False, group_max=True)
    got = dense_.double().cpu().numpy()
    assert np.max(np.abs(got - want)) <= 1e-5 and ((got > 0) == (want > 0)).all()
    assert np.allclose(np.take_along_axis(got, chosen.cpu().numpy().astype(np.int64), 1), weights.cpu().numpy())


def _softmax(q, k, v, vis, scale, slope, sink):
    T, H, _ = q.shape
    out = np.zeros((T, H, v.shape[2]))
    back = np.arange(T)[:, None] - np.arange(T)[None, :]
    for h in range(H):
        g = h // (H // k.shape[1])
        s = q[:, h] @ k[:, g].T * scale - (0.0 if slope is None else slope[h]) * back
        out[:, h] = M.softmax_read(s, vis, v[:, g], None if sink is None else sink[h])
    return out.reshape(T, -1)


@pytest.mark.parametrize("H,Gk,D,Dv,window,sunk", [(4, 2, 12, 20, 50, False), (3, 3, 20, 22, 5, True), (8, 1, 64, 64, 130, False), (4, 4, 32, 48, 64, True),
                                                   (4, 2, 128, 128, 100, False), (2, 1, 64, 64, 1, False), (20, 1, 32, 32, 77, False), (8, 2, 64, 64, 0, False),
                                                   (2, 2, 128, 128, 64, False), (16, 4, 64, 64, 65, False), (6, 6, 40, 24, 0, True)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_attention_with_distance_biases_over_windows(H, Gk, D, Dv, window, sunk, dtype):
    """A paged cache whose pages lie in no order, queries at every position in blocks (prompt) and single queries at chosen
    positions (decode steps, cut into ranges), steep and faint slopes, with and without sinks, against the softmax written
    out."""
    from stratum_b200 import kernels as K
    from stratum_b200.parts.attention_dispatch import _plain_heads, plan_general_splits
    rng = np.random.default_rng(H + D)
    td = _td(dtype)
    T = 333
    r = _bf16 if dtype == "bfloat16" else (lambda a: a)
    q, k, v = r(rng.standard_normal((T, H, D))), r(rng.standard_normal((T, Gk, D))), r(rng.standard_normal((T, Gk, Dv)))
    scale, slope = 1.5 / np.sqrt(D), M.slopes(H)
    if H > 1:
        slope[0] = 3.0                                       # only the nearest keys count for this head
    sink = rng.uniform(-1, 3, H) if sunk else None
    vis = M.visible(T, window)
    want = _softmax(q, k, v, vis, scale, slope, sink)
    pages = [7, 2, 9, 4, 0, 5]
    kc, vc = np.zeros((10, Gk, 64, D)), np.zeros((10, Gk, 64, Dv))
    for t in range(T):
        kc[pages[t // 64], :, t % 64], vc[pages[t // 64], :, t % 64] = k[t], v[t]
    kc, vc = _dev(kc, td), _dev(vc, td)
    shape = K.AttentionShape(H, H // Gk, 1, D, Dv, False, scale, window=window, slope=_dev(slope),
                             sink=None if sink is None else _dev(sink))
    bt = _i32([pages])
    tol = 2e-5 if dtype == "float32" else 1e-2

    def run(rows, single):
        n = len(rows)
        qd = torch.zeros(n, (H * D + 7) // 8 * 8, dtype=td, device="cuda")
        qd[:, :H * D] = _dev(q[rows].reshape(n, H * D), td)
        out = torch.zeros(n, (H * Dv + 7) // 8 * 8, dtype=td, device="cuda")
        pos = _i32(rows)
        if single:                                           # every row a sequence of its own, over the same pages
            tables, seq = bt.repeat(n, 1), _i32(np.arange(n))
        else:
            tables, seq = bt, torch.zeros(n, dtype=torch.int32, device="cuda")
        if K.attention_general_mma_ok(shape, qd, out, 64):
            if single:
                streams = Gk * ((H // Gk + 15) // 16)
                for splits, per in (plan_general_splits(n * streams, T, shape.span), (6, 64), (2, 192)):
                    po = torch.empty(n * H * splits * Dv, device="cuda")
                    ml = torch.empty(n * H * splits * 2, device="cuda")
                    out.zero_()
                    K.attention_general_mma(shape, qd, kc, vc, pos, seq, tables, out, 64, None, 16 // min(H // Gk, 16), splits,
                                            per, po, ml, 1)
                    yield out[:, :H * Dv].double().cpu().numpy()
            else:
                per_block = 16 // min(H // Gk, 16)
                for groups in (1, 2):
                    b = per_block * groups
                    starts = np.arange(0, n, b)
                    qb = (torch.zeros(len(starts), dtype=torch.int32, device="cuda"), _i32(starts), _i32(np.minimum(b, n - starts)))
                    out.zero_()
                    K.attention_general_mma(shape, qd, kc, vc, pos, seq, tables, out, 64, qb, per_block, 1, 384, None, None, groups)
                    yield out[:, :H * Dv].double().cpu().numpy()
        if not single and _plain_heads(shape, qd, None, out, None):                    # the tcgen05 kernel
            b = 2 * (128 // (H // Gk))
            starts = np.arange(0, n, b)
            qb = (torch.zeros(len(starts), dtype=torch.int32, device="cuda"), _i32(starts), _i32(np.minimum(b, n - starts)))
            out.zero_()
            K.attention_tc(qd, kc, vc, pos, bt, qb, out, H, Gk, D, 64, window, scale, halves=2, split=True, slope=shape.slope)
            K.check_status()
            got = out[:, :H * Dv].double().cpu().numpy()
            assert np.max(np.abs(got - want)) <= 5e-3 * np.max(np.abs(want))        # (the output's rounding alone)
            yield got
        out.zero_()
        K.attention_general(shape, qd, kc, vc, pos, seq, tables, out, 64)
        yield out[:, :H * Dv].double().cpu().numpy()

    for got in run(np.arange(T), False):
        assert np.max(np.abs(got - want)) <= tol * np.max(np.abs(want))
    rows = sorted({0, 1, max(window - 1, 0), window, window + 1, 63, 64, 65, 255, 256, T - 1})
    for got in run(np.asarray(rows), True):
        assert np.max(np.abs(got - want[rows])) <= tol * np.max(np.abs(want))


# ------------------------------------------------------------------------------------------ mechanisms alone
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["attention", "mix", "latent", "lightning", "moe", "dense"])
def test_each_mechanism_alone(name, dtype, tmp_path):
    from stratum_b200.engine import StepEntry
    path, cfg, w = make(str(tmp_path / name), name, dtype, seed=3)
    engine = _engine(path, dtype)
    rng = np.random.default_rng(1)
    for n in (1, 2, 7, 100):
        toks = clear_tokens(rng, n, cfg, w, dtype)
        slot = engine.acquire()
        got = engine.step([StepEntry(slot, toks, list(range(n)))]).cpu().numpy()
        engine.release(slot)
        assert_close(got, plain_logits(cfg, w, toks), dtype, f"{name} n={n}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_model_of_what_may_be_left_out(dtype, tmp_path):
    """Convolution, mixing, windows, groups, shared experts and feed-forwards left out: they do not exist."""
    import copy
    from stratum_b200.engine import StepEntry
    raw = copy.deepcopy(MEM_A)
    for key in ("conv", "v_mix", "mask"):
        del raw["layers"][2]["mixer"][key]
    del raw["layers"][3]["mixer"]["mask"]
    del raw["layers"][0]["mlp"]["router"]["groups"]
    del raw["layers"][0]["mlp"]["shared"]
    raw["layers"][1]["mlp"] = None
    path, cfg, w = make(str(tmp_path / "bare"), None, dtype, seed=12, cfg=raw)
    engine = _engine(path, dtype)
    toks = clear_tokens(np.random.default_rng(0), 90, cfg, w, dtype)
    ref = plain_logits(cfg, w, toks)
    slot = engine.acquire()
    got = engine.step([StepEntry(slot, toks[:70], list(range(70)))]).cpu().numpy()
    got = np.concatenate([got] + [engine.step([StepEntry(slot, [t], [0])]).cpu().numpy() for t in toks[70:]])
    engine.release(slot)
    assert_close(got, ref, dtype, "a bare model")


def test_the_stream_after_every_layer(tmp_path):
    from stratum_b200.engine import StepEntry
    path, cfg, w = make(str(tmp_path / "streams"), "A", "float32", seed=5)
    engine = _engine(path, "float32")
    seen = []
    for lay in engine.model.layers:
        def wrapped(layer_, x, step, cache, _f=lay.arrangement.forward, **kw):
            out = _f(layer_, x, step, cache, **kw)
            seen.append(x.cpu().numpy().copy())
            return out
        lay.arrangement.forward = wrapped
    toks = clear_tokens(np.random.default_rng(0), 60, cfg, w, "float32")
    slot = engine.acquire()
    engine.step([StepEntry(slot, toks, [59])])
    engine.release(slot)
    want = []
    M.forward(cfg, w, toks, want)
    assert len(seen) == len(want) == 6
    for i, (a, b) in enumerate(zip(seen, want)):
        assert np.max(np.abs(a - b)) <= 2e-5 * np.max(np.abs(b)), i


@pytest.mark.parametrize("name", ["TC", "latent", "BIG"])
def test_latent_attention_both_forms(name, tmp_path, monkeypatch):
    """bfloat16 prompts from position 0 form the heads' keys and values (from 256 tokens on; here from 32 on), everything
    else carries the queries into the latent space and attends over the cached rows, over windows and with sinks: both
    against the plain implementation, and decoded tokens read the cache that either form wrote."""
    from stratum_b200.engine import StepEntry
    from stratum_b200.parts import latent_attention as L
    path, cfg, w = make(str(tmp_path / name), name, "bfloat16", seed=8)
    engine = _engine(path, "bfloat16")
    rng = np.random.default_rng(12)
    prompts = [clear_tokens(rng, n, cfg, w, "bfloat16") for n in (190, 70, 41)]
    refs = [plain_logits(cfg, w, p) for p in prompts]
    for minimum in (32, 1 << 30):
        monkeypatch.setattr(L, "PER_HEAD_MIN_TOKENS", minimum)
        slots = [engine.acquire() for _ in prompts]
        cut = [len(p) - 3 for p in prompts]
        out = engine.step([StepEntry(s, p[:c], list(range(c))) for s, p, c in zip(slots, prompts, cut)]).cpu().numpy()
        at = 0
        for i, c in enumerate(cut):
            assert_close(out[at:at + c], refs[i][:c], "bfloat16", f"{name} form {minimum} prompt {i}")
            at += c
        for k in range(3):
            out = engine.step([StepEntry(s, [p[c + k]], [0]) for s, p, c in zip(slots, prompts, cut)]).cpu().numpy()
            for i, c in enumerate(cut):
                assert_close(out[i], refs[i][c + k], "bfloat16", f"{name} form {minimum} seq {i} +{k}")
        for s in slots:
            engine.release(s)


def test_experts_both_ways(tmp_path, monkeypatch):
    """All experts stacked into one product, and each on its own gathered rows: limits, groups, the shared expert's limit."""
    from stratum_b200.engine import StepEntry
    from stratum_b200.parts import moe as R
    for dtype in DTYPES:
        path, cfg, w = make(str(tmp_path / dtype), "TC", dtype, seed=3)
        engine = _engine(path, dtype)
        toks = clear_tokens(np.random.default_rng(3), 200, cfg, w, dtype)
        ref = plain_logits(cfg, w, toks)
        for least in (0, 1 << 30):
            monkeypatch.setattr(R, "GROUPED_MIN_ROWS", least)
            slot = engine.acquire()
            got = engine.step([StepEntry(slot, toks, list(range(200)))]).cpu().numpy()
            engine.release(slot)
            assert_close(got, ref, dtype, f"experts, rows from {least}")


# ------------------------------------------------------------------------------------------ whole models
def test_whole_prompt_all_positions(setup):
    from stratum_b200.engine import StepEntry
    name, dtype, cfg, w, engine, _ = setup
    rng = np.random.default_rng(1)
    for n in (1, 2, 3, 5, 6, 63, 64, 65, 300):
        toks = clear_tokens(rng, n, cfg, w, dtype)
        slot = engine.acquire()
        got = engine.step([StepEntry(slot, toks, list(range(n)))]).cpu().numpy()
        engine.release(slot)
        assert_close(got, plain_logits(cfg, w, toks), dtype, f"{name} whole n={n}")
    engine.cache.check()


def test_prefill_against_token_by_token(setup):
    """The same tokens whole, and one by one from the first: the same logits (float32: to rounding)."""
    from stratum_b200.engine import StepEntry
    name, dtype, cfg, w, engine, _ = setup
    n = 150
    toks = clear_tokens(np.random.default_rng(2), n, cfg, w, dtype)
    a, b = engine.acquire(), engine.acquire()
    whole = engine.step([StepEntry(a, toks, list(range(n)))]).cpu().numpy()
    single = np.concatenate([engine.step([StepEntry(b, [t], [0])]).cpu().numpy() for t in toks])
    engine.release(a); engine.release(b)
    ref = plain_logits(cfg, w, toks)
    assert_close(whole, ref, dtype, f"{name} whole")
    assert_close(single, ref, dtype, f"{name} one by one")
    if dtype == "float32":
        assert np.max(np.abs(whole - single)) <= 2e-5 * np.max(np.abs(ref))


def test_the_same_bits_every_run(setup):
    """A batch of prompts and some decoded tokens, three times over in slots, pages and state rows that were just given
    back: every run's logits are the same bits."""
    from stratum_b200.engine import StepEntry
    name, dtype, cfg, w, engine, _ = setup
    rng = np.random.default_rng(17)
    prompts = [_tokens(rng, n, cfg) for n in (90, 7, 64, 33)]
    more = [_tokens(rng, 6, cfg) for _ in prompts]
    runs = []
    for _ in range(3):
        slots = [engine.acquire() for _ in prompts]
        got = [engine.step([StepEntry(s, p, list(range(len(p)))) for s, p in zip(slots, prompts)]).cpu().numpy()]
        for i in range(6):
            got.append(engine.step([StepEntry(s, [m[i]], [0]) for s, m in zip(slots, more)]).cpu().numpy())
        for s in slots:
            engine.release(s)
        runs.append(np.concatenate(got))
    assert np.isfinite(runs[0]).all()
    assert np.array_equal(runs[0], runs[1]) and np.array_equal(runs[0], runs[2]), f"{name} {dtype}: runs differ"


@pytest.mark.parametrize("portion", [2, 3, 31, 64, 100])
def test_prompt_in_portions(setup, portion):
    """A prompt cut into portions of a few sizes, down to two tokens; portions start inside pages and windows and on their
    borders, and the convolutions reach back over the cuts (over several, where a portion is shorter than the taps)."""
    from stratum_b200.engine import StepEntry
    name, dtype, cfg, w, engine, _ = setup
    n = 150 if portion > 3 else 80
    toks = clear_tokens(np.random.default_rng(portion), n, cfg, w, dtype)
    ref = plain_logits(cfg, w, toks)
    slot = engine.acquire()
    got = [engine.step([StepEntry(slot, toks[i:i + portion], list(range(len(toks[i:i + portion]))))]).cpu().numpy()
           for i in range(0, n, portion)]
    engine.release(slot)
    assert_close(np.concatenate(got), ref, dtype, f"{name} portions of {portion}")


def test_unequal_batches_against_each_alone_slots_reused(setup):
    from stratum_b200.engine import StepEntry
    name, dtype, cfg, w, engine, _ = setup
    rng = np.random.default_rng(3)
    for batch_no, lens in enumerate([(5, 9, 12), (1, 67), (70, 3, 33, 64), tuple(range(1, 20))]):
        extra_n = [3 + (2 * i) % 9 for i in range(len(lens))]
        full = [clear_tokens(rng, n + k, cfg, w, dtype) for n, k in zip(lens, extra_n)]
        prompts = [f[:n] for f, n in zip(full, lens)]
        extra = [f[n:] for f, n in zip(full, lens)]
        refs = [plain_logits(cfg, w, f) for f in full]
        slots = [engine.acquire() for _ in lens]
        out = engine.step([StepEntry(s, p, [len(p) - 1]) for s, p in zip(slots, prompts)]).cpu().numpy()
        alone = []
        for p in prompts:                                   # each alone, where there is room beside the batch
            if len(lens) > 4:
                break
            s = engine.acquire()
            alone.append(engine.step([StepEntry(s, p, [len(p) - 1])]).cpu().numpy()[0])
            engine.release(s)
        for i, p in enumerate(prompts):
            assert_close(out[i], refs[i][len(p) - 1], dtype, f"{name} batch {batch_no} prompt {i}")
            if dtype == "float32" and alone:
                assert np.max(np.abs(out[i] - alone[i])) <= 2e-5 * np.max(np.abs(refs[i]))
        live, step = list(range(len(lens))), 0
        while live:
            out = engine.step([StepEntry(slots[i], [extra[i][step]], [0]) for i in live]).cpu().numpy()
            for row, i in enumerate(live):
                assert_close(out[row], refs[i][len(prompts[i]) + step], dtype, f"{name} batch {batch_no} seq {i} +{step}")
            step += 1
            for i in list(live):
                if step >= len(extra[i]):
                    engine.release(slots[i])
                    live.remove(i)
        engine.cache.check()
    assert engine.cache.tokens_held() == 0


def test_portions_and_single_tokens_in_one_step(setup):
    """A step in which one sequence starts, one goes on by a portion and one by a single token."""
    from stratum_b200.engine import StepEntry
    name, dtype, cfg, w, engine, _ = setup
    rng = np.random.default_rng(31)
    toks = [clear_tokens(rng, n, cfg, w, dtype) for n in (95, 140, 66)]
    refs = [plain_logits(cfg, w, t) for t in toks]
    s = [engine.acquire() for _ in toks]
    engine.step([StepEntry(s[1], toks[1][:77], []), StepEntry(s[2], toks[2][:64], [])])
    got = engine.step([StepEntry(s[2], toks[2][64:65], [0]), StepEntry(s[0], toks[0][:90], [0, 89]),
                       StepEntry(s[1], toks[1][77:], [0, 1, 62])]).cpu().numpy()
    want = np.stack([refs[2][64], refs[0][0], refs[0][89], refs[1][77], refs[1][78], refs[1][139]])
    assert_close(got, want, dtype, f"{name} mixed step")
    got = engine.step([StepEntry(s[0], toks[0][90:], [4]), StepEntry(s[2], toks[2][65:], [0])]).cpu().numpy()
    assert_close(got, np.stack([refs[0][94], refs[2][65]]), dtype, f"{name} the step after")
    for x in s:
        engine.release(x)


def test_pages_and_slots_used_again(setup):
    """A cache of four pages and few slots: every request takes pages and state rows that another one has just given
    back."""
    from stratum_b200.engine import StepEntry
    name, dtype, cfg, w, _, path = setup
    engine = _engine(path, dtype, max_tokens=256)
    rng = np.random.default_rng(4)
    held = []
    for n in (130, 60, 190, 64, 129):
        while held and sum((engine.length(s) + 63) // 64 for s in held) + (n + 63) // 64 > 4:
            engine.release(held.pop(0))
        toks = clear_tokens(rng, n, cfg, w, dtype)
        slot = engine.acquire()
        got = engine.step([StepEntry(slot, toks[:-1], [n - 2])]).cpu().numpy()
        got = np.concatenate([got, engine.step([StepEntry(slot, toks[-1:], [0])]).cpu().numpy()])
        assert_close(got, plain_logits(cfg, w, toks)[-2:], dtype, f"{name} reuse n={n}")
        held.append(slot)
        engine.cache.check()


def test_first_tokens_and_long_decoding(setup):
    """Positions 0, 1, 2 one by one, then on across several pages and windows; a windowed layer gives back the pages that
    lie in front of its window."""
    from stratum_b200.engine import StepEntry
    name, dtype, cfg, w, engine, _ = setup
    n = 270
    toks = clear_tokens(np.random.default_rng(5), n, cfg, w, dtype)
    ref = plain_logits(cfg, w, toks)
    slot = engine.acquire()
    check = {0, 1, 2, 3, 4, 5, 6} | set(range(7, n, 29)) | {63, 64, 65, 127, 128, 129, 191, 192, 193, 255, 256, 257, n - 1}
    got = []
    for i in range(n):
        out = engine.step([StepEntry(slot, [toks[i]], [0] if i in check else [])])
        if i in check:
            got.append(out.cpu().numpy())
    for gi, g in enumerate(engine.cache.groups):
        if g.pool is not None and g.spec.window:
            held = sum(p >= 0 for p in engine.cache.page_table_rows([slot], gi)[0])
            assert held <= (g.spec.window + 126) // 64
    engine.release(slot)
    assert_close(np.concatenate(got), ref[sorted(check)], dtype, f"{name} long decode")
    engine.cache.check()
    assert engine.cache.tokens_held() == 0


# ------------------------------------------------------------------------------------------ one token decides
def _marked_key_model(path, dtype, form):
    """One layer in which token 7 is the only one with anything in the embedding's first dimension, and token 8 the only
    one with anything in the second.  One dimension of every key reads the first (through the latent, where there is one)
    and nothing else, the same dimension of every query reads the second: when token 8 asks, the marked key's score stands
    far above the hundreds of others wherever it lies, and the heads' outputs are its value.  The convolutions, which have
    tests of their own, hand on the current token alone."""
    mixer = {"small": attention(heads=4, kv=2, dim=16, vdim=24, scale=0.25, conv=3, size=45),
             "mma": attention(heads=8, kv=1, dim=32, vdim=48, scale=0.15, conv=4, size=130),
             "wide": attention(heads=4, kv=2, dim=64, vdim=64, scale=0.1, conv=2, size=100),
             "latent": latent(heads=3, dim=16, vdim=24, q_rank=24, kv_rank=40, scale=0.3, size=70),
             "latent odd": latent(heads=2, dim=9, vdim=5, q_rank=11, kv_rank=21, scale=0.5, size=33)}[form]
    kind = "latent_attention" if form.startswith("latent") else "attention"
    cfg_raw = config([layer(kind, mixer)], vocab=120, width=64)
    H, D = mixer["heads"], mixer["dim"]

    def edit(t):
        e = t["embed"].float()
        e[:, :2] = 0.0
        e[7, 0] = e[8, 1] = 24.0
        t["embed"] = e.to(t["embed"].dtype)
        t["l0.norm1"] = torch.zeros_like(t["l0.norm1"])
        t["l0.mix.o"] = (t["l0.mix.o"].float() * (30 if form == "latent odd" else 8)).to(t["l0.mix.o"].dtype)

        def only(name, row, col, value):
            m = t[name].float()
            m[row] = 0.0
            m[row, col] = value
            t[name] = m.to(t[name].dtype)
        if kind == "attention":
            for name, heads, col in (("l0.mix.k", mixer["kv_heads"], 0), ("l0.mix.q", H, 1)):
                m = t[name].float()
                m[:, :2] = 0.0
                t[name] = m.to(t[name].dtype)
                for h in range(heads):
                    only(name, h * D + D - 1, col, 8.0)
            for name in ("q", "k", "v"):
                c = torch.zeros_like(t[f"l0.mix.{name}.conv"])
                c[:, -1] = 1.0
                t[f"l0.mix.{name}.conv"] = c
                t[f"l0.mix.{name}.b"] = torch.zeros_like(t[f"l0.mix.{name}.b"])
        else:
            for name, col in (("l0.mix.dkv", 0), ("l0.mix.dq", 1)):
                m = t[name].float()
                m[:, :2] = 0.0
                t[name] = m.to(t[name].dtype)
                only(name, 0, col, 8.0)
                t[name + ".norm"] = torch.ones_like(t[name + ".norm"])
            for name in ("l0.mix.uk", "l0.mix.uq"):
                for h in range(H):
                    only(name, h * D + D - 1, 0, 3.0)
    return make(path, None, dtype, seed=9, edit=edit, cfg=cfg_raw)


def _three_forms(engine, toks, dtype, ref, what, first=201):
    """The last token's logits as a whole prompt, as the last token of a prompt's second portion, and decoded alone
    after a few decoded tokens."""
    from stratum_b200.engine import StepEntry
    n = len(toks)
    slot = engine.acquire()
    whole = engine.step([StepEntry(slot, toks, [n - 1])]).cpu().numpy()[0]
    engine.release(slot)
    slot = engine.acquire()
    first = min(first, n - 2)
    engine.step([StepEntry(slot, toks[:first], [])])
    cut = engine.step([StepEntry(slot, toks[first:], [n - first - 1])]).cpu().numpy()[0]
    engine.release(slot)
    slot = engine.acquire()
    engine.step([StepEntry(slot, toks[:n - 4], [])])
    for t in toks[n - 4:n - 1]:
        engine.step([StepEntry(slot, [t], [])])
    decoded = engine.step([StepEntry(slot, toks[n - 1:], [0])]).cpu().numpy()[0]
    engine.release(slot)
    assert_close(whole, ref, dtype, f"{what}, whole")
    assert_close(cut, ref, dtype, f"{what}, second portion")
    assert_close(decoded, ref, dtype, f"{what}, decoded")


@pytest.mark.parametrize("form", ["small", "mma", "wide", "latent", "latent odd"])
@pytest.mark.parametrize("dtype", DTYPES)
def test_keys_just_inside_and_just_outside_the_windows(dtype, form, tmp_path):
    """A marked key at the last place a window reaches decides the logits; one place further out it changes nothing (both
    shown on the plain implementation).  The asking token stands before, on and behind pages' borders, and where the
    window still holds everything; prompts of more than 256 tokens take latent attention's other form."""
    path, cfg, w = _marked_key_model(str(tmp_path / "edge"), dtype, form)
    size = cfg["layers"][0]["mixer"]["mask"]["size"]
    engine = _engine(path, dtype)
    rng = np.random.default_rng(1)
    for n in (size, size + 1, 129, 192, 193, 257, 300):
        for back in (size - 1, size, 1, n - 1):
            if back >= n or (back == n - 1 and back in (size - 1, size)):
                continue
            toks = [int(x) for x in rng.integers(9, cfg["vocab"], n)]
            toks[-1] = 8
            toks[n - 1 - back] = 7
            ref = plain_logits(cfg, w, toks)[-1]
            moved = list(toks)
            moved[n - 1 - back] = 9
            changed = np.max(np.abs(plain_logits(cfg, w, moved)[-1] - ref)) / np.max(np.abs(ref))
            assert changed > 0.1 if back < size else changed < 1e-6, f"n={n}: the marked key {back} back changes the logits by {changed}"
            _three_forms(engine, toks, dtype, ref, f"n={n}, marked key {back} back", first=max(n - 1 - back, 1))
            if dtype == "float32" or back < size:
                _three_forms(engine, toks, dtype, ref, f"n={n}, marked key {back} back", first=64)


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_key_far_back_decides(dtype, tmp_path):
    """Without a window: the marked key 1, 63, 64, 65, 128 and 300 places back and at position 0, among 420 keys."""
    for name, mixer in (("attention", attention(heads=12, kv=4, dim=16, vdim=24, scale=0.25, conv=3, size=0)),
                        ("latent_attention", latent(heads=3, dim=16, vdim=24, q_rank=24, kv_rank=40, scale=0.3, size=0))):
        raw = config([layer(name, mixer)], vocab=120, width=64)
        H, D, n = mixer["heads"], mixer["dim"], 420

        def edit(t):
            e = t["embed"].float()
            e[:, :2] = 0.0
            e[7, 0] = e[8, 1] = 24.0
            t["embed"] = e.to(t["embed"].dtype)
            t["l0.norm1"] = torch.zeros_like(t["l0.norm1"])
            t["l0.mix.o"] = (t["l0.mix.o"].float() * 8).to(t["l0.mix.o"].dtype)
            pairs = ((("k", mixer.get("kv_heads"), 0), ("q", H, 1)) if name == "attention" else (("dkv", 1, 0), ("dq", 1, 1)))
            for key, heads, col in pairs:
                m = t["l0.mix." + key].float()
                m[:, :2] = 0.0
                for h in range(heads):
                    m[h * D + D - 1 if name == "attention" else 0] = 0.0
                    m[h * D + D - 1 if name == "attention" else 0, col] = 8.0
                t["l0.mix." + key] = m.to(t["l0.mix." + key].dtype)
            if name != "attention":
                for key in ("uk", "uq"):
                    m = t["l0.mix." + key].float()
                    for h in range(H):
                        m[h * D + D - 1] = 0.0
                        m[h * D + D - 1, 0] = 3.0
                    t["l0.mix." + key] = m.to(t["l0.mix." + key].dtype)
        path, cfg, w = make(str(tmp_path / name), None, dtype, seed=9, edit=edit, cfg=raw)
        engine = _engine(path, dtype)
        rng = np.random.default_rng(0)
        for back in (1, 63, 64, 65, 128, 300, n - 1):
            toks = [int(x) for x in rng.integers(9, cfg["vocab"], n)]
            toks[-1] = 8
            toks[n - 1 - back] = 7
            ref = plain_logits(cfg, w, toks)[-1]
            moved = list(toks)
            moved[n - 1 - back] = 9
            assert np.max(np.abs(plain_logits(cfg, w, moved)[-1] - ref)) > 0.1 * np.max(np.abs(ref)), (name, back)
            _three_forms(engine, toks, dtype, ref, f"{name}, {back} back")


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_sink_takes_its_share(dtype, tmp_path):
    """At a sequence's first token the only key competes with the sink: its value counts by e^s / (e^s + e^sink), which the
    sinks of this model make small for one head and nearly one for another."""
    from stratum_b200.engine import StepEntry
    raw = config([layer("latent_attention", latent(heads=2, dim=16, vdim=24, q_rank=24, kv_rank=40, size=30))], vocab=120, width=64)
    ref = {}
    for what, sinks in (("as they are", (6.0, -5.0)), ("turned", (-5.0, 6.0))):
        def edit(t):
            t["l0.mix.sink"] = torch.tensor(sinks).to(t["l0.mix.sink"].dtype)
            t["l0.mix.o"] = (t["l0.mix.o"].float() * 6).to(t["l0.mix.o"].dtype)
        path, cfg, w = make(str(tmp_path / what.replace(" ", "_")), None, dtype, seed=2, edit=edit, cfg=raw)
        engine = _engine(path, dtype)
        toks = _tokens(np.random.default_rng(3), 80, cfg)
        ref[what] = plain_logits(cfg, w, toks)
        slot = engine.acquire()
        got = engine.step([StepEntry(slot, toks[:60], list(range(60)))]).cpu().numpy()
        got = np.concatenate([got] + [engine.step([StepEntry(slot, [t], [0])]).cpu().numpy() for t in toks[60:]])
        assert_close(got, ref[what], dtype, f"sinks {what}")
    a, b = ref["as they are"], ref["turned"]
    assert (np.max(np.abs(a - b), axis=-1) > 0.1 * np.max(np.abs(a))).mean() > 0.9


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("taps", [4, 2, 9, 1])
def test_the_convolutions_edge(taps, dtype, tmp_path):
    """Attention that sees its own token alone hands on that token's convolved value: a marked token taps - 1 places back
    changes the logits, one place further out it does not, within a prompt, across the border of two steps (cut anywhere
    between the two, and in portions shorter than the taps) and for decoded tokens."""
    from stratum_b200.engine import StepEntry
    raw = config([layer("attention", attention(heads=2, kv=1, dim=8, vdim=12, conv=taps, size=1))], vocab=90, width=48)

    def edit(t):
        t["l0.mix.v.conv"] = torch.full_like(t["l0.mix.v.conv"], 0.8)
        t["l0.mix.o"] = (t["l0.mix.o"].float() * 6).to(t["l0.mix.o"].dtype)
        e = t["embed"].float()
        e[1] = torch.sign(e[1]) * 3.0
        t["embed"] = e.to(t["embed"].dtype)
    path, cfg, w = make(str(tmp_path / "conv"), None, dtype, seed=4, edit=edit, cfg=raw)
    engine = _engine(path, dtype)
    rng = np.random.default_rng(taps)
    n = 30
    for back in (taps - 1, taps):
        toks = [int(x) for x in rng.integers(2, 90, n)]
        toks[n - 1 - back] = 1
        ref = plain_logits(cfg, w, toks)
        moved = list(toks)
        moved[n - 1 - back] = 5
        changed = np.max(np.abs(plain_logits(cfg, w, moved)[-1] - ref[-1])) / np.max(np.abs(ref[-1]))
        assert changed > 0.03 if back < taps else changed < 1e-9, (back, changed)
        for cut in range(n - 1 - taps, n):
            slot = engine.acquire()
            engine.step([StepEntry(slot, toks[:cut], [])])
            got = engine.step([StepEntry(slot, toks[cut:], [n - 1 - cut])]).cpu().numpy()[0]
            engine.release(slot)
            assert_close(got, ref[-1], dtype, f"{taps} taps, marked {back} back, cut at {cut}")
        for portion in (1, 2, 3):
            slot = engine.acquire()
            got = [engine.step([StepEntry(slot, toks[i:i + portion], list(range(len(toks[i:i + portion]))))]).cpu().numpy()
                   for i in range(0, n, portion)]
            engine.release(slot)
            assert_close(np.concatenate(got), ref, dtype, f"{taps} taps, marked {back} back, portions of {portion}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("at", [0, 5, 63, 64])
@pytest.mark.parametrize("dim", [8, 16])
def test_the_state_carries_a_token_from_far_back(dim, at, dtype, tmp_path):
    """A layer that hardly forgets: hundreds of tokens later the output is still shaped by one marked token (shown on the
    plain implementation), through a prompt cut in two, a state row used before, and decoded tokens."""
    from stratum_b200.engine import StepEntry
    raw = config([layer("lightning", lightning(heads=2, dim=dim, vdim=12, decay=[1.0 - 2.0 ** -12, 1.0 - 2.0 ** -11]))], vocab=90, width=48)

    def edit(t):
        e = t["embed"].float()
        e[:, :2] = 0.0
        e[:, 1] = 0.5                                        # every token has the same second dimension
        e[1, 0] = 30.0                                       # the marked token alone has a first one
        t["embed"] = e.to(t["embed"].dtype)
        t["l0.mix.o"] = (t["l0.mix.o"].float() * 4).to(t["l0.mix.o"].dtype)
        for name, col in (("l0.mix.k", 0), ("l0.mix.q", 1)):       # keys read the first in one dimension, queries the second
            m = t[name].float()
            m[:, :2] = 0.0
            for h in range(2):
                m[h * dim + dim - 1] = 0.0
                m[h * dim + dim - 1, col] = 8.0
            t[name] = m.to(t[name].dtype)
    path, cfg, w = make(str(tmp_path / "state"), None, "float32", seed=4, edit=edit, cfg=raw) if dtype == "float32" else \
        make(str(tmp_path / "state"), None, dtype, seed=4, edit=edit, cfg=raw)
    toks = [int(t) for t in np.random.default_rng(1).integers(2, 90, 400)]
    toks[at] = 1
    ref = plain_logits(cfg, w, toks)
    other = list(toks)
    other[at] = 2
    assert np.max(np.abs(plain_logits(cfg, w, other)[-1] - ref[-1])) > 0.1 * np.max(np.abs(ref[-1]))
    engine = _engine(path, dtype)
    slot = engine.acquire()                                  # somebody else's state in the row first
    engine.step([StepEntry(slot, other[:90], [])])
    engine.release(slot)
    slot = engine.acquire()
    engine.step([StepEntry(slot, toks[:131], [])])
    got = engine.step([StepEntry(slot, toks[131:390], [258])]).cpu().numpy()
    got = np.concatenate([got] + [engine.step([StepEntry(slot, [t], [0])]).cpu().numpy() for t in toks[390:]])
    engine.release(slot)
    assert_close(got, ref[389:], dtype, "state from far back")


@pytest.mark.parametrize("dtype", DTYPES)
def test_the_first_layers_values_reach_the_later_ones(dtype, tmp_path):
    """The share decides how much of the first layer's values a later layer reads; the first layer's own share, and what
    lies in its cache, do nothing."""
    from stratum_b200.engine import StepEntry
    ref = {}
    for what, share in (("none", 0.0), ("all", 1.0), ("beyond", 1.6)):
        for first in (0.4, 5.0):
            def edit(t):
                t["l0.mix.vmix"] = torch.full_like(t["l0.mix.vmix"], first)
                t["l1.mix.vmix"] = torch.full_like(t["l1.mix.vmix"], share)
                t["l1.mix.o"] = (t["l1.mix.o"].float() * 4).to(t["l1.mix.o"].dtype)
            path, cfg, w = make(str(tmp_path / f"{what}{first}"), None, dtype, seed=7, edit=edit, cfg=MEM_MIX)
            toks = _tokens(np.random.default_rng(3), 90, cfg)
            logits = plain_logits(cfg, w, toks)
            assert what not in ref or np.array_equal(logits, ref[what])
            ref[what] = logits
            engine = _engine(path, dtype)
            slot = engine.acquire()
            got = [engine.step([StepEntry(slot, toks[a:b], list(range(b - a)))]).cpu().numpy() for a, b in ((0, 40), (40, 75))]
            got += [engine.step([StepEntry(slot, [t], [0])]).cpu().numpy() for t in toks[75:]]
            assert_close(np.concatenate(got), logits, dtype, f"share {share}")
    for a, b in (("none", "all"), ("all", "beyond")):
        assert np.max(np.abs(ref[a] - ref[b])) > 0.1 * np.max(np.abs(ref[a]))


# ------------------------------------------------------------------------------------------ generation
@pytest.mark.parametrize("name", ["A", "TC"])
@pytest.mark.parametrize("dtype", DTYPES)
def test_greedy_generation_through_the_entry_point(name, dtype, tmp_path):
    """Stratum.generate: the scheduler's batches, replayed decode graphs (with padding rows), slots given back; every
    picked token is the plain implementation's best (or within rounding of it)."""
    from stratum_b200 import Stratum
    path, cfg, w = make(str(tmp_path / "gen"), name, dtype, seed=11)
    rng = np.random.default_rng(0)
    prompts = [_tokens(rng, n, cfg) for n in (5, 70, 12, 1, 45, 33, 2, 28, 9)]
    llm = Stratum(path, dtype=dtype, max_tokens=2048)
    res = llm.generate(prompts, max_new_tokens=10, stop_ids=())
    for p, r in zip(prompts, res):
        assert len(r.tokens) == 10
        ref = plain_logits(cfg, w, list(p) + r.tokens[:-1])[len(p) - 1:]
        ref = ref - ref.mean(axis=-1, keepdims=True)
        for tok, row in zip(r.tokens, ref):
            assert row[tok] >= row.max() - 2 * TOL[dtype] * float(np.max(np.abs(row))), (p, r.tokens, tok)
    serial = llm.generate(prompts, max_new_tokens=10, stop_ids=(), max_batch=2)
    if dtype == "float32":
        assert [r.tokens for r in serial] == [r.tokens for r in res]
    llm.engine.cache.check()
    assert llm.engine.cache.tokens_held() == 0


def test_trace_replay_program(tmp_path):
    """`bin/trace_run` fed steps on standard input: a batch of two requests, then single tokens, one request ending
    earlier, then a request that takes the pages and the state rows given back."""
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    path, cfg, w = make(str(tmp_path / "replay"), "A", "float32", seed=21)
    rng = np.random.default_rng(8)
    vocab = cfg["vocab"]
    a, b, c = (clear_tokens(rng, n, cfg, w, "float32") for n in (70, 9, 33))
    ra, rb, rc = (plain_logits(cfg, w, t) for t in (a, b, c))
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:60], "want": [0, 59]},
                                     {"id": "b", "tokens": b[:5], "want": []}], "end": []}]
    for i in range(10):
        ents = [{"id": "a", "tokens": [a[60 + i]], "want": [0]}]
        end = ["a"] if i == 9 else []
        if i < 4:
            ents.append({"id": "b", "tokens": [b[5 + i]], "want": [0]})
            if i == 3:
                end.append("b")
        steps.append({"step": 1 + i, "entries": ents, "end": end})
    steps.append({"step": 11, "entries": [{"id": "c", "tokens": c, "want": list(range(33))}], "end": ["c"]})
    out = str(tmp_path / "out")
    p = subprocess.Popen([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", path, "--dtype", "float32",
                          "--out", out, "--max-tokens", "192"], stdin=subprocess.PIPE, stdout=subprocess.PIPE, text=True)
    for s in steps:
        p.stdin.write(json.dumps(s) + "\n")
        p.stdin.flush()
        assert p.stdout.readline().strip() == f"done {s['step']}"
    p.stdin.close()
    assert p.wait(timeout=600) == 0
    read = lambda n: np.fromfile(os.path.join(out, f"{n}.f32"), dtype="<f4").reshape(-1, vocab)   # noqa: E731
    assert_close(read(0), ra[[0, 59]], "float32", "trace step 0")
    for i in range(10):
        got = read(1 + i)
        assert_close(got[0], ra[60 + i], "float32", f"trace a {i}")
        if i < 4:
            assert_close(got[1], rb[5 + i], "float32", f"trace b {i}")
    assert_close(read(11), rc, "float32", "trace c")
