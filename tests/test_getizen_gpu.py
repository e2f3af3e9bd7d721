"""Getizen on the GPU against the plain implementation: each kernel and each mechanism alone, whole prompts against
token-by-token decoding, prompts fed in portions, unequal batches, pages, slots and state rows used again, keys on
either side of the chunks' edges and on the pages' borders, the convolution's edge, states carried from the first token,
long decoding, generation through the entry point."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

from helpers import TOL
from plain import getizen_plain as G
from getizen_helpers import (GET_A, assert_rows_close as assert_close, config, dense, layer, left, make, parallel,
                             plain_logits, retention, right)

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
    path, cfg, w = make(str(tmp_path_factory.mktemp(f"get{name}_{dtype}")), name, dtype, seed=len(name) + 1)
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


# ------------------------------------------------------------------------------------------ kernels alone
@pytest.mark.parametrize("hidden,groups", [(72, 3), (70, 5), (64, 1), (128, 32), (96, 4), (2048, 2), (4096, 2), (4096, 64),
                                           (8192, 1), (16384, 2), (33, 33), (50000, 4)])
def test_norm_of_a_sum(hidden, groups):
    """The stream times a factor plus no, one and two terms, with and without a norm of their own; in place, into another
    tensor, with a rounded copy; picked rows; no norm over the sum."""
    from stratum_b200 import kernels as K
    from stratum_b200.parts.base import Term
    rng = np.random.default_rng(hidden)
    T = 5
    x, gain = rng.standard_normal((T, hidden)) * 2, rng.uniform(0.5, 1.5, hidden)
    ys = [rng.standard_normal((T, hidden)) * 3, rng.standard_normal((T, hidden))]
    gs = [rng.uniform(0.5, 1.5, hidden), rng.uniform(0.5, 1.5, hidden)]
    eps = 0.3                                                # large: where it stands shows

    def close(a, b, tol=3e-6):
        b = torch.from_numpy(b)
        assert float((a.double().cpu() - b).abs().max()) <= tol * float(b.abs().max())

    for n_terms in (0, 1, 2):
        for normed in ((), (0,), (1,), (0, 1)):
            if any(j >= n_terms for j in normed):
                continue
            terms = [Term(_dev(ys[j]), _dev(gs[j]) if j in normed else None, 0.1 * (j + 1)) for j in range(n_terms)]
            z = 1.7 * x + sum((G.rms_norm(ys[j], gs[j], 0.1 * (j + 1)) if j in normed else ys[j]) for j in range(n_terms))
            want = G.group_norm(z, gain, eps, groups)
            xd = _dev(x)
            copy = torch.empty(T, hidden, dtype=torch.bfloat16, device="cuda")
            K.sum_norm(xd, 1.7, terms, _dev(gain), groups, eps, xd, copy=copy)
            close(xd, want)
            assert torch.equal(copy, xd.to(torch.bfloat16))
            out = torch.empty(T, hidden, device="cuda")
            K.sum_norm(_dev(x), 1.7, terms, None, 0, 0.0, out)
            close(out, z)
            K.sum_norm(out, 0.0, terms, None, 0, 0.0, out)   # a factor of zero: what was there does not matter
            close(out, z - 1.7 * x) if n_terms else None
    rows = [4, 0, 0, 3]
    for dt in (torch.float32, torch.bfloat16):
        out = torch.empty(len(rows), hidden, dtype=dt, device="cuda")
        K.sum_norm(_dev(x), 1.0, (), _dev(gain), groups, eps, out, rows=_i32(rows))
        close(out, G.group_norm(x[rows], gain, eps, groups), 3e-6 if dt == torch.float32 else 5e-3)


@pytest.mark.parametrize("M,N,K_", [(1, 192, 72), (5, 320, 128), (8, 64, 264), (17, 1024, 256), (64, 2048, 512),
                                    (100, 768, 1024), (150, 512, 256), (300, 4096, 192), (2100, 512, 128)])
def test_clamped_gate_rides_on_every_product(M, N, K_):
    """Pairs of gate and up whose values lie on both sides of the limit, through every kernel that serves such shapes."""
    from stratum_b200 import kernels as K
    from stratum_b200.parts.base import Runtime
    from stratum_b200.parts.linear import SWIGLU, Linear
    rng = np.random.default_rng(M)
    x, w = _bf16(rng.standard_normal((M, K_))), _bf16(rng.standard_normal((N, K_)) * 3 / np.sqrt(K_))
    bias = rng.standard_normal(N)
    limit = 1.3
    for dt, tol in ((torch.float32, 2e-5), (torch.bfloat16, 2e-2)):
        for b in (None, bias):
            lin = Linear(Runtime(dt, "cuda"), _dev(w, dt), None if b is None else _dev(b))
            got = lin(_dev(x, dt), mode=SWIGLU, act=K.ACT_CLAMPED_GATE, limit=limit).double().cpu().numpy()
            s = x @ w.T + (0 if b is None else b)
            g, u = np.minimum(s[:, 0::2], limit), np.clip(s[:, 1::2], -limit, limit)
            want = g * G.sigmoid(1.702 * g) * (u + 1)
            assert np.abs(s).max() > 2 * limit
            assert np.max(np.abs(got - want)) <= tol * np.max(np.abs(want))


@pytest.mark.parametrize("heads,dim,vdim,pairs", [(3, 12, 20, 4), (2, 40, 8, 20), (1, 9, 7, 0), (4, 64, 32, 32), (2, 130, 70, 10),
                                                  (1, 260, 8, 2), (2, 128, 128, 64), (8, 64, 64, 16), (2, 256, 36, 128),
                                                  (1, 208, 100, 0), (3, 16, 4, 8)])
@pytest.mark.parametrize("long", [77, 520])
@pytest.mark.parametrize("form", ["tokens", "tokens, neighbouring pairs", "chunks"])
def test_retention_kernels(heads, dim, vdim, pairs, long, form):
    """Rotation, recurrence with a constant decay per head and the heads' norm on projections made here: two sequences of
    unequal lengths whose tokens come in four steps (many, one of each, three and two, one), in slots that lie apart; the
    recurrence token by token, and in chunks on tensor cores where sizes allow."""
    from stratum_b200 import kernels as K
    interleaved = form.endswith("pairs")
    if form == "chunks" and (dim % 16 or dim > 256):
        pytest.skip("sizes the chunked form does not take")
    rng = np.random.default_rng(dim + vdim)
    HD, HV = heads * dim, heads * vdim
    lens = (long, 11)
    proj = [rng.standard_normal((n, 2 * HD + 2 * HV)) for n in lens]
    decay = [0.999, 0.6, 0.97, 1.0, 0.5, 0.9, 0.99, 0.8][:heads]
    eye = np.eye(2 * HD + 2 * HV)
    w = {"q": eye[:HD], "k": eye[HD:2 * HD], "v": eye[2 * HD:2 * HD + HV], "g": eye[2 * HD + HV:], "o": np.eye(HV)}
    m = {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay, "rot": {"base": 100.0, "dims": 2 * pairs}}
    f = G.frequencies(m["rot"])
    if interleaved:                                          # the oracle turns (i, i + n/2): hand it the columns in that order
        order = np.arange(dim)
        order[:2 * pairs] = np.concatenate([np.arange(0, 2 * pairs, 2), np.arange(1, 2 * pairs, 2)])
        cols = np.concatenate([h * dim + order for h in range(2 * heads)] + [np.arange(2 * HD, 2 * HD + 2 * HV)])
        want = [G.retention(m, 1e-5, w, p[:, cols], "") for p in proj]
    else:
        want = [G.retention(m, 1e-5, w, p, "") for p in proj]
    st = torch.zeros(6, HD * vdim + 4, device="cuda")
    slots, done, got = (4, 1), [0, 0], [[], []]
    for cut in ((long - 5, 7), (1, 1), (3, 2), (1, 1)):
        rows = np.concatenate([proj[i][done[i]:done[i] + cut[i]] for i in range(2)])
        pos = np.concatenate([np.arange(done[i], done[i] + cut[i]) for i in range(2)])
        T = rows.shape[0]
        seq = np.concatenate([np.full(cut[i], i) for i in range(2)])
        g = K.GlaStep(_dev(rows), heads, dim, vdim, 0, 1.0, dim ** -0.5, 1e-5, head_decay=_dev(decay))
        if pairs:
            ang = pos[:, None] * f[None, :]
            g.rotate(_dev(np.stack([np.cos(ang), np.sin(ang)], axis=-1)), interleaved)
        o_raw = torch.empty(T, HV, device="cuda")
        out = torch.empty(T, HV + 5, device="cuda")
        if form == "chunks":
            assert g.chunks_ok()
        g.recur(o_raw, st, _i32(seq), _i32([0, cut[0], T]), _i32(slots), True, chunked=form == "chunks")
        g.finish(None, out)
        o = out[:, :HV].cpu().numpy()
        got[0].append(o[:cut[0]]); got[1].append(o[cut[0]:])
        done = [done[i] + cut[i] for i in range(2)]
    for i in range(2):
        o = np.concatenate(got[i])
        assert np.isfinite(o).all()
        assert np.max(np.abs(o - want[i])) <= 1e-4 * np.max(np.abs(want[i])), (i, np.max(np.abs(o - want[i])))
    assert float(st[0].abs().max()) == 0.0 and float(st[5].abs().max()) == 0.0            # rows of nobody stay clean
    assert float(st[:, HD * vdim:].abs().max()) == 0.0                                    # nothing beyond a state


@pytest.mark.parametrize("heads,dim,vdim", [(3, 64, 32), (2, 128, 128), (2, 256, 36)])
def test_chunks_of_retention_are_as_wide_as_float32(heads, dim, vdim):
    """Projections that two bfloat16 parts hold exactly (16 bits): what is left is the width of scores, decayed values and
    state.  Read-outs and state in chunks against float64, next to the token-by-token form's own float32 rounding."""
    from stratum_b200 import kernels as K
    rng = np.random.default_rng(dim)
    T, HD, HV = 500, heads * dim, heads * vdim
    proj = _bf16(rng.standard_normal((T, 2 * HD + 2 * HV))) * (1.0 + 2.0 ** -12)
    proj = _bf16(proj) + _bf16(proj - _bf16(proj))
    decay = np.float32([0.997, 0.9985, 0.6])[:heads]
    q, k, v = (proj[:, a:b].reshape(T, heads, -1) for a, b in ((0, HD), (HD, 2 * HD), (2 * HD, 2 * HD + HV)))
    S, want = np.zeros((heads, dim, vdim)), np.zeros((T, heads, vdim))
    for t in range(T):
        S = decay.astype(np.float64)[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        want[t] = np.einsum("hdv,hd->hv", S, q[t])
    err = {}
    for chunked in (False, True):
        st = torch.zeros(1, HD * vdim, device="cuda")
        g = K.GlaStep(_dev(proj), heads, dim, vdim, 0, 1.0, 1.0, 1e-5, head_decay=_dev(decay))
        o = torch.empty(T, HV, device="cuda")
        g.recur(o, st, torch.zeros(T, dtype=torch.int32, device="cuda"), _i32([0, T]), _i32([0]), True, chunked=chunked)
        got = o.double().cpu().numpy().reshape(T, heads, vdim)
        err[chunked] = (np.sqrt(np.mean((got - want) ** 2)) / np.sqrt(np.mean(want ** 2)),
                        np.max(np.abs(st.double().cpu().numpy().reshape(heads, vdim, dim).transpose(0, 2, 1) - S)) / np.max(np.abs(S)))
    assert err[True][0] < 2e-6 and err[True][1] < 3e-6, err


class _Step:
    """The fields of a step's description that the recurrence reads."""

    def __init__(self, n_new, before, slots):
        self.n_new = n_new
        self.token_pos = _i32(np.concatenate([np.arange(b, b + n) for b, n in zip(before, n_new)]))
        self.token_seq = _i32(np.concatenate([np.full(n, i if s >= 0 else -1) for i, (n, s) in enumerate(zip(n_new, slots))]))
        self.seq_start = _i32(np.concatenate([[0], np.cumsum(n_new)]))
        self.seq_slot = _i32([s if s >= 0 else 0 for s in slots])
        self.max_new, self.all_single = max(n_new), all(n == 1 for n in n_new)


@pytest.mark.parametrize("width,blocks,taps", [(60, 5, 3), (35, 7, 1), (22, 1, 6), (192, 3, 4), (264, 1, 2), (512, 2, 4),
                                               (96, 12, 9), (1024, 4, 4), (640, 1, 4)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_linear_recurrence_kernels(width, blocks, taps, dtype):
    """The recurrence on projections made here: three sequences of unequal lengths, in steps of many tokens, a few, one
    each (the decode kernel), again a few, and then one each with a row of no sequence between them."""
    from stratum_b200 import kernels as K
    from stratum_b200.parts.base import Runtime
    rng = np.random.default_rng(width + taps)
    td, size = _td(dtype), width // blocks
    lens = (301, 40, 12)
    W = {"conv": rng.uniform(-0.7, 0.7, (width, taps)), "conv.b": rng.uniform(-0.5, 0.5, width),
         "ra": _bf16(rng.standard_normal((blocks, size, size)) * 2 / np.sqrt(size)),
         "ri": _bf16(rng.standard_normal((blocks, size, size)) * 2 / np.sqrt(size)),
         "ra.b": rng.standard_normal((blocks, size)), "ri.b": rng.standard_normal((blocks, size)),
         "lam": rng.uniform(-8.0, 1.0, width)}
    proj = [rng.standard_normal((n, 2 * width)) * 1.5 for n in lens]
    want = [G.linear_recurrence(G.causal_conv(p[:, width:], W["conv"], W["conv.b"]), blocks, W, "") *
            G.gelu_tanh(p[:, :width]) for p in proj]
    unit = K.LinearRecurrence(_dev(W["conv"].T), _dev(W["conv.b"]), _dev(np.concatenate([W["ra"], W["ri"]], axis=1), td),
                              _dev(np.concatenate([W["ra.b"], W["ri.b"]], axis=1)), _dev(-8.0 * np.logaddexp(0.0, W["lam"])))
    assert unit.tensor_cores == (dtype == "bfloat16" and size % 8 == 0)
    rt = Runtime(td, "cuda")
    stride = ((1 + taps) * width + 3) // 4 * 4 + 4
    state = torch.zeros(6, stride, device="cuda")
    state[5] = 7.0
    slots, done, got = [3, 0, 4], [0, 0, 0], [[], [], []]
    for cut in ((280, 20, 2), (2, 5, 1), (1, 1, 1), (1, 1, 1), (3, 2, 2), (1, 1, 1), None, (1, 1, 1)):
        if cut is None:                                      # a step in which the second row belongs to nobody
            rows = np.concatenate([proj[0][done[0]:done[0] + 1], proj[0][:1], proj[2][done[2]:done[2] + 1]])
            step, live, cut = _Step([1, 1, 1], [done[0], 0, done[2]], [3, -1, 4]), (0, 2), (1, 1, 1)
        else:
            rows = np.concatenate([proj[i][done[i]:done[i] + cut[i]] for i in range(3)])
            step, live = _Step(list(cut), done, slots), (0, 1, 2)
        ld = (2 * width + 3) // 4 * 4
        p = torch.zeros(rows.shape[0], ld, device="cuda")
        p[:, :2 * width] = _dev(rows)
        out = torch.full((rows.shape[0], width + 8), 3.0, dtype=td, device="cuda")
        unit.run(rt, p, out, state, step, True)
        o, r = out[:, :width].float().cpu().numpy(), 0
        for i in range(3):
            if i in live:
                got[i].append(o[r:r + cut[i]])
                done[i] += cut[i]
            else:
                assert not o[r:r + cut[i]].any()             # rows of no sequence: zero
            r += cut[i]
    for i in range(3):
        g = np.concatenate(got[i])
        tol = 2e-5 if dtype == "float32" else 6e-3           # the output's rounding
        assert np.max(np.abs(g - want[i][:len(g)])) <= tol * np.max(np.abs(want[i])), i
    assert float(state[1].abs().max()) == 0.0 and float(state[2].abs().max()) == 0.0 and bool((state[5] == 7.0).all())
    assert float(state[:5, (1 + taps) * width:].abs().max()) == 0.0
    # the state itself is float32-exact in both dtypes: S of a sequence against the plain loop
    u = G.causal_conv(proj[0][:done[0], width:], W["conv"], W["conv.b"])
    S = G.linear_recurrence(u, blocks, W, "")[-1]
    assert np.max(np.abs(state[3, :width].cpu().numpy() - S)) <= (2e-5 if dtype == "float32" else 5e-5) * np.max(np.abs(S))
    before = state.clone()
    unit.run(rt, p, out, state, step, False)                 # told not to write: nothing changes
    assert torch.equal(before, state)


def _softmax(q, k, v, vis, scales):
    T, H, _ = q.shape
    out = np.zeros((T, H, v.shape[2]))
    for h in range(H):
        g = h // (H // k.shape[1])
        s = np.where(vis, q[:, h] @ k[:, g].T * scales[h], -np.inf)
        e = np.exp(s - s.max(-1, keepdims=True))
        out[:, h] = e / e.sum(-1, keepdims=True) @ v[:, g]
    return out.reshape(T, -1)


@pytest.mark.parametrize("H,Gk,D,Dv,chunk", [(4, 2, 12, 20, 50), (3, 3, 20, 22, 5), (8, 1, 64, 64, 130), (4, 4, 32, 48, 64),
                                             (4, 2, 128, 128, 100), (2, 1, 64, 64, 1), (20, 1, 32, 32, 77), (8, 2, 64, 64, 200), (2, 2, 128, 128, 64)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_chunked_attention_with_head_factors_and_an_output_gate(H, Gk, D, Dv, chunk, dtype):
    """A paged cache whose pages lie in no order, queries at every position in blocks (prompt) and single queries at
    chosen positions (decode steps, cut into ranges), against the softmax written out."""
    from stratum_b200 import kernels as K
    from stratum_b200.parts.attention_dispatch import plan_general_splits
    rng = np.random.default_rng(H + D)
    td = _td(dtype)
    T = 333
    r = _bf16 if dtype == "bfloat16" else (lambda a: a)
    q, k, v = r(rng.standard_normal((T, H, D))), r(rng.standard_normal((T, Gk, D))), r(rng.standard_normal((T, Gk, Dv)))
    gate, temp, scale = rng.standard_normal((T, H * Dv)) * 2, rng.uniform(0.3, 2.5, H), 1.5 / np.sqrt(D)
    temp[0] = -0.7
    vis = G.visible(T, chunk)
    want = _softmax(q, k, v, vis, scale * temp) * G.sigmoid(gate)
    pages = [7, 2, 9, 4, 0, 5]
    kc, vc = np.zeros((10, Gk, 64, D)), np.zeros((10, Gk, 64, Dv))
    for t in range(T):
        kc[pages[t // 64], :, t % 64], vc[pages[t // 64], :, t % 64] = k[t], v[t]
    kc, vc = _dev(kc, td), _dev(vc, td)
    if D == Dv and D in (64, 128):
        temp[:] = 1.0                                        # (the tcgen05 kernel takes no factor per head)
        want = _softmax(q, k, v, vis, np.full(H, scale)) * G.sigmoid(gate)
    shape = K.AttentionShape(H, H // Gk, 1, D, Dv, False, scale, chunk=chunk, head_scale=_dev(temp))
    bt = _i32([pages])
    tol = 2e-5 if dtype == "float32" else 1e-2

    def run(rows, single):
        n = len(rows)
        qd = torch.zeros(n, (H * D + 7) // 8 * 8, dtype=td, device="cuda")
        qd[:, :H * D] = _dev(q[rows].reshape(n, H * D), td)
        gd = torch.zeros(n, (H * Dv + 7) // 8 * 8, device="cuda")
        gd[:, :H * Dv] = _dev(gate[rows])
        out = torch.zeros(n, (H * Dv + 7) // 8 * 8, dtype=td, device="cuda")
        pos = _i32(rows)
        if single:                                           # every row a sequence of its own, over the same pages
            tables, seq = bt.repeat(n, 1), _i32(np.arange(n))
        else:
            tables, seq = bt, torch.zeros(n, dtype=torch.int32, device="cuda")
        if K.attention_general_mma_ok(shape, qd, out, 64, gd):
            if single:
                streams = Gk * ((H // Gk + 15) // 16)
                for splits, per in (plan_general_splits(n * streams, T, shape.span), (6, 64), (2, 192)):
                    po = torch.empty(n * H * splits * Dv, device="cuda")
                    ml = torch.empty(n * H * splits * 2, device="cuda")
                    out.zero_()
                    K.attention_general_mma(shape, qd, kc, vc, pos, seq, tables, out, 64, None, 16 // min(H // Gk, 16), splits,
                                            per, po, ml, 1, gate=gd)
                    yield out[:, :H * Dv].double().cpu().numpy()
            else:
                per_block = 16 // min(H // Gk, 16)
                for groups in (1, 2):
                    b = per_block * groups
                    starts = np.arange(0, n, b)
                    qb = (torch.zeros(len(starts), dtype=torch.int32, device="cuda"), _i32(starts), _i32(np.minimum(b, n - starts)))
                    out.zero_()
                    K.attention_general_mma(shape, qd, kc, vc, pos, seq, tables, out, 64, qb, per_block, 1, 384, None, None,
                                            groups, gate=gd)
                    yield out[:, :H * Dv].double().cpu().numpy()
        if D == Dv and D in (64, 128) and td == torch.bfloat16 and not single:      # the tcgen05 kernel
            b = 2 * (128 // (H // Gk))
            starts = np.arange(0, n, b)
            qb = (torch.zeros(len(starts), dtype=torch.int32, device="cuda"), _i32(starts), _i32(np.minimum(b, n - starts)))
            out.zero_()
            K.attention_tc(qd, kc, vc, pos, bt, qb, out, H, Gk, D, 64, 0, scale, halves=2, split=True, chunk=chunk, gate=gd)
            K.check_status()
            got = out[:, :H * Dv].double().cpu().numpy()
            assert np.max(np.abs(got - want)) <= 5e-3 * np.max(np.abs(want))        # (the output's rounding alone)
            yield got
        out.zero_()
        K.attention_general(shape, qd, kc, vc, pos, seq, tables, out, 64, gd)
        yield out[:, :H * Dv].double().cpu().numpy()

    for got in run(np.arange(T), False):
        assert np.max(np.abs(got - want)) <= tol * np.max(np.abs(want))
    rows = sorted({0, 1, chunk - 1, chunk, min(chunk + 1, T - 1), 63, 64, 65, 2 * chunk % T, 255, 256, T - 1})
    for got in run(np.asarray(rows), True):
        assert np.max(np.abs(got - want[rows])) <= tol * np.max(np.abs(want))


# ------------------------------------------------------------------------------------------ mechanisms alone
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["parallel", "retention", "dense"])
def test_each_mechanism_alone(name, dtype, tmp_path):
    from stratum_b200.engine import StepEntry
    path, cfg, w = make(str(tmp_path / name), name, dtype, seed=3)
    engine = _engine(path, dtype)
    rng = np.random.default_rng(1)
    for n in (1, 2, 7, 100):
        toks = _tokens(rng, n, cfg)
        slot = engine.acquire()
        got = engine.step([StepEntry(slot, toks, list(range(n)))]).cpu().numpy()
        engine.release(slot)
        assert_close(got, plain_logits(cfg, w, toks), dtype, f"{name} n={n}")


def test_the_mean_of_mixers_under_another_arrangement():
    """A mixer of mixers asked to add to a stream or to store, as any mixer is: the same numbers as its terms'."""
    from stratum_b200 import kernels as K
    from stratum_b200.parts import PartSpec, Runtime, find_part
    from stratum_b200.cache import SequenceCache
    rt = Runtime(torch.float32, "cuda")
    one = PartSpec("gated_linear_recurrence", {"hidden": 24, "width": 20, "blocks": 2, "taps": 3, "prefix": "a."})
    two = PartSpec("retention", {"hidden": 24, "n_heads": 2, "head_dim": 6, "v_dim": 5, "decay": (0.5, 0.9), "eps": 1e-5,
                                 "prefix": "b."})
    mix = find_part("mixer", "mixer_mean")(PartSpec("mixer_mean", {
        "hidden": 24, "mixers": (one, two), "norms": ("a.out", "b.out"), "eps": 1e-5, "prefix": ""}), rt)
    rng = np.random.default_rng(0)
    w = {n: _dev(rng.standard_normal(t.shape)) for n, t in mix.tensors().items()}
    mix.bind(w)
    cache = SequenceCache([mix.cache_spec()], 64, 1, torch.float32, "cuda")
    step = _Step([6], [0], [0])
    step.n_tokens = 6
    x, res = _dev(rng.standard_normal((6, 24))), rng.standard_normal((6, 24))

    def run(**kw):
        for g in cache.groups:
            g.state.zero_()
        y = _dev(res)
        mix.forward(x, y, step, cache.layer_view(0, True, {}), **kw)
        return y.cpu().numpy()
    stored, added = run(store=True), run()
    h = x.double().cpu().numpy()
    w64 = {n: t.double().cpu().numpy() for n, t in w.items()}
    ya = G.recurrent_block({"blocks": 2}, w64, h, "a.")
    yb = G.retention({"heads": 2, "dim": 6, "vdim": 5, "decay": (0.5, 0.9)}, 1e-5, w64, h, "b.")
    want = 0.5 * (G.rms_norm(ya, w64["a.out"], 1e-5) + G.rms_norm(yb, w64["b.out"], 1e-5))
    assert np.max(np.abs(stored - want)) <= 2e-5 * np.max(np.abs(want))
    assert np.max(np.abs(added - want - res)) <= 2e-5 * np.max(np.abs(want))
    K.check_status()


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_model_without_rotation_chunks_and_feed_forwards(dtype, tmp_path):
    """What a file does not mention does not exist: the same layers with those keys left out."""
    import copy
    from stratum_b200.engine import StepEntry
    raw = copy.deepcopy(GET_A)
    del raw["layers"][0]["mixer"]["left"]["rot"]
    del raw["layers"][0]["mixer"]["left"]["mask"]
    del raw["layers"][2]["mixer"]["left"]["rot"]["scaling"]
    del raw["layers"][1]["mixer"]["rot"]
    raw["layers"][1]["mlp"] = None
    path, cfg, w = make(str(tmp_path / "bare"), None, dtype, seed=12, cfg=raw)
    engine = _engine(path, dtype)
    toks = _tokens(np.random.default_rng(0), 90, cfg)
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
    toks = _tokens(np.random.default_rng(0), 60, cfg)
    slot = engine.acquire()
    engine.step([StepEntry(slot, toks, [59])])
    engine.release(slot)
    want = []
    G.forward(cfg, w, toks, want)
    assert len(seen) == len(want) == 4
    for i, (a, b) in enumerate(zip(seen, want)):
        assert np.max(np.abs(a - b)) <= 2e-5 * np.max(np.abs(b)), i


# ------------------------------------------------------------------------------------------ whole models
def test_whole_prompt_all_positions(setup):
    from stratum_b200.engine import StepEntry
    name, dtype, cfg, w, engine, _ = setup
    rng = np.random.default_rng(1)
    for n in (1, 2, 3, 5, 6, 63, 64, 65, 200):
        toks = _tokens(rng, n, cfg)
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
    toks = _tokens(np.random.default_rng(2), n, cfg)
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
    """A prompt cut into portions of a few sizes, down to two tokens; portions start inside pages and chunks and on their
    borders, and the convolutions reach back over the cuts."""
    from stratum_b200.engine import StepEntry
    name, dtype, cfg, w, engine, _ = setup
    n = 150 if portion > 3 else 80
    toks = _tokens(np.random.default_rng(portion), n, cfg)
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
        full = [_tokens(rng, n + k, cfg) for n, k in zip(lens, extra_n)]
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
    toks = [_tokens(rng, n, cfg) for n in (95, 140, 66)]
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
        toks = _tokens(rng, n, cfg)
        slot = engine.acquire()
        got = engine.step([StepEntry(slot, toks[:-1], [n - 2])]).cpu().numpy()
        got = np.concatenate([got, engine.step([StepEntry(slot, toks[-1:], [0])]).cpu().numpy()])
        assert_close(got, plain_logits(cfg, w, toks)[-2:], dtype, f"{name} reuse n={n}")
        held.append(slot)
        engine.cache.check()


def test_first_tokens_and_long_decoding(setup):
    """Positions 0, 1, 2 one by one, then on across several pages and chunks; a chunked layer gives back the pages of the
    chunks that are through."""
    from stratum_b200.engine import StepEntry
    name, dtype, cfg, w, engine, _ = setup
    n = 270
    toks = _tokens(np.random.default_rng(5), n, cfg)
    ref = plain_logits(cfg, w, toks)
    slot = engine.acquire()
    check = {0, 1, 2, 3, 4, 5, 6} | set(range(7, n, 29)) | {63, 64, 65, 127, 128, 129, 191, 192, 193, 255, 256, 257, n - 1}
    got = []
    for i in range(n):
        out = engine.step([StepEntry(slot, [toks[i]], [0] if i in check else [])])
        if i in check:
            got.append(out.cpu().numpy())
    for gi, g in enumerate(engine.cache.groups):
        if g.pool is not None and g.spec.chunk:
            held = sum(p >= 0 for p in engine.cache.page_table_rows([slot], gi)[0])
            assert held <= (g.spec.chunk + 126) // 64
    engine.release(slot)
    assert_close(np.concatenate(got), ref[sorted(check)], dtype, f"{name} long decode")
    engine.cache.check()
    assert engine.cache.tokens_held() == 0


# ------------------------------------------------------------------------------------------ one token decides
def _marked_key_model(path, dtype, form):
    """One layer whose attention side alone counts, in which token 7 is the only one with anything in the embedding's
    first dimension, and token 8 the only one with anything in the second.  The last dimension of every key head (which
    is not rotated) reads the first dimension and nothing else, the last dimension of every query head reads the second;
    with gains of 3 on the normalised queries and keys the marked key's score stands far above the hundreds of others
    when token 8 asks, wherever the key lies, and the heads' outputs are its value."""
    lf = {"small": left(heads=4, kv=2, dim=16, vdim=24, rot=8, chunk=40, scale=0.25),
          "mma": left(heads=8, kv=1, dim=32, vdim=48, rot=16, chunk=130, scale=0.15),
          "wide": left(heads=4, kv=2, dim=64, vdim=64, rot=32, chunk=100, scale=0.1)}[form]
    cfg_raw = config([layer("parallel", parallel(lf, right(width=24, blocks=2, conv=2)))], vocab=120, width=64, groups=2,
                     alpha=0.3)
    H, Gk, D = lf["heads"], lf["kv_heads"], lf["dim"]

    def edit(t):
        e = t["embed"].float()
        e[:, :2] = 0.0
        e[7, 0] = e[8, 1] = 24.0
        t["embed"] = e.to(t["embed"].dtype)
        for name, heads, col in (("l0.mix.left.k", Gk, 0), ("l0.mix.left.q", H, 1)):
            m = t[name].float()
            m[:, :2] = 0.0
            for h in range(heads):
                m[h * D + D - 1] = 0.0
                m[h * D + D - 1, col] = 4.0
            t[name] = m.to(t[name].dtype)
        for name in ("l0.mix.left.q.norm", "l0.mix.left.k.norm"):
            t[name] = torch.full_like(t[name], 3.0)
        t["l0.mix.left.temp"] = torch.ones_like(t["l0.mix.left.temp"])
        t["l0.mix.right.out"] = torch.zeros_like(t["l0.mix.right.out"])
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


@pytest.mark.parametrize("form", ["small", "mma", "wide"])
@pytest.mark.parametrize("dtype", DTYPES)
def test_keys_on_either_side_of_the_chunks_edges(dtype, form, tmp_path):
    """A marked key at the first place of the asking token's chunk decides the logits, from however far back in the chunk
    the token asks; one place further out it changes nothing (both shown on the plain implementation).  The asking token
    stands at the chunk's second and last place and between, in the first and later chunks; chunks begin inside pages."""
    path, cfg, w = _marked_key_model(str(tmp_path / "edge"), dtype, form)
    size = cfg["layers"][0]["mixer"]["left"]["mask"]["size"]
    engine = _engine(path, dtype)
    rng = np.random.default_rng(1)
    for n in (size, 2 * size, 2 * size + 2, 3 * size, 3 * size - size // 3, 3 * size + 7):
        start = (n - 1) - (n - 1) % size
        for at, seen in ((start, True), (start - 1, False), (n - 2, True), (0, start == 0)):
            if at < 0 or (at == n - 2 and at < start):
                continue
            toks = [int(x) for x in rng.integers(9, cfg["vocab"], n)]
            toks[-1] = 8
            toks[at] = 7
            ref = plain_logits(cfg, w, toks)[-1]
            moved = list(toks)
            moved[at] = 9
            changed = np.max(np.abs(plain_logits(cfg, w, moved)[-1] - ref)) / np.max(np.abs(ref))
            assert changed > 0.15 if seen else changed < 1e-6, f"n={n}: the marked key at {at} changes the logits by {changed}"
            _three_forms(engine, toks, dtype, ref, f"n={n}, marked key at {at}", first=start if start > 0 else 201)
            if dtype == "float32" or seen:
                _three_forms(engine, toks, dtype, ref, f"n={n}, marked key at {at}", first=max(at, 1))


@pytest.mark.parametrize("dtype", DTYPES)
def test_the_first_token_of_a_chunk_sees_itself_alone(dtype, tmp_path):
    """At a chunk's first place the softmax has one key: the attention's output is that key's value, whatever came
    before; so tokens in front of it reach its logits only where they may (nowhere, with the other side off)."""
    from stratum_b200.engine import StepEntry
    path, cfg, w = _marked_key_model(str(tmp_path / "first"), dtype, "mma")
    size = cfg["layers"][0]["mixer"]["left"]["mask"]["size"]
    engine = _engine(path, dtype)
    rng = np.random.default_rng(2)
    alone = plain_logits(cfg, w, [33])[0]
    for n in (size, 2 * size):
        toks = _tokens(rng, n, cfg) + [33]
        slot = engine.acquire()
        whole = engine.step([StepEntry(slot, toks, [n])]).cpu().numpy()[0]
        engine.release(slot)
        slot = engine.acquire()
        engine.step([StepEntry(slot, toks[:n], [])])
        single = engine.step([StepEntry(slot, [33], [0])]).cpu().numpy()[0]
        engine.release(slot)
        assert_close(whole, alone, dtype, "whole")
        assert_close(single, alone, dtype, "decoded")


def _one_sided(t, side):
    other = "right" if side == "left" else "left"
    t[f"l0.mix.{other}.out"] = torch.zeros_like(t[f"l0.mix.{other}.out"])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("taps,width,blocks", [(4, 48, 3), (2, 40, 5), (7, 64, 2), (1, 48, 3)])
def test_the_convolutions_edge(taps, width, blocks, dtype, tmp_path):
    """A recurrence that forgets at once: a marked token taps - 1 places back changes the logits, one place further out it
    does not, within a prompt, across the border of two steps (cut anywhere between the two) and for decoded tokens."""
    from stratum_b200.engine import StepEntry
    cfg_raw = config([layer("parallel", parallel(left(heads=2, kv=1, dim=8, vdim=8, rot=4), right(width, blocks, taps)))],
                     vocab=90, width=48, groups=2, alpha=0.4)

    def edit(t):
        _one_sided(t, "right")
        t["l0.mix.right.lam"] = torch.full_like(t["l0.mix.right.lam"], 40.0)
        t["l0.mix.right.ra.b"] = torch.full_like(t["l0.mix.right.ra.b"], 4.0)
        t["l0.mix.right.conv"] = torch.full_like(t["l0.mix.right.conv"], 0.8)
        e = t["embed"].float()
        e[1] *= 6.0
        t["embed"] = e.to(t["embed"].dtype)
    path, cfg, w = make(str(tmp_path / "conv"), None, dtype, seed=4, edit=edit, cfg=cfg_raw)
    engine = _engine(path, dtype)
    rng = np.random.default_rng(taps)
    n = 30
    for back in (taps - 1, taps):
        toks = [int(x) for x in rng.integers(2, 90, n)]
        toks[n - 1 - back] = 1
        ref = plain_logits(cfg, w, toks)[-1]
        moved = list(toks)
        moved[n - 1 - back] = 5
        changed = np.max(np.abs(plain_logits(cfg, w, moved)[-1] - ref)) / np.max(np.abs(ref))
        assert changed > 0.03 if back < taps else changed < 1e-4, (back, changed)
        for cut in range(n - 1 - taps, n):
            slot = engine.acquire()
            engine.step([StepEntry(slot, toks[:cut], [])])
            got = engine.step([StepEntry(slot, toks[cut:], [n - 1 - cut])]).cpu().numpy()[0]
            engine.release(slot)
            assert_close(got, ref, dtype, f"{taps} taps, marked {back} back, cut at {cut}")
        slot = engine.acquire()
        engine.step([StepEntry(slot, toks[:n - 1 - taps], [])])
        for t in toks[n - 1 - taps:-1]:
            engine.step([StepEntry(slot, [t], [])])
        got = engine.step([StepEntry(slot, toks[-1:], [0])]).cpu().numpy()[0]
        engine.release(slot)
        assert_close(got, ref, dtype, f"{taps} taps, marked {back} back, decoded")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("at", [0, 5, 63, 64])
@pytest.mark.parametrize("kind", ["recurrence", "retention"])
def test_the_state_carries_a_token_from_far_back(kind, at, dtype, tmp_path):
    """A layer that hardly forgets: hundreds of tokens later the output is still shaped by one marked token (shown on the
    plain implementation), through a prompt cut in two, a state row used before, and decoded tokens."""
    from stratum_b200.engine import StepEntry
    if kind == "recurrence":
        lay = layer("parallel", parallel(left(heads=2, kv=1, dim=8, vdim=8, rot=4), right(width=48, blocks=3, conv=3)))
    else:
        lay = layer("retention", retention(heads=2, dim=8, vdim=12, rot=4, decay=[1.0 - 2.0 ** -12, 1.0 - 2.0 ** -11]))
    cfg_raw = config([lay], vocab=90, width=48, groups=2, alpha=0.4)

    def edit(t):
        e = t["embed"].float()
        e[:, :2] = 0.0
        e[:, 1] = 0.5                                        # every token has the same second dimension
        e[1, 0] = 30.0                                       # the marked token alone has a first one
        t["embed"] = e.to(t["embed"].dtype)
        if kind == "recurrence":
            _one_sided(t, "right")
            t["l0.mix.right.lam"] = torch.full_like(t["l0.mix.right.lam"], -9.0)
            m = t["l0.mix.right.x"].float()
            m *= 0.1
            m[:, 0] = torch.sign(m[:, 5]) * 6.0              # the marked token's input dwarfs the others'
            t["l0.mix.right.x"] = m.to(t["l0.mix.right.x"].dtype)
            t["l0.mix.right.x.b"] = torch.zeros_like(t["l0.mix.right.x.b"])
            t["l0.mix.right.conv.b"] = torch.zeros_like(t["l0.mix.right.conv.b"])
            t["l0.mix.right.ri.b"] = torch.full_like(t["l0.mix.right.ri.b"], 2.0)
        else:
            for name, col in (("l0.mix.k", 0), ("l0.mix.q", 1)):   # the last dimension of every head is not rotated: keys
                m = t[name].float()                               # read the first there, queries the second
                m[:, :2] = 0.0
                for h in range(2):
                    m[h * 8 + 7] = 0.0
                    m[h * 8 + 7, col] = 8.0
                t[name] = m.to(t[name].dtype)
    path, cfg, w = make(str(tmp_path / "state"), None, dtype, seed=4, edit=edit, cfg=cfg_raw)
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
def test_each_sides_share_of_a_pair(dtype, tmp_path):
    """Both sides count by half, whatever the size of their outputs: one side's output matrix made a hundred times larger
    changes next to nothing, its norm's weight made twice as large does."""
    from stratum_b200.engine import StepEntry
    cfg_raw = config([layer("parallel", parallel(left(heads=2, kv=1, dim=8, vdim=8, rot=4), right(width=48, blocks=3)))],
                     vocab=90, width=48, groups=2)
    logits = {}
    for what in ("plain", "larger", "weightier"):
        def edit(t):
            t["l0.mix.left.o"] = (t["l0.mix.left.o"].float() * 4).to(t["l0.mix.left.o"].dtype)      # well above eps
            if what == "larger":
                t["l0.mix.left.o"] = (t["l0.mix.left.o"].float() * 128).to(t["l0.mix.left.o"].dtype)
            if what == "weightier":
                t["l0.mix.left.out"] = (t["l0.mix.left.out"].float() * 2).to(t["l0.mix.left.out"].dtype)
        path, cfg, w = make(str(tmp_path / what), None, dtype, seed=4, edit=edit, cfg=cfg_raw)
        toks = [int(t) for t in np.random.default_rng(1).integers(2, 90, 25)]
        ref = plain_logits(cfg, w, toks)
        engine = _engine(path, dtype)
        slot = engine.acquire()
        got = engine.step([StepEntry(slot, toks, list(range(25)))]).cpu().numpy()
        assert_close(got, ref, dtype, what)
        logits[what] = ref
    size = np.max(np.abs(logits["plain"]))
    assert np.max(np.abs(logits["larger"] - logits["plain"])) < 0.01 * size
    assert np.max(np.abs(logits["weightier"] - logits["plain"])) > 0.1 * size


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
    a, b, c = (_tokens(rng, n, cfg) for n in (70, 9, 33))
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
