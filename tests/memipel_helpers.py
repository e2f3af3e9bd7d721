"""Small Memipel configurations and model folders for the tests.  None of them is anyone's model: sizes are chosen so that
no two of a layer's sizes are equal by accident, that counts are not 1 where the formulas divide by them, and that the
layers of one model differ from one another (heads, key and value sizes, taps, windows, ranks, decays, experts, groups,
limits)."""
import numpy as np
import torch

from helpers import load_plain, make_model_dir
from mokatar_helpers import assert_rows_close  # noqa: F401  (the same comparison)
from plain import memipel_plain as M

STEADY = 6.0


def attention(heads=4, kv=2, dim=24, vdim=16, scale=0.2, conv=3, mix=True, size=50):
    d = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "v_mix": mix}
    if conv:
        d["conv"] = conv
    if size:
        d["mask"] = {"size": size}
    return d


def latent(heads=3, dim=20, vdim=12, q_rank=28, kv_rank=36, scale=0.3, size=45):
    d = {"heads": heads, "dim": dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale}
    if size:
        d["mask"] = {"size": size}
    return d


def lightning(heads=3, dim=12, vdim=20, decay=None):
    return {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay or [1.0 - 2.0 ** (-1 - 3 * h) for h in range(heads)]}


def dense(ff=96):
    return {"kind": "dense", "ff": ff}


def moe(experts=6, top=2, groups=3, keep=2, ff=20, limit=1.1, shared=36, shared_limit=0.7):
    d = {"kind": "moe", "router": {"experts": experts, "top": top, "groups": {"count": groups, "keep": keep}},
         "expert": {"ff": ff, "limit": limit}}
    if shared:
        d["shared"] = {"ff": shared, "limit": shared_limit}
    return d


def layer(kind, mixer, mlp=None):
    return {"type": kind, "mixer": mixer, "mlp": mlp}


def config(layers, vocab=211, width=72, eps=1e-5):
    return {"architecture": "Memipel", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


# the first layer that lends its values stands third; a layer of plain attention between those that mix; sizes in
# multiples of four
MEM_A = config([layer("lightning", lightning(), moe()),
                layer("attention", attention(mix=False, conv=2, size=30), dense()),
                layer("attention", attention(), moe(experts=8, top=3, groups=2, keep=1, ff=24, limit=0.6, shared=0)),
                layer("latent_attention", latent()),
                layer("attention", attention(heads=2, kv=1, dim=20, vdim=32, conv=4, size=0), dense(80)),
                layer("lightning", lightning(heads=2, dim=20, vdim=8))])
# sizes that no vector load divides: every fallback kernel; one tap and six and none, one kv head, one group, one expert a
# token, tiny windows, a negative scale
MEM_B = config([layer("attention", attention(heads=3, kv=1, dim=18, vdim=10, conv=6, size=5), moe(experts=5, top=1, groups=1, keep=1, ff=15, limit=3.0, shared=9)),
                layer("lightning", lightning(heads=1, dim=9, vdim=7, decay=[0.8]), dense(50)),
                layer("attention", attention(heads=4, kv=2, dim=7, vdim=5, conv=0, scale=-0.4, size=1)),
                layer("latent_attention", latent(heads=5, dim=11, vdim=6, q_rank=13, kv_rank=22, size=7), dense(34)),
                layer("attention", attention(heads=2, kv=2, dim=15, vdim=5, conv=1, size=33), dense(30))],
               vocab=97, width=70, eps=1e-6)
# sizes of the tensor-core kernels: eight query heads on a kv head, windows longer and shorter than pages, values smaller
# and larger than keys
MEM_TC = config([layer("attention", attention(heads=8, kv=1, dim=64, vdim=64, scale=0.1, conv=4, size=130), dense(160)),
                 layer("attention", attention(heads=4, kv=2, dim=48, vdim=32, scale=0.15, conv=3, size=70), moe(experts=8, top=3, groups=4, keep=2, ff=32, shared=64)),
                 layer("lightning", lightning(heads=4, dim=64, vdim=32), moe(experts=4, top=2, groups=2, keep=2, ff=48, limit=0.8, shared=0)),
                 layer("latent_attention", latent(heads=6, dim=32, vdim=48, q_rank=80, kv_rank=64, scale=0.2, size=100), dense(96)),
                 layer("attention", attention(heads=4, kv=4, dim=32, vdim=16, scale=0.2, conv=4, size=64), dense(96))],
                vocab=331, width=128)
# heads of 128 and of 64 in groups: the prompt kernel for such heads; more heads than a tile of queries over one latent row
MEM_BIG = config([layer("attention", attention(heads=4, kv=2, dim=128, vdim=128, scale=0.08, conv=4, size=150), moe(experts=4, top=2, groups=2, keep=1, ff=64, shared=128)),
                  layer("lightning", lightning(heads=2, dim=128, vdim=128, decay=[0.96, 1.0 - 2.0 ** -9]), dense(192)),
                  layer("attention", attention(heads=8, kv=4, dim=64, vdim=64, scale=0.12, conv=2, size=0)),
                  layer("latent_attention", latent(heads=20, dim=64, vdim=64, q_rank=96, kv_rank=128, scale=0.1, size=0), dense(128))],
                 vocab=257, width=192)
# one mechanism each, alone
MEM_ATTENTION = config([layer("attention", attention(heads=4, kv=2, dim=16, vdim=8, size=42))], width=64)
MEM_MIX = config([layer("attention", attention(heads=2, kv=2, dim=8, vdim=12)), layer("attention", attention(heads=6, kv=3, dim=12, vdim=8))], width=64)
MEM_LATENT = config([layer("latent_attention", latent(heads=4, dim=16, vdim=8, q_rank=24, kv_rank=32))], width=64)
MEM_LIGHTNING = config([layer("lightning", lightning(heads=4, dim=8, vdim=16))], width=64)
MEM_MOE = config([layer("lightning", lightning(heads=1, dim=8, vdim=8), moe(experts=12, top=4, groups=4, keep=3))], width=64)
MEM_DENSE = config([layer("lightning", lightning(heads=1, dim=8, vdim=8), dense(120))], width=64)

CONFIGS = {"A": MEM_A, "B": MEM_B, "TC": MEM_TC, "BIG": MEM_BIG, "attention": MEM_ATTENTION, "mix": MEM_MIX,
           "latent": MEM_LATENT, "lightning": MEM_LIGHTNING, "moe": MEM_MOE, "dense": MEM_DENSE}


def lively(tensors, seed=0, decisive=False):
    """Random weights as the writer makes them are tame: gains of one, sinks and biases of zero, shares of nearly zero,
    routers that hardly prefer anyone.  Give every constant a value of its own and make scores spread.

    decisive: the routers' choices survive the rounding of the bfloat16 path.  Every token's embedding carries the same
    large number in its first dimension, and the routers read it with weights that lie apart and everything else faintly.
    The choice is then nearly the same for every token (the scores, which are the weights, still vary); the float32 tests
    have routers that choose freely."""
    g = torch.Generator().manual_seed(seed)
    rnd = lambda t, lo, hi: (torch.rand(t.shape, generator=g) * (hi - lo) + lo).to(t.dtype)      # noqa: E731
    for name, t in list(tensors.items()):
        if name.endswith(("norm1", "final.norm")):             # stored around zero
            tensors[name] = rnd(t, -0.5, 0.5)
        elif name.endswith(".norm"):
            tensors[name] = rnd(t, 0.5, 1.5)
        elif name.endswith(".sink"):
            tensors[name] = rnd(t, -1.0, 2.0)
        elif name.endswith(".vmix"):
            tensors[name] = rnd(t, 0.2, 0.8)
        elif name.endswith(".conv"):
            tensors[name] = rnd(t, -0.8, 0.8)
        elif name.endswith(".b"):
            tensors[name] = rnd(t, -0.5, 0.5)
        elif name.endswith(".router"):
            m = t.float() * (0.1 if decisive else 6.0)
            if decisive:
                m[:, 0] = 0.4 * torch.randperm(t.shape[0], generator=g).float()
            tensors[name] = m.to(t.dtype)
        elif name == "embed":
            m = t.float() * 30
            if decisive:
                m[:, 0] = STEADY
            tensors[name] = m.to(t.dtype)
        else:
            tensors[name] = (t.float() * 2.5).to(t.dtype)


def make(path, name, dtype, seed=0, edit=None, cfg=None):
    def both(tensors):
        lively(tensors, seed, dtype == "bfloat16")
        if edit is not None:
            edit(tensors)
    path = make_model_dir(path, cfg or CONFIGS[name], seed=seed, dtype=dtype, std=0.05, edit=both)
    cfg, w = load_plain(path)
    return path, cfg, w


def plain_logits(cfg, w, tokens):
    return M.forward(cfg, w, tokens)


def clear_tokens(rng, n, cfg, w, dtype):
    """n random tokens on which no router is near a tie: a choice that rounding could turn is no test of anything.  float32
    keeps 1e-4 away (in logits), bfloat16 (with decisive routers) 0.08."""
    need = 1e-4 if dtype == "float32" else 0.08
    for _ in range(200):
        toks = [int(t) for t in rng.integers(0, cfg["vocab"], n)]
        margins = []
        M.forward(cfg, w, toks, margins=margins)
        if not margins or min(margins) > need:
            return toks
    raise AssertionError("no token sequence keeps the routers away from ties")
