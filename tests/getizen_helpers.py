"""Small Getizen configurations and model folders for the tests.  None of them is anyone's model: sizes are chosen so that
no two of a layer's sizes are equal by accident, that counts are not 1 where the formulas divide by them, and that the
layers of one model differ from one another (heads, key and value sizes, rotated dimensions, chunks, blocks, taps,
decays)."""
import torch

from helpers import load_plain, make_model_dir
from mokatar_helpers import assert_rows_close  # noqa: F401  (the same comparison)
from plain import getizen_plain as G


def left(heads=4, kv=2, dim=24, vdim=16, rot=12, base=10000.0, scale=0.2, factor=4.0, low=1.0, high=4.0, original=64,
         chunk=50):
    d = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale,
         "rot": {"base": base, "dims": rot, "scaling": {"factor": factor, "low": low, "high": high, "original": original}}}
    if chunk:
        d["mask"] = {"size": chunk}
    return d


def right(width=60, blocks=5, conv=3):
    return {"width": width, "blocks": blocks, "conv": conv}


def parallel(lf=None, rt=None):
    return {"left": lf or left(), "right": rt or right()}


def retention(heads=3, dim=12, vdim=20, rot=8, base=1000.0, decay=None):
    return {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay or [1.0 - 2.0 ** (-2 - 2 * h) for h in range(heads)],
            "rot": {"base": base, "dims": rot}}


def dense(ff=96, limit=1.2):
    return {"kind": "dense", "ff": ff, "limit": limit}


def layer(kind, mixer, mlp=None):
    return {"type": kind, "mixer": mixer, "mlp": mlp}


def config(layers, vocab=211, width=72, eps=1e-5, groups=3, alpha=1.7):
    return {"architecture": "Getizen", "vocab": vocab, "width": width, "norm": {"eps": eps, "groups": groups},
            "postln_alpha": alpha, "layers": layers}


# block sizes of 12 (the float32 products of the CUDA cores in both dtypes); the layers' constants differ
GET_A = config([layer("parallel", parallel(), dense()),
                layer("retention", retention(), dense(80, 0.9)),
                layer("parallel", parallel(left(heads=6, kv=6, dim=16, vdim=20, rot=16, chunk=33, original=128, factor=2.0),
                                           right(width=44, blocks=2, conv=4))),
                layer("retention", retention(heads=2, dim=20, vdim=8, rot=20, base=50.0))])
# sizes that no vector load divides: every fallback kernel; one tap, one kv head, one block, six taps, tiny chunks
GET_B = config([layer("parallel", parallel(left(heads=3, kv=1, dim=18, vdim=10, rot=18, chunk=5, factor=0.5, original=20),
                                           right(width=35, blocks=7, conv=1)), dense(50, 3.0)),
                layer("retention", retention(heads=1, dim=9, vdim=7, rot=4)),
                layer("parallel", parallel(left(heads=2, kv=2, dim=7, vdim=5, rot=2, chunk=0, scale=-0.4),
                                           right(width=22, blocks=1, conv=6)), dense(34, 0.7))],
               vocab=97, width=70, eps=1e-6, groups=5, alpha=0.8)
# sizes of the tensor-core kernels: eight query heads on a kv head, chunks longer and shorter than pages, blocks of 64
# and of 264 (no multiple of 32) channels, values larger than keys
GET_TC = config([layer("parallel", parallel(left(heads=8, kv=1, dim=64, vdim=64, rot=32, scale=0.1, chunk=130, original=32),
                                            right(width=192, blocks=3, conv=4)), dense(160, 2.0)),
                 layer("retention", retention(heads=4, dim=64, vdim=32, rot=64), dense(96, 1.1)),
                 layer("parallel", parallel(left(heads=4, kv=4, dim=32, vdim=48, rot=32, scale=0.15, chunk=64, original=300),
                                            right(width=264, blocks=1, conv=2)), dense(160, 1.3))],
                vocab=331, width=128, groups=2)
# heads of 128 and of 64 in groups, keys and values of one size: the prompt kernel for such heads; retention with wide heads
GET_BIG = config([layer("parallel", parallel(left(heads=4, kv=2, dim=128, vdim=128, rot=128, scale=0.08, chunk=150, original=256),
                                             right(width=128, blocks=4, conv=4)), dense(192, 1.6)),
                  layer("parallel", parallel(left(heads=4, kv=2, dim=64, vdim=64, rot=64, scale=0.12, chunk=0),
                                             right(width=320, blocks=2, conv=3))),
                  layer("retention", retention(heads=2, dim=128, vdim=128, rot=128, base=5000.0,
                                               decay=[0.96, 1.0 - 2.0 ** -9]), dense(128, 0.8))],
                 vocab=257, width=192, groups=1, alpha=2.3)
# one mechanism each, alone
GET_PARALLEL = config([layer("parallel", parallel(left(heads=4, kv=2, dim=16, vdim=16, rot=8, chunk=40), right(width=48, blocks=3)))],
                      width=64, groups=2)
GET_RETENTION = config([layer("retention", retention(heads=4, dim=8, vdim=16, rot=4))], width=64, groups=4)
GET_DENSE = config([layer("retention", retention(heads=1, dim=8, vdim=8, rot=2), dense(120, 0.6))], width=64, groups=1)

CONFIGS = {"A": GET_A, "B": GET_B, "TC": GET_TC, "BIG": GET_BIG, "parallel": GET_PARALLEL, "retention": GET_RETENTION,
           "dense": GET_DENSE}


def lively(tensors, seed=0):
    """Random weights as the writer makes them are tame: gains and factors of one, biases of zero, decays that are all
    alike.  Give every constant a value of its own and make scores and gates spread."""
    g = torch.Generator().manual_seed(seed)
    rnd = lambda t, lo, hi: (torch.rand(t.shape, generator=g) * (hi - lo) + lo).to(t.dtype)      # noqa: E731
    for name, t in list(tensors.items()):
        if name.endswith(("norm1", "norm2", "embed.norm", "final.norm", ".q.norm", ".k.norm", ".out")):
            tensors[name] = rnd(t, 0.5, 1.5)
        elif name.endswith(".temp"):
            tensors[name] = rnd(t, 0.4, 2.0)
        elif name.endswith(".lam"):
            tensors[name] = rnd(t, -7.0, 0.5)                       # from nearly no decay to a quick one
        elif name.endswith(".conv"):
            tensors[name] = rnd(t, -0.7, 0.7)
        elif name.endswith((".b",)):
            tensors[name] = rnd(t, -0.5, 0.5)
        elif name.endswith((".ra", ".ri")):
            tensors[name] = (t.float() * 6).to(t.dtype)
        elif name == "embed":
            tensors[name] = (t.float() * 10).to(t.dtype)
        else:
            tensors[name] = (t.float() * 2.5).to(t.dtype)


def make(path, name, dtype, seed=0, edit=None, cfg=None):
    def both(tensors):
        lively(tensors, seed)
        if edit is not None:
            edit(tensors)
    path = make_model_dir(path, cfg or CONFIGS[name], seed=seed, dtype=dtype, std=0.05, edit=both)
    cfg, w = load_plain(path)
    return path, cfg, w


def plain_logits(cfg, w, tokens):
    return G.forward(cfg, w, tokens)
