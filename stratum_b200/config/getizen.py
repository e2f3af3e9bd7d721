"""GetizenConfig: the sizes and constants of a Getizen decoder, read from config.json.

A Getizen config.json names its architecture under "architecture", gives "vocab", "width", "norm": {"eps", "groups"},
"postln_alpha" and lists its layers one by one: each entry gives the mixer's kind ("type": "parallel" or "retention"),
the mixer's sizes and constants ("mixer") and its feed-forward ("mlp": a dense one, or null for a layer that is a mixer
alone).  Nothing about a layer is assumed from another layer: sizes and constants may differ from one entry to the next,
and the kinds may come in any order.

  parallel    left: heads, kv_heads, dim, vdim, scale, rot: {base, dims, scaling: {factor, low, high, original}},
              mask: {size};  right: width, blocks, conv
  retention   heads, dim, vdim, decay (one number per head), rot: {base, dims}
  mlp dense   kind "dense"; ff, limit
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Optional, Tuple

from .base import KeyReader, ModelConfig

MIXER_KINDS = ("parallel", "retention")
MLP_KINDS = ("dense",)


@dataclass(frozen=True)
class WavelengthScaling:
    """Frequencies rescaled by their wavelength: kept below original / high, divided by `factor` above original / low,
    mixed in between."""
    factor: float
    low: float
    high: float
    original: float

    def to_dict(self) -> Dict[str, Any]:
        return {"factor": self.factor, "low": self.low, "high": self.high, "original": self.original}


@dataclass(frozen=True)
class GetizenRotation:
    base: float
    dims: int
    scaling: Optional[WavelengthScaling] = None

    @classmethod
    def from_reader(cls, r: KeyReader, head_dim: Optional[int]) -> "GetizenRotation":
        base, dims = r.number("base", lo=1.0), r.integer("dims", lo=0, hi=1 << 14)
        scaling = None
        sc = r.child("scaling")
        if sc is not None:
            scaling = WavelengthScaling(sc.number("factor", lo=1e-6), sc.number("low", lo=1e-6),
                                        sc.number("high", lo=1e-6), sc.number("original", lo=1e-6))
            r.adopt(sc)
        if dims and head_dim:
            r.require(dims % 2 == 0 and dims <= head_dim, f"rot.dims={dims} must be even and at most dim={head_dim}")
        return cls(base, dims, scaling)

    def to_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {"base": self.base, "dims": self.dims}
        if self.scaling is not None:
            d["scaling"] = self.scaling.to_dict()
        return d


def _rotation(r: KeyReader, head_dim: Optional[int]) -> Optional[GetizenRotation]:
    rr = r.child("rot")              # a mixer without "rot" rotates nothing
    if rr is None:
        return None
    rot = GetizenRotation.from_reader(rr, head_dim)
    r.adopt(rr)
    return rot


@dataclass(frozen=True)
class ChunkedAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: Optional[GetizenRotation]
    chunk: int = 0                   # mask.size; 0: every earlier key

    @classmethod
    def from_reader(cls, r: KeyReader) -> "ChunkedAttentionConfig":
        heads, kv = r.integer("heads", hi=1 << 14), r.integer("kv_heads", hi=1 << 14)
        dim, vdim = r.integer("dim", hi=1 << 14), r.integer("vdim", hi=1 << 14)
        scale = r.number("scale")
        rot = _rotation(r, dim)
        chunk = 0
        mk = r.child("mask")
        if mk is not None:
            chunk = mk.integer("size", lo=1, hi=1 << 30)
            r.adopt(mk)
        if heads and kv:
            r.require(heads % kv == 0, f"heads={heads} is not a multiple of kv_heads={kv}")
        return cls(heads, kv, dim, vdim, scale, rot, chunk or 0)

    def to_dict(self) -> Dict[str, Any]:
        d = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale}
        if self.rot is not None:
            d["rot"] = self.rot.to_dict()
        if self.chunk:
            d["mask"] = {"size": self.chunk}
        return d


@dataclass(frozen=True)
class RecurrentBlockConfig:
    width: int
    blocks: int
    conv: int                        # taps of the convolution

    @classmethod
    def from_reader(cls, r: KeyReader) -> "RecurrentBlockConfig":
        width, blocks = r.integer("width", hi=1 << 20), r.integer("blocks", hi=1 << 14)
        if width and blocks:
            r.require(width % blocks == 0, f"width={width} is not a multiple of blocks={blocks}")
        return cls(width, blocks, r.integer("conv", hi=64))

    def to_dict(self) -> Dict[str, Any]:
        return {"width": self.width, "blocks": self.blocks, "conv": self.conv}


@dataclass(frozen=True)
class ParallelMixerConfig:
    left: ChunkedAttentionConfig
    right: RecurrentBlockConfig

    @classmethod
    def from_reader(cls, r: KeyReader) -> Optional["ParallelMixerConfig"]:
        built = []
        for key, kind in (("left", ChunkedAttentionConfig), ("right", RecurrentBlockConfig)):
            sub = r.child(key)
            if sub is None:
                r.problems.append(f"missing required key '{key}'")
            else:
                built.append(kind.from_reader(sub))
                r.adopt(sub)
        return cls(*built) if len(built) == 2 else None

    def to_dict(self) -> Dict[str, Any]:
        return {"left": self.left.to_dict(), "right": self.right.to_dict()}


@dataclass(frozen=True)
class RetentionConfig:
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]
    rot: Optional[GetizenRotation]

    @classmethod
    def from_reader(cls, r: KeyReader) -> "RetentionConfig":
        heads, dim, vdim = r.integer("heads", hi=1 << 14), r.integer("dim", hi=512), r.integer("vdim", hi=1 << 14)
        decay = r.raw.get("decay")
        if not isinstance(decay, list) or not all(isinstance(v, (int, float)) and not isinstance(v, bool) for v in decay):
            r.problems.append("'decay' must be a list of numbers")
            decay = []
        elif heads:
            r.require(len(decay) == heads, f"'decay' has {len(decay)} numbers for {heads} heads")
        return cls(heads, dim, vdim, tuple(float(v) for v in decay), _rotation(r, dim))

    def to_dict(self) -> Dict[str, Any]:
        d = {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "decay": list(self.decay)}
        if self.rot is not None:
            d["rot"] = self.rot.to_dict()
        return d


_MIXER_CONFIGS = {"parallel": ParallelMixerConfig, "retention": RetentionConfig}


@dataclass(frozen=True)
class GetizenMlp:
    ff: int
    limit: float
    kind: str = "dense"

    @classmethod
    def from_reader(cls, r: KeyReader) -> "GetizenMlp":
        r.string("kind", choices=MLP_KINDS)
        return cls(ff=r.integer("ff", hi=1 << 24), limit=r.number("limit", lo=0.0))

    def to_dict(self) -> Dict[str, Any]:
        return {"kind": self.kind, "ff": self.ff, "limit": self.limit}


@dataclass(frozen=True)
class GetizenLayer:
    kind: str                            # one of MIXER_KINDS
    mixer: Any
    mlp: Optional[GetizenMlp]            # None: no feed-forward

    def to_dict(self) -> Dict[str, Any]:
        return {"type": self.kind, "mixer": self.mixer.to_dict(), "mlp": None if self.mlp is None else self.mlp.to_dict()}


@dataclass(frozen=True)
class GetizenConfig(ModelConfig):
    vocab: int
    width: int
    eps: float
    norm_groups: int
    alpha: float                         # the factor on the stream in front of a norm of the sum
    layers: Tuple[GetizenLayer, ...]
    torch_dtype: str = "bfloat16"

    architecture = "Getizen"

    @classmethod
    def from_dict(cls, raw: Dict[str, Any]) -> "GetizenConfig":
        r = KeyReader(raw)
        vocab, width = r.integer("vocab", hi=1 << 26), r.integer("width", hi=1 << 20)
        alpha = r.number("postln_alpha", default=1.0)
        norm = r.child("norm")
        eps = groups = None
        if norm is None:
            r.problems.append("missing required key 'norm'")
        else:
            eps = norm.number("eps", lo=0.0, hi=1.0)
            groups = norm.integer("groups", default=1, hi=1 << 14)
            r.adopt(norm)
            if width and groups:
                r.require(width % groups == 0, f"width={width} does not form norm.groups={groups} equal parts")
        entries = raw.get("layers")
        layers = []
        if not isinstance(entries, list) or not entries:
            r.problems.append("'layers' must be a non-empty list")
            entries = []
        for i, e in enumerate(entries):
            lr = KeyReader(e if isinstance(e, dict) else {}, f"config.json:layers[{i}]")
            if not isinstance(e, dict):
                lr.problems.append("must be an object")
            kind = lr.string("type", choices=MIXER_KINDS)
            mr = lr.child("mixer")
            mixer = mlp = None
            if mr is None:
                lr.problems.append("missing required key 'mixer'")
            elif kind is not None:
                mixer = _MIXER_CONFIGS[kind].from_reader(mr)
                lr.adopt(mr)
            fr = lr.child("mlp")
            if fr is not None:
                mlp = GetizenMlp.from_reader(fr)
                lr.adopt(fr)
            layers.append(GetizenLayer(kind, mixer, mlp))
            r.adopt(lr)
        r.finish()
        return cls(vocab=vocab, width=width, eps=eps, norm_groups=groups, alpha=alpha, layers=tuple(layers),
                   torch_dtype=raw.get("torch_dtype", "bfloat16"))

    def to_dict(self) -> Dict[str, Any]:
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
                "norm": {"eps": self.eps, "groups": self.norm_groups}, "postln_alpha": self.alpha,
                "layers": [layer.to_dict() for layer in self.layers], "torch_dtype": self.torch_dtype}
