"""MemipelConfig: the sizes and constants of a Memipel decoder, read from config.json.

A Memipel config.json names its architecture under "architecture", gives "vocab", "width", "norm": {"eps"} and lists its
layers one by one: each entry gives the mixer's kind ("type": "attention", "latent_attention" or "lightning"), the mixer's
sizes and constants ("mixer") and its feed-forward ("mlp": dense or a mixture of experts, or null for a layer that is a
mixer alone).  Nothing about a layer is assumed from another layer: sizes and constants may differ from one entry to the
next, and the kinds may come in any order.

  attention         heads, kv_heads, dim, vdim, scale, conv (taps; absent: no convolution), v_mix, mask: {size}
  latent_attention  heads, dim, vdim, q_rank, kv_rank, scale, mask: {size}
  lightning         heads, dim, vdim, decay (one number per head)
  mlp dense         kind "dense"; ff
  mlp moe           kind "moe"; router: {experts, top, groups: {count, keep}}, expert: {ff, limit}, shared: {ff, limit}
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Optional, Tuple

from .base import KeyReader, ModelConfig

MIXER_KINDS = ("attention", "latent_attention", "lightning")
MLP_KINDS = ("dense", "moe")


def _window(r: KeyReader) -> int:
    mk = r.child("mask")             # a mixer without "mask" sees every earlier key
    if mk is None:
        return 0
    size = mk.integer("size", lo=1, hi=1 << 30)
    r.adopt(mk)
    return size or 0


@dataclass(frozen=True)
class MemipelAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    conv: int = 0                    # taps of the convolution; 0: none
    v_mix: bool = False
    window: int = 0

    @classmethod
    def from_reader(cls, r: KeyReader) -> "MemipelAttention":
        heads, kv = r.integer("heads", hi=1 << 14), r.integer("kv_heads", hi=1 << 14)
        dim, vdim = r.integer("dim", hi=1 << 14), r.integer("vdim", hi=1 << 14)
        if heads and kv:
            r.require(heads % kv == 0, f"heads={heads} is not a multiple of kv_heads={kv}")
        return cls(heads, kv, dim, vdim, r.number("scale"), r.integer("conv", default=0, lo=0, hi=64),
                   r.boolean("v_mix", default=False), _window(r))

    def to_dict(self) -> Dict[str, Any]:
        d = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale,
             "v_mix": self.v_mix}
        if self.conv:
            d["conv"] = self.conv
        if self.window:
            d["mask"] = {"size": self.window}
        return d


@dataclass(frozen=True)
class MemipelLatentAttention:
    heads: int
    dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    window: int = 0

    @classmethod
    def from_reader(cls, r: KeyReader) -> "MemipelLatentAttention":
        return cls(r.integer("heads", hi=1 << 14), r.integer("dim", hi=1 << 14), r.integer("vdim", hi=1 << 14),
                   r.integer("q_rank", hi=1 << 16), r.integer("kv_rank", hi=1 << 14), r.number("scale"), _window(r))

    def to_dict(self) -> Dict[str, Any]:
        d = {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "q_rank": self.q_rank, "kv_rank": self.kv_rank,
             "scale": self.scale}
        if self.window:
            d["mask"] = {"size": self.window}
        return d


@dataclass(frozen=True)
class LightningConfig:
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]

    @classmethod
    def from_reader(cls, r: KeyReader) -> "LightningConfig":
        heads, dim, vdim = r.integer("heads", hi=1 << 14), r.integer("dim", hi=512), r.integer("vdim", hi=1 << 14)
        decay = r.raw.get("decay")
        if not isinstance(decay, list) or not all(isinstance(v, (int, float)) and not isinstance(v, bool) for v in decay):
            r.problems.append("'decay' must be a list of numbers")
            decay = []
        elif heads:
            r.require(len(decay) == heads, f"'decay' has {len(decay)} numbers for {heads} heads")
        return cls(heads, dim, vdim, tuple(float(v) for v in decay))

    def to_dict(self) -> Dict[str, Any]:
        return {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "decay": list(self.decay)}


_MIXER_CONFIGS = {"attention": MemipelAttention, "latent_attention": MemipelLatentAttention, "lightning": LightningConfig}


@dataclass(frozen=True)
class ClampedExpert:
    ff: int
    limit: float

    @classmethod
    def from_reader(cls, r: KeyReader) -> "ClampedExpert":
        return cls(r.integer("ff", hi=1 << 24), r.number("limit", lo=0.0))

    def to_dict(self) -> Dict[str, Any]:
        return {"ff": self.ff, "limit": self.limit}


@dataclass(frozen=True)
class MemipelMlp:
    kind: str
    ff: int = 0                              # dense
    experts: int = 0                         # moe, as everything below
    top: int = 0
    groups: int = 1
    keep: int = 1
    expert: Optional[ClampedExpert] = None
    shared: Optional[ClampedExpert] = None   # None: no shared expert

    @classmethod
    def from_reader(cls, r: KeyReader) -> "MemipelMlp":
        kind = r.string("kind", choices=MLP_KINDS)
        if kind != "moe":
            return cls(kind or "dense", ff=r.integer("ff", hi=1 << 24) or 0)
        experts = top = 0
        groups = keep = 1
        rt = r.child("router")
        if rt is None:
            r.problems.append("missing required key 'router'")
        else:
            experts, top = rt.integer("experts", hi=1 << 12), rt.integer("top", hi=1 << 12)
            gr = rt.child("groups")          # absent: one group
            if gr is not None:
                groups, keep = gr.integer("count", hi=1 << 12), gr.integer("keep", hi=1 << 12)
                rt.adopt(gr)
            if experts and top and groups and keep:
                rt.require(experts % groups == 0, f"experts={experts} do not form groups.count={groups} equal groups")
                rt.require(keep <= groups, f"groups.keep={keep} of groups.count={groups}")
                rt.require(top <= (experts // groups) * keep,
                           f"top={top} of {(experts // groups) * keep} experts that can be chosen")
            r.adopt(rt)
        built = {}
        for key in ("expert", "shared"):
            sub = r.child(key)
            if sub is not None:
                built[key] = ClampedExpert.from_reader(sub)
                r.adopt(sub)
            elif key == "expert":
                r.problems.append("missing required key 'expert'")
        return cls(kind, experts=experts or 0, top=top or 0, groups=groups or 1, keep=keep or 1, **built)

    def to_dict(self) -> Dict[str, Any]:
        if self.kind == "dense":
            return {"kind": "dense", "ff": self.ff}
        d = {"kind": "moe", "expert": self.expert.to_dict(),
             "router": {"experts": self.experts, "top": self.top, "groups": {"count": self.groups, "keep": self.keep}}}
        if self.shared is not None:
            d["shared"] = self.shared.to_dict()
        return d


@dataclass(frozen=True)
class MemipelLayer:
    kind: str                            # one of MIXER_KINDS
    mixer: Any
    mlp: Optional[MemipelMlp]            # None: no feed-forward

    def to_dict(self) -> Dict[str, Any]:
        return {"type": self.kind, "mixer": self.mixer.to_dict(), "mlp": None if self.mlp is None else self.mlp.to_dict()}


@dataclass(frozen=True)
class MemipelConfig(ModelConfig):
    vocab: int
    width: int
    eps: float
    layers: Tuple[MemipelLayer, ...]
    torch_dtype: str = "bfloat16"

    architecture = "Memipel"

    @classmethod
    def from_dict(cls, raw: Dict[str, Any]) -> "MemipelConfig":
        r = KeyReader(raw)
        vocab, width = r.integer("vocab", hi=1 << 26), r.integer("width", hi=1 << 20)
        norm = r.child("norm")
        eps = None
        if norm is None:
            r.problems.append("missing required key 'norm'")
        else:
            eps = norm.number("eps", lo=0.0, hi=1.0)
            r.adopt(norm)
        entries = raw.get("layers")
        layers = []
        if not isinstance(entries, list) or not entries:
            r.problems.append("'layers' must be a non-empty list")
            entries = []
        mixed = None                     # the layer whose values the later ones mix in
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
                mlp = MemipelMlp.from_reader(fr)
                lr.adopt(fr)
            if kind == "attention" and mixer is not None and mixer.v_mix and mixer.kv_heads and mixer.vdim:
                size = mixer.kv_heads * mixer.vdim
                if mixed is None:
                    mixed = (i, size)
                lr.require(size == mixed[1], f"mixes its {size} values with the {mixed[1]} of layers[{mixed[0]}]")
            layers.append(MemipelLayer(kind, mixer, mlp))
            r.adopt(lr)
        r.finish()
        return cls(vocab=vocab, width=width, eps=eps, layers=tuple(layers), torch_dtype=raw.get("torch_dtype", "bfloat16"))

    def to_dict(self) -> Dict[str, Any]:
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps},
                "layers": [layer.to_dict() for layer in self.layers], "torch_dtype": self.torch_dtype}
