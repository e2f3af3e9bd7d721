"""Retention: linear attention with a fixed decay per head, without a softmax or a denominator; per sequence and head
it keeps one matrix S [d][dv] in float32.

Per token, with h the mixer's input and p its position:  q = Wq h, k = Wk h ([heads][d]), v = Wv h ([heads][dv]); the
first dimensions of every head of q and k are rotated by the position encoding, in pairs (i, i + n/2) or (2i, 2i + 1).
Head j, with its constant decay c_j:

    S <- c_j S + k v^T;   o = S^T q / sqrt(d)          (o sees the token's own write)

    o <- o / sqrt(mean(o^2) + eps) * silu(Wg h)_j;     result = Wo concat_j(o)

Variants, each a parameter: q, k and v taken through silu before they enter the recurrence (`activation: silu`); the heads'
read-outs normed together, with a weight, and gated by sigmoid(Wg h) (`norm: whole`); a scale of one's own.  Lightning
attention is retention with all three and no rotation.

The four projections run as one product with float32 sums; everything from there to the output product is float32
(csrc/gla.cu, the kernels of gated linear attention with a decay per head in place of one per token and key channel; the
prompts of the bfloat16 path go chunk by chunk through tensor cores, csrc/gla_chunked.cu).
"""
from __future__ import annotations

from typing import Dict, Mapping, Optional

import torch

from .. import kernels as K
from ..cache.store import LayerCache, StateSpec
from .base import Mixer
from .latent_attention import padded
from .linear import ADD_TO_F32, STORE_F32, Linear
from .registry import find_part, register_part
from .spec import PartSpec, TensorSpec


CHUNKED_FROM = 16             # new tokens of a sequence from which a step goes through chunks


@register_part("mixer", "retention")
class Retention(Mixer):
    """params: hidden, n_heads, head_dim, v_dim, decay (a number per head), eps (of the heads' norm, which has no
    weight, or with norm "whole" of the norm over all heads together, whose weight has n_heads * v_dim values), activation (None
    or "silu", on q, k and v), position (PartSpec of a rotating position encoding, or None), scale (default head_dim^-1/2), prefix, and the
    tensor names q, k, v, g, o, norm (defaults: those words)."""
    stores_output = True

    def __init__(self, spec, runtime):
        super().__init__(spec, runtime)
        self.hidden, self.n_heads = int(spec["hidden"]), int(spec["n_heads"])
        self.d, self.dv, self.eps = int(spec["head_dim"]), int(spec["v_dim"]), float(spec["eps"])
        self.decay = tuple(float(v) for v in spec["decay"])
        if len(self.decay) != self.n_heads:
            raise ValueError(f"retention: {len(self.decay)} decays for {self.n_heads} heads")
        self.scale = float(spec.get("scale") or self.d ** -0.5)
        pos: Optional[PartSpec] = spec.get("position")
        self.position = find_part("position", pos.kind)(pos, runtime) if pos is not None else None
        if self.position is not None:
            layout = self.position.pair_layout()
            if layout is None or 2 * layout[0] > self.d:
                raise ValueError("retention rotates pairs among a head's first dimensions")
        self.names = {k: self.prefix + str(spec.get(k + "_tensor", k)) for k in ("q", "k", "v", "g", "o", "norm")}
        act, norm = spec.get("activation"), spec.get("norm", "per_head")
        if act not in (None, "silu") or norm not in ("per_head", "whole"):
            raise ValueError(f"retention: activation {act!r} or norm {norm!r} is not known")
        self.silu, self.whole = act == "silu", norm == "whole"
        self.gain: Optional[torch.Tensor] = None
        self.qk_cols, self.v_cols = self.n_heads * self.d, self.n_heads * self.dv
        self.width = 2 * self.qk_cols + 2 * self.v_cols
        self.w_in: Optional[Linear] = None
        self.w_o: Optional[Linear] = None

    def tensors(self) -> Dict[str, TensorSpec]:
        n, H = self.names, self.hidden
        t = {n["q"]: TensorSpec((self.qk_cols, H)), n["k"]: TensorSpec((self.qk_cols, H)),
             n["v"]: TensorSpec((self.v_cols, H)), n["g"]: TensorSpec((self.v_cols, H)),
             n["o"]: TensorSpec((H, self.v_cols))}
        if self.whole:
            t[n["norm"]] = TensorSpec((self.v_cols,), role="vector", init="ones")
        return t

    def bind(self, weights: Mapping[str, torch.Tensor]) -> None:
        n = self.names
        self.w_in = Linear(self.runtime, torch.cat([weights[n[k]] for k in ("q", "k", "v", "g")], dim=0).contiguous())
        self.w_o = Linear(self.runtime, weights[n["o"]])
        self.gain = weights[n["norm"]].contiguous() if self.whole else None
        self.head_decay = torch.tensor(self.decay, dtype=torch.float32, device=self.runtime.device)

    def cache_spec(self) -> StateSpec:
        return StateSpec((self.n_heads * self.d * self.dv,), "float32")

    def forward(self, xin, residual: torch.Tensor, step, cache: LayerCache, store: bool = False) -> None:
        T = xin.shape[0]
        f32 = torch.float32
        proj = self.runtime.empty(T, padded(self.width), dtype=f32)
        self.w_in(xin, out=proj[:, :self.width], mode=STORE_F32)
        step_ = K.GlaStep(proj, self.n_heads, self.d, self.dv, 0, 1.0, self.scale, self.eps, head_decay=self.head_decay,
                          silu_qkv=self.silu, norm_all=self.whole)
        if self.position is not None:
            rot = self.position.rotary()
            step_.rotate(step.rotation_table(rot), rot.interleaved)
        o_raw = self.runtime.empty(T, self.v_cols, dtype=f32)
        chunked = xin.dtype == torch.bfloat16 and step.max_new >= CHUNKED_FROM and step_.chunks_ok()
        step_.recur(o_raw, cache.state, step.token_seq, step.seq_start, step.seq_slot, cache.writes, chunked)
        out = self.runtime.empty(T, padded(self.v_cols))
        step_.finish(self.gain, out)
        self.w_o(out[:, :self.v_cols], out=residual, mode=STORE_F32 if store else ADD_TO_F32)
