"""Mixers side by side: several mixers read the same input, each one's output passes an RMS norm of its own over the
model width, and the result is the mean of the normed outputs.

    result = (1 / n) sum_j  y_j / sqrt(mean(y_j^2) + eps) * w_j,      y_j = mixer_j(h)

Mixers that allow it (Mixer.splits_projection) have their input projections run as one product over the stacked
matrices.  What a sequence keeps is what each mixer keeps, in the mixers' order.  An arrangement that forms a sum anyway
takes the outputs as terms (Mixer.gives_terms), normed and added by its own kernel; the factor 1 / n rides on the gains.
"""
from __future__ import annotations

from typing import Dict, List, Mapping, Optional

import torch

from .. import kernels as K
from ..cache.store import LayerCache
from .base import Mixer, Term
from .latent_attention import padded
from .linear import STORE_F32, Linear
from .registry import find_part, register_part
from .spec import TensorSpec


@register_part("mixer", "mixer_mean")
class MixerMean(Mixer):
    """params: hidden, mixers (a list of PartSpecs, with prefixes of their own), norms (the names of the norms' weights,
    in the same order), eps, prefix."""
    gives_terms = True
    stores_output = True

    def __init__(self, spec, runtime):
        super().__init__(spec, runtime)
        self.hidden, self.eps = int(spec["hidden"]), float(spec["eps"])
        self.mixers: List[Mixer] = [find_part("mixer", ps.kind)(ps, runtime) for ps in spec["mixers"]]
        self.norm_names = [self.prefix + str(n) for n in spec["norms"]]
        if not 1 <= len(self.mixers) <= K.SUM_NORM_TERMS or len(self.norm_names) != len(self.mixers):
            raise ValueError(f"mixer_mean takes one to {K.SUM_NORM_TERMS} mixers and a norm for each")
        self.w_in: Optional[Linear] = None
        self.columns: List[Optional[tuple]] = [None] * len(self.mixers)

    def tensors(self) -> Dict[str, TensorSpec]:
        t: Dict[str, TensorSpec] = {}
        for m, name in zip(self.mixers, self.norm_names):
            t.update(m.tensors())
            t[name] = TensorSpec((self.hidden,), role="vector", init="ones")
        return t

    def bind(self, weights: Mapping[str, torch.Tensor]) -> None:
        for m in self.mixers:
            if m.splits_projection:
                m.bind(weights, own_projection=False)
            else:
                m.bind(weights)
        self.gains = [(weights[n] / len(self.mixers)).contiguous() for n in self.norm_names]
        stack, biases, col = [], [], 0
        for i, m in enumerate(self.mixers):
            if not m.splits_projection:
                continue
            w, b = m.input_weights(weights)
            n = w.shape[0]
            gap = padded(n) - n                       # every mixer's columns begin on a boundary of eight
            if gap:
                w = torch.cat([w, torch.zeros(gap, w.shape[1], dtype=w.dtype, device=w.device)])
            full = torch.zeros(n + gap, dtype=torch.float32, device=w.device)
            if b is not None:
                full[:n] = b
            stack.append(w)
            biases.append(full)
            self.columns[i] = (col, col + n)
            col += n + gap
        self.width = col
        if stack:
            bias = torch.cat(biases).contiguous()
            self.w_in = Linear(self.runtime, torch.cat(stack, dim=0).contiguous(), bias if bool(bias.any()) else None)

    def cache_spec(self):
        return tuple(m.cache_spec() for m in self.mixers)

    def terms(self, xin, step, cache: LayerCache) -> List[Term]:
        T = xin.shape[0]
        proj = None
        if self.w_in is not None:
            proj = self.runtime.empty(T, self.width, dtype=torch.float32)
            self.w_in(xin, out=proj, mode=STORE_F32)
        out = []
        for m, gain, cols, view in zip(self.mixers, self.gains, self.columns, cache.parts):
            y = self.runtime.empty(T, self.hidden, dtype=torch.float32)
            kw = {} if cols is None else {"proj": proj[:, cols[0]:cols[1]]}
            if m.stores_output:
                m.forward(xin, y, step, view, store=True, **kw)
            else:
                y.zero_()
                m.forward(xin, y, step, view, **kw)
            out.append(Term(y, gain, self.eps))
        return out

    def forward(self, xin, residual: torch.Tensor, step, cache: LayerCache, store: bool = False) -> None:
        K.sum_norm(residual, 0.0 if store else 1.0, self.terms(xin, step, cache), None, 0, 0.0, residual)
