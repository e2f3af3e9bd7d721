"""A gated linear recurrence on two branches (the recurrent block of Griffin with its real-gated linear recurrent unit):
per sequence it keeps one number per channel in float32.

Per token, with h the mixer's input:  y = gelu_tanh(Wy h + by);  u = the causal convolution over time, per channel, of
Wx h + bx (`taps` taps and a bias, the last tap the current token's, zeros before the sequence's start).  u is cut into
`blocks` equal parts; in part b, with square matrices A_b and B_b:

    r = sigmoid(A_b u_b + a_b),   i = sigmoid(B_b u_b + c_b)
    log a = -8 r softplus(lam);   S <- a S + sqrt(1 - a^2) i u;      result = Wo (S y)

What a sequence keeps between steps is S and the convolution's last inputs: a block of fixed size per sequence
(cache.StateSpec).  Both input projections run as one product with float32 sums; everything between it and the output
product is float32 (csrc/lru.cu): prompts by a convolution, the gates' block-diagonal product and a scan over time in
parallel stretches; bfloat16 decode steps by one kernel that does all three.
"""
from __future__ import annotations

from typing import Dict, Mapping, Optional

import torch

from .. import kernels as K
from ..cache.store import LayerCache, StateSpec
from .base import Mixer
from .latent_attention import padded
from .linear import ADD_TO_F32, STORE_F32, Linear
from .registry import register_part
from .spec import TensorSpec

DECAY_STRENGTH = 8.0


@register_part("mixer", "gated_linear_recurrence")
class GatedLinearRecurrence(Mixer):
    """params: hidden, width, blocks, taps, prefix, and the tensor names y, x, conv, ra, ri, lam, o (defaults: those words;
    every bias is its tensor's name + ".b")."""
    stores_output = True
    splits_projection = True

    def __init__(self, spec, runtime):
        super().__init__(spec, runtime)
        self.hidden, self.width = int(spec["hidden"]), int(spec["width"])
        self.blocks, self.taps = int(spec["blocks"]), int(spec["taps"])
        if self.width % self.blocks:
            raise ValueError(f"linear recurrence: {self.width} channels do not form {self.blocks} equal blocks")
        self.size = self.width // self.blocks
        self.names = {k: self.prefix + str(spec.get(k + "_tensor", k)) for k in ("y", "x", "conv", "ra", "ri", "lam", "o")}
        self.w_in: Optional[Linear] = None
        self.w_o: Optional[Linear] = None

    def tensors(self) -> Dict[str, TensorSpec]:
        n, H, W, B, S = self.names, self.hidden, self.width, self.blocks, self.size
        t = {n["o"]: TensorSpec((H, W)), n["lam"]: TensorSpec((W,), role="vector", init="ones"),
             n["conv"]: TensorSpec((W, self.taps), role="vector"),
             n["conv"] + ".b": TensorSpec((W,), role="vector", init="zeros")}
        for key in ("y", "x"):
            t[n[key]] = TensorSpec((W, H))
            t[n[key] + ".b"] = TensorSpec((W,), role="vector", init="zeros")
        for key in ("ra", "ri"):
            t[n[key]] = TensorSpec((B, S, S))
            t[n[key] + ".b"] = TensorSpec((B, S), role="vector", init="zeros")
        return t

    def input_weights(self, weights: Mapping[str, torch.Tensor]):
        n = self.names
        return (torch.cat([weights[n["y"]], weights[n["x"]]], dim=0).contiguous(),
                torch.cat([weights[n["y"] + ".b"], weights[n["x"] + ".b"]]).contiguous())

    def bind(self, weights: Mapping[str, torch.Tensor], own_projection: bool = True) -> None:
        n = self.names
        if own_projection:
            self.w_in = Linear(self.runtime, *self.input_weights(weights))
        self.w_o = Linear(self.runtime, weights[n["o"]])
        gates = torch.cat([weights[n["ra"]], weights[n["ri"]]], dim=1).contiguous()           # [blocks][2 size][size]
        bias = torch.cat([weights[n["ra"] + ".b"], weights[n["ri"] + ".b"]], dim=1).contiguous()
        # what multiplies r in log a: evaluated once, in float64, rounded to float32
        rate = (-DECAY_STRENGTH * torch.nn.functional.softplus(weights[n["lam"]].double())).float().contiguous()
        self.unit = K.LinearRecurrence(weights[n["conv"]].t().contiguous(), weights[n["conv"] + ".b"].contiguous(), gates,
                                       bias, rate)

    def cache_spec(self) -> StateSpec:
        return StateSpec(((1 + self.taps) * self.width,), "float32")

    def forward(self, xin, residual: torch.Tensor, step, cache: LayerCache, store: bool = False, proj=None) -> None:
        T = xin.shape[0]
        if proj is None:
            proj = self.runtime.empty(T, padded(2 * self.width), dtype=torch.float32)[:, :2 * self.width]
            self.w_in(xin, out=proj, mode=STORE_F32)
        out = self.runtime.empty(T, padded(self.width))
        self.unit.run(self.runtime, proj, out, cache.state, step, cache.writes)
        self.w_o(out[:, :self.width], out=residual, mode=STORE_F32 if store else ADD_TO_F32)
