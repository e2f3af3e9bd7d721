"""Grouped-query attention whose queries, keys and values pass a short causal convolution over time, with a linear
distance bias in place of a position encoding.

Per token, with h the mixer's input and p its position:  u = W h + b, the rows of Wq ([heads][d]), Wk ([kv heads][d]) and
Wv ([kv heads][dv]) one above the other; channel by channel  y_p = sum_j w_j u_(p - taps + 1 + j)  (inputs before the
sequence's start are zero); q, k, v = y.  Values may be mixed with those of an earlier layer for the same token,
v <- (1 - lambda) v + lambda v_first.  Head j (kv head j / (heads / kv heads)):

    s_t = (q_j . k_t) * scale - slope_j (p - t)       for the keys t with 0 <= p - t < window (window 0: every t <= p)
    o_j = sum_t softmax_t(s) v_t;      result = Wo concat_j(o_j) + bo

Per sequence it keeps keys and values in pages and, with a convolution, the last taps - 1 rows u in a block of state of
fixed size (float32).  One product makes u with float32 sums; one kernel does everything from there to the rounded
queries and the appended keys and values (csrc/short_conv.cu); the attention is the general one (kernels.AttentionShape).
"""
from __future__ import annotations

from typing import Dict, Mapping, Optional

import torch

from .. import kernels as K
from ..cache.pages import PAGE_TOKENS
from ..cache.store import KVSpec, LayerCache, StateSpec
from .base import Mixer
from .latent_attention import padded
from .linear import ADD_TO_F32, STORE_F32, Linear
from .registry import register_part
from .spec import TensorSpec

RUN_TOKENS = 8                # tokens of a sequence that a thread of the convolution takes, at least


def geometric_slopes(n_heads: int):
    """2^(-8 (h + 1) / H), h = 0 .. H - 1."""
    return tuple(2.0 ** (-8.0 * (h + 1) / n_heads) for h in range(n_heads))


@register_part("mixer", "conv_attention")
class ConvAttention(Mixer):
    """params: hidden, n_heads, n_kv_heads, head_dim, v_dim, scale, window (0: all keys), taps (0: no convolution), bias
    (biases on all four projections: name + ".b"), slopes (None, or a number per head), value_mix (None; "first": this
    layer's values are left for later layers of the step; "mix": they are mixed with those left, with the learned share
    vmix; both expect the tensor), prefix, and the tensor names q, k, v, o, vmix (defaults: those words; the convolutions'
    are name + ".conv")."""
    stores_output = True

    def __init__(self, spec, runtime):
        super().__init__(spec, runtime)
        self.hidden, self.n_heads, self.n_kv = int(spec["hidden"]), int(spec["n_heads"]), int(spec["n_kv_heads"])
        self.d, self.dv = int(spec["head_dim"]), int(spec["v_dim"])
        if self.n_heads % self.n_kv:
            raise ValueError(f"attention: {self.n_heads} heads are not a multiple of {self.n_kv} kv heads")
        self.scale, self.window = float(spec["scale"]), int(spec.get("window", 0) or 0)
        self.taps = int(spec.get("taps", 0) or 0)
        self.bias = bool(spec.get("bias", False))
        self.slopes = spec.get("slopes")
        if self.slopes is not None and len(self.slopes) != self.n_heads:
            raise ValueError(f"conv_attention: {len(self.slopes)} slopes for {self.n_heads} heads")
        self.value_mix = spec.get("value_mix")
        if self.value_mix not in (None, "first", "mix"):
            raise ValueError(f"conv_attention: value_mix {self.value_mix!r} is not one of None, 'first', 'mix'")
        self.names = {k: self.prefix + str(spec.get(k + "_tensor", k)) for k in ("q", "k", "v", "o", "vmix")}
        self.cols = {"q": self.n_heads * self.d, "k": self.n_kv * self.d, "v": self.n_kv * self.dv}
        self.width, self.o_cols = sum(self.cols.values()), self.n_heads * self.dv
        self.w_in: Optional[Linear] = None
        self.w_o: Optional[Linear] = None
        self.shape: Optional[K.AttentionShape] = None

    def tensors(self) -> Dict[str, TensorSpec]:
        n = self.names
        t = {n[key]: TensorSpec((rows, self.hidden)) for key, rows in self.cols.items()}
        t[n["o"]] = TensorSpec((self.hidden, self.o_cols))
        if self.bias:
            t.update({n[key] + ".b": TensorSpec((rows,), role="vector", init="zeros")
                      for key, rows in list(self.cols.items()) + [("o", self.hidden)]})
        if self.taps:
            t.update({n[key] + ".conv": TensorSpec((rows, self.taps), role="vector") for key, rows in self.cols.items()})
        if self.value_mix:
            t[n["vmix"]] = TensorSpec((), role="vector")
        return t

    def bind(self, weights: Mapping[str, torch.Tensor]) -> None:
        n = self.names
        b = torch.cat([weights[n[key] + ".b"] for key in self.cols]).contiguous() if self.bias else None
        self.w_in = Linear(self.runtime, torch.cat([weights[n[key]] for key in self.cols], dim=0).contiguous(), b)
        self.w_o = Linear(self.runtime, weights[n["o"]], weights[n["o"] + ".b"] if self.bias else None)
        self.conv_w = None
        if self.taps:
            self.conv_w = torch.cat([weights[n[key] + ".conv"] for key in self.cols], dim=0).t().contiguous()
        self.lam = weights[n["vmix"]].reshape(1).contiguous() if self.value_mix == "mix" else None
        slope = None
        if self.slopes is not None:
            slope = torch.tensor(self.slopes, dtype=torch.float32, device=self.runtime.device)
        self.shape = K.AttentionShape(self.n_heads, self.n_heads // self.n_kv, 1, self.d, self.dv, False, self.scale,
                                      window=self.window, slope=slope)

    def cache_spec(self):
        kv = KVSpec(self.n_kv, self.d, self.window, "convolved" if self.taps else "as_projected", value_heads=self.n_kv,
                    value_dim=self.dv)
        return (kv, StateSpec(((self.taps - 1) * self.width,), "float32")) if self.taps > 1 else kv

    def forward(self, xin, residual: torch.Tensor, step, cache: LayerCache, store: bool = False) -> None:
        T = xin.shape[0]
        kv, state = (cache.parts[0], cache.parts[1].state) if self.taps > 1 else (cache, None)
        u = self.runtime.empty(T, padded(self.width), dtype=torch.float32)[:, :self.width]
        self.w_in(xin, out=u, mode=STORE_F32)
        first_in = first_out = None
        if self.value_mix == "mix":
            first_in = step.kept["values"]
        elif self.value_mix == "first":
            first_out = step.kept["values"] = self.runtime.empty(T, padded(self.cols["v"]))
        runs = None if step.all_single else step.query_blocks(padded(max(RUN_TOKENS, self.taps - 1)))
        q = self.runtime.empty(T, padded(self.cols["q"]))
        K.short_conv(u, self.conv_w, step, runs, state, kv.block_table, q, kv.k, kv.v, self.n_heads, self.n_kv, self.d, self.dv,
                     PAGE_TOKENS, cache.writes, self.lam, first_in, first_out)
        out = self.runtime.empty(T, padded(self.o_cols))
        from . import attention_dispatch
        attention_dispatch.run_general(self, self.shape, q, kv, step, out)
        self.w_o(out[:, :self.o_cols], out=residual, mode=STORE_F32 if store else ADD_TO_F32)
