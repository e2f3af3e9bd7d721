"""The Memipel decoder as data: MemipelConfig -> ModelSpec.

Every layer has one RMS norm (its weight stored around zero) whose rows both sublayers read, x += mixer(h) + ff(h); a layer
may have no feed-forward.  The mixer is attention behind a short convolution with a linear distance bias, whose values the
first such layer lends to the later ones; latent attention without positions and with a sink; or lightning attention with
state of a fixed size, layer by layer as the configuration lists them.  The feed-forward is dense (exact GELU) or a mixture
of experts with clamped gates chosen in groups by softmax scores, with a shared expert.  The head is the embedding table.
Tensor names: embed, l<i>.norm1, l<i>.mix.*, l<i>.mlp.*, final.norm.
"""
from __future__ import annotations

from ..config.memipel import MemipelConfig
from ..config.registry import Architecture, register_architecture
from ..parts.conv_attention import geometric_slopes
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry


def _mixer(cfg: MemipelConfig, layer, value_mix) -> PartSpec:
    m = layer.mixer
    if layer.kind == "attention":
        return PartSpec("conv_attention", {
            "hidden": cfg.width, "n_heads": m.heads, "n_kv_heads": m.kv_heads, "head_dim": m.dim, "v_dim": m.vdim,
            "scale": m.scale, "window": m.window, "taps": m.conv, "bias": True, "slopes": geometric_slopes(m.heads),
            "value_mix": value_mix, "prefix": "mix."})
    if layer.kind == "latent_attention":
        return PartSpec("latent_attention", {
            "hidden": cfg.width, "n_heads": m.heads, "head_dim": m.dim, "rot_dim": 0, "v_dim": m.vdim,
            "kv_rank": m.kv_rank, "q_rank": m.q_rank, "scale": m.scale, "eps": cfg.eps, "position": None, "sink": True,
            "window": m.window, "prefix": "mix."})
    return PartSpec("retention", {
        "hidden": cfg.width, "n_heads": m.heads, "head_dim": m.dim, "v_dim": m.vdim, "decay": m.decay, "eps": cfg.eps,
        "scale": 1.0, "activation": "silu", "norm": "whole", "prefix": "mix."})


def _feed_forward(cfg: MemipelConfig, f) -> PartSpec:
    if f.kind == "dense":
        return PartSpec("dense_gelu", {"hidden": cfg.width, "intermediate": f.ff, "activation": "gelu_erf", "prefix": "mlp."})
    return PartSpec("routed_experts", {
        "hidden": cfg.width, "n_experts": f.experts, "top": f.top, "scale": 1.0, "n_groups": f.groups, "keep": f.keep,
        "group_score": "max", "intermediate": f.expert.ff, "shared_intermediate": f.shared.ff if f.shared else None,
        "score": "softmax", "renorm": False, "correction": False, "activation": "clamped", "limit": f.expert.limit,
        "shared_limit": f.shared.limit if f.shared else None, "prefix": "mlp."})


def describe_memipel(cfg: MemipelConfig) -> ModelSpec:
    def norm(name):
        return PartSpec("rmsnorm", {"size": cfg.width, "eps": cfg.eps, "tensor": name, "one_plus": True})

    layers, lent = [], False
    for i, layer in enumerate(cfg.layers):
        value_mix = None
        if layer.kind == "attention" and layer.mixer.v_mix:
            value_mix, lent = ("mix" if lent else "first"), True
        parts = {"mixer_norm": norm("norm1"), "mixer": _mixer(cfg, layer, value_mix)}
        if layer.mlp is not None:
            parts["feed_forward"] = _feed_forward(cfg, layer.mlp)
        layers.append(LayerSpec("parallel_residual", parts, f"l{i}."))
    return ModelSpec(
        hidden=cfg.width, vocab=cfg.vocab,
        embedding=PartSpec("token_embedding", {"vocab": cfg.vocab, "hidden": cfg.width, "tensor": "embed"}),
        layers=tuple(layers), schedule=tuple(ScheduleEntry(i) for i in range(len(layers))),
        final_norm=norm("final.norm"),
        head=PartSpec("linear_head", {"vocab": cfg.vocab, "hidden": cfg.width, "own_matrix": False}))


MEMIPEL = register_architecture(Architecture(
    names=("Memipel",),
    description="Memipel decoder: sublayers side by side on one norm, attention behind short convolutions with distance "
                "biases, latent attention with sinks, lightning attention, clamped experts chosen in groups",
    config_class=MemipelConfig,
    describe_model=describe_memipel), replace=True)
