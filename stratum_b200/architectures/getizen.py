"""The Getizen decoder as data: GetizenConfig -> ModelSpec.

The embedded tokens pass the model's norm; every layer then replaces the residual stream by the norm of its sum with a
sublayer's output, x = norm1(alpha x + mixer(x)); x = norm2(alpha x + ff(x)), the sublayers reading x itself (a layer
may have no feed-forward).  The norm is an RMS norm over equal groups of the row.  The mixer is a pair of mixers side by
side, attention within chunks (queries and keys normalised over the whole projection, a factor per head on the scores,
an output gate) and a gated linear recurrence, whose normed outputs are averaged; or retention with state of a fixed
size, layer by layer as the configuration lists them.  The feed-forward is dense with a clamped gate.  The head is the
embedding table.  Tensor names: embed, embed.norm, l<i>.norm1 / norm2, l<i>.mix.*, l<i>.mlp.*, final.norm.
"""
from __future__ import annotations

from ..config.getizen import GetizenConfig
from ..config.registry import Architecture, register_architecture
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry


def _rotation(rot):
    if rot is None or not rot.dims:
        return None
    scaling = None
    if rot.scaling is not None:
        s = rot.scaling
        scaling = {"kind": "llama3", "factor": s.factor, "low_freq_factor": s.low, "high_freq_factor": s.high,
                   "original_max_position": s.original}
    return PartSpec("rope", {"rope_dim": rot.dims, "theta": rot.base, "interleaved": False, "scaling": scaling,
                             "precise": True})


def _mixer(cfg: GetizenConfig, layer) -> PartSpec:
    m = layer.mixer
    if layer.kind == "retention":
        return PartSpec("retention", {
            "hidden": cfg.width, "n_heads": m.heads, "head_dim": m.dim, "v_dim": m.vdim, "decay": m.decay, "eps": cfg.eps,
            "position": _rotation(m.rot), "prefix": "mix."})
    a, r = m.left, m.right
    left = PartSpec("sink_attention", {
        "hidden": cfg.width, "n_heads": a.heads, "n_kv_heads": a.kv_heads, "head_dim": a.dim, "v_dim": a.vdim,
        "scale": a.scale, "chunk": a.chunk, "eps": cfg.eps, "position": _rotation(a.rot), "qk_norm": "whole",
        "sink": False, "temp": True, "gate": True, "prefix": "mix.left."})
    right = PartSpec("gated_linear_recurrence", {
        "hidden": cfg.width, "width": r.width, "blocks": r.blocks, "taps": r.conv, "prefix": "mix.right."})
    return PartSpec("mixer_mean", {"hidden": cfg.width, "mixers": (left, right), "norms": ("left.out", "right.out"),
                                   "eps": cfg.eps, "prefix": "mix."})


def describe_getizen(cfg: GetizenConfig) -> ModelSpec:
    def norm(name, stream=1.0):
        return PartSpec("grouped_rmsnorm", {"size": cfg.width, "groups": cfg.norm_groups, "eps": cfg.eps, "tensor": name,
                                            "stream": stream})

    layers = []
    for i, layer in enumerate(cfg.layers):
        parts = {"mixer": _mixer(cfg, layer), "mixer_norm": norm("norm1", cfg.alpha)}
        if layer.mlp is not None:
            parts.update({"feed_forward": PartSpec("swiglu", {
                "hidden": cfg.width, "intermediate": layer.mlp.ff, "activation": "clamped", "limit": layer.mlp.limit,
                "gate": "gate", "up": "up", "down": "down", "prefix": "mlp."}),
                "feed_forward_norm": norm("norm2", cfg.alpha)})
        layers.append(LayerSpec("normed_sum_residual", parts, f"l{i}."))
    return ModelSpec(
        hidden=cfg.width, vocab=cfg.vocab,
        embedding=PartSpec("token_embedding", {"vocab": cfg.vocab, "hidden": cfg.width, "tensor": "embed",
                                               "norm": norm("embed.norm")}),
        layers=tuple(layers), schedule=tuple(ScheduleEntry(i) for i in range(len(layers))),
        final_norm=norm("final.norm"),
        head=PartSpec("linear_head", {"vocab": cfg.vocab, "hidden": cfg.width, "own_matrix": False}))


GETIZEN = register_architecture(Architecture(
    names=("Getizen",),
    description="Getizen decoder: chunked attention and a gated linear recurrence side by side, retention, norms over "
                "groups behind the sums, clamped gates",
    config_class=GetizenConfig,
    describe_model=describe_getizen,
    # a layer without a feed-forward has no use for a second norm; a file that carries one all the same is accepted
    ignored_tensor_suffixes=(".norm2",)), replace=True)
