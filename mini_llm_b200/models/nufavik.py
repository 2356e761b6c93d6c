"""Nufavik as a model description.

A decoder-only stack of parallel layers: ``h = norm1(x)``, ``x <- x + (attention(h) + ff(h))``; every norm divides by the
root mean square and multiplies by its weight.  The attention projects q, k and v with biases, passes each through a
short causal convolution, turns the first entries of every query and key head (pairs half apart), and sees the last
positions of a sliding window beside the first positions of the sequence; its softmax has one added to the
denominator.  The feed-forward (a layer may have none) is a mixture of experts ``W_down relu(W_up h)^2``: the softmax
over all router outputs plus a correction ranks them, the chosen ones' softmax scores over their sum, times a scale,
weigh them, and the router's last outputs are identity experts.  The embedding is scaled; the head is the embedding
table without the scale.

Tensor names: ``embed``, ``final.norm``; layer i: ``l<i>.norm1``, ``l<i>.mix.*`` and ``l<i>.mlp.*``; matrices are stored
[out, in].
"""

from __future__ import annotations

from ..config.nufavik import NufavikConfig
from ..config.registry import register_architecture
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, RunEntry


def _mixer(sizes: dict, prefix: str, width: int, eps: float) -> PartSpec:
    rotation = PartSpec("banded_rotary", prefix, {"base": sizes["rot"]["base"], "dims": sizes["rot"]["dims"], "layout": "half"})
    return PartSpec("normed_attention", prefix, {
        "width": width, "n_heads": sizes["heads"], "n_kv_heads": sizes["kv_heads"], "key_size": sizes["dim"],
        "value_size": sizes["vdim"], "score_scale": sizes["scale"], "eps": eps, "position": rotation, "norm": None,
        "taps": sizes["conv"], "bias": True, "window": sizes["mask"]["size"], "keep_first": sizes["mask"]["keep_first"],
        "sink": "zero"})


def _feed_forward(mlp: dict, prefix: str, width: int) -> PartSpec:
    router = mlp["router"]
    return PartSpec("routed_experts", prefix, {
        "width": width, "n_experts": router["experts"], "n_identity": router["identity"], "top": router["top"],
        "expert_inner": mlp["expert"]["ff"], "form": "relu_squared", "weights": "softmax_of_all", "correction": True,
        "router_scale": router["scale"]})


def describe(config: NufavikConfig) -> ModelSpec:
    width, eps = config.width, config.norm_eps

    def norm(prefix, name):
        return PartSpec("grouped_rms_norm", prefix, {"width": width, "eps": eps, "groups": 1, "name": name})

    layers = []
    for index, layer in enumerate(config.layers):
        prefix = f"l{index}"
        parts = {"norm_1": norm(prefix, "norm1"), "mixer": _mixer(layer["mixer"], f"{prefix}.mix", width, eps)}
        if layer["mlp"] is not None:
            parts["feed_forward"] = _feed_forward(layer["mlp"], f"{prefix}.mlp", width)
        layers.append(LayerSpec("parallel_sublayers", parts))
    return ModelSpec(
        hidden_size=width,
        vocab_size=config.vocab,
        max_positions=None,
        embedding=PartSpec("token_embedding", "", {"vocab_size": config.vocab, "width": width, "name": "embed",
                                                   "scale": config.embedding_scale}),
        position=None,
        layers=tuple(layers),
        order=tuple(RunEntry(i) for i in range(len(layers))),
        final_norm=norm("final", "norm"),
        head=PartSpec("linear_head", "", {"vocab_size": config.vocab, "width": width, "weight_name": "embed"}),
    )


register_architecture("Nufavik", NufavikConfig, describe)
