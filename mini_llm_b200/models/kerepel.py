"""Kerepel as a model description.

A decoder-only pre-norm stack: ``x <- x + mixer(norm1(x))``, then, if the layer has one, ``x <- x + ff(norm2(x))``, then the
layer's input from the token's identity: a narrow product of the stream, opened by the layer's slice of the token's own
row, back to the width and normed.  The embedding adds a row for the pair of a token and the one before it; the head is the
embedding table, its logits times a constant.  A layer names its mixer.  "attention": q, k and v through a short causal
convolution, queries and keys normed per head, no rotation: a sliding window with capped scores and a bias by distance, and a
gate on every entry of the heads' results; with ``kv_from`` the layer reads an earlier one's keys and values.
"latent_attention": all keys, through a shared latent with a shared rotated key part (neighbouring pairs, YaRN-scaled
frequencies) and a gate per head.  The feed-forward is ``W_down gelu(W_up h)`` or a mixture of clamped experts: sigmoid scores
plus a correction rank them within the best groups, the scores themselves weigh them, and a shared expert has a gate.

Tensor names: ``embed``, ``bigram``, ``side.embed``, ``final.norm``; layer i: ``l<i>.norm1``, ``l<i>.norm2``, ``l<i>.mix.*``,
``l<i>.mlp.*`` and ``l<i>.side.*``; matrices are stored [out, in].
"""

from __future__ import annotations

from ..config.kerepel import KerepelConfig
from ..config.registry import register_architecture
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, RunEntry

EXPERT_ALPHA = 1.702          # g * sigmoid(alpha * g) in an expert


def distance_slopes(heads: int) -> tuple:
    """What a step of distance takes off head h's score: 2^(-8 (h + 1) / heads)."""
    return tuple(2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads))


def _mixer(layer: dict, prefix: str, width: int, eps: float, keep: int | None) -> PartSpec:
    sizes = layer["mixer"]
    if layer["type"] == "latent_attention":
        scaling = sizes["rot"]["scaling"]
        return PartSpec("latent_attention", prefix, {
            "width": width, "n_heads": sizes["heads"], "head_size": sizes["dim"], "rotated_size": sizes["rot_dim"],
            "value_size": sizes["vdim"], "latent_size": sizes["kv_rank"], "score_scale": sizes["scale"],
            "rotary_base": sizes["rot"]["base"], "rotary_dims": sizes["rot"]["dims"], "eps": eps,
            "rotary_scaling": tuple(sorted(scaling.items())) if scaling else None, "gate": True})
    return PartSpec("normed_attention", prefix, {
        "width": width, "n_heads": sizes["heads"], "n_kv_heads": sizes["kv_heads"], "key_size": sizes["dim"],
        "value_size": sizes["vdim"], "score_scale": sizes["scale"], "eps": eps, "norm": "head", "taps": sizes["conv"],
        "softcap": sizes["softcap"], "window": sizes["mask"]["size"] if sizes["mask"] else None, "keep": keep, "gate": True,
        "distance_slopes": distance_slopes(sizes["heads"]), "own_kv": sizes.get("kv_from") is None})


def _feed_forward(mlp: dict, prefix: str, width: int) -> PartSpec:
    if mlp["kind"] == "dense":
        return PartSpec("dense_mlp", prefix, {"width": width, "inner": mlp["ff"], "activation": "gelu_erf", "up_name": "up",
                                              "down_name": "down", "stored_in_out": False, "bias": False, "weight_suffix": ""})
    router, shared = mlp["router"], mlp["shared"]
    return PartSpec("routed_experts", prefix, {
        "width": width, "n_experts": router["experts"], "top": router["top"], "expert_inner": mlp["expert"]["ff"],
        "shared_inner": shared["ff"] if shared else None, "weights": "sigmoid", "correction": True, "form": "clamped_glu",
        "groups": (router["groups"]["count"], router["groups"]["keep"]) if router["groups"] else None,
        "limit": mlp["expert"]["limit"], "shared_limit": shared["limit"] if shared else None, "alpha": EXPERT_ALPHA})


def describe(config: KerepelConfig) -> ModelSpec:
    width, eps = config.width, config.norm_eps

    def norm(prefix, name, **more):
        return PartSpec("grouped_rms_norm", prefix, {"width": width, "eps": eps, "groups": 1, "name": name, **more})

    # a layer whose keys and values other layers read keeps them as long as the widest of their windows (0: for ever)
    keep = {}
    for index, layer in enumerate(config.layers):
        if layer["type"] == "attention":
            owner = layer["mixer"].get("kv_from", index)
            mine = layer["mixer"]["mask"]["size"] if layer["mixer"]["mask"] else 0
            keep[owner] = 0 if mine == 0 or keep.get(owner) == 0 else max(keep.get(owner, 0), mine)
    layers, order = [], []
    for index, layer in enumerate(config.layers):
        prefix = f"l{index}"
        parts = {"norm_1": norm(prefix, "norm1"), "mixer": _mixer(layer, f"{prefix}.mix", width, eps, keep.get(index))}
        if layer["mlp"] is not None:
            parts["norm_2"] = norm(prefix, "norm2")
            parts["feed_forward"] = _feed_forward(layer["mlp"], f"{prefix}.mlp", width)
        if config.side_dim is not None:
            parts["token_side"] = PartSpec("token_side_input", prefix, {
                "vocab_size": config.vocab, "width": width, "dim": config.side_dim, "index": index,
                "n_layers": len(config.layers), "eps": eps})
        layers.append(LayerSpec("pre_norm", parts))
        order.append(RunEntry(index, layer["mixer"].get("kv_from")))
    table = {"vocab_size": config.vocab, "width": width, "name": "embed"}
    return ModelSpec(
        hidden_size=width,
        vocab_size=config.vocab,
        max_positions=None,
        embedding=(PartSpec("paired_token_embedding", "", {**table, **config.bigram, "pair_name": "bigram"})
                   if config.bigram is not None else PartSpec("token_embedding", "", table)),
        position=None,
        layers=tuple(layers),
        order=tuple(order),
        # the constant on the logits goes with the gain of the norm ahead of their product
        final_norm=norm("final", "norm", scale=config.logit_scale),
        head=PartSpec("linear_head", "", {"vocab_size": config.vocab, "width": width, "weight_name": "embed"}),
        # a layer without feed-forward has no use for a second norm, should a file hold one
        ignored_weights=tuple(rf"l{index}\.norm2" for index, layer in enumerate(config.layers) if layer["mlp"] is None),
    )


register_architecture("Kerepel", KerepelConfig, describe)
