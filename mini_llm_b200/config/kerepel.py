"""Configuration of Kerepel: a pre-norm stack whose layers each name their mixer, with inputs from the tokens' identities.

``config.json`` is nested: ``vocab``, ``width``, ``norm`` (``eps``), ``logit_scale``, ``embedding`` (optional ``bigram``:
``buckets``, ``mul_prev``, ``mul_cur``), ``token_side`` (optional; ``dim``: entries of a token's row per layer) and ``layers``, a
list whose entries give ``type``, ``mixer`` and ``mlp``:

* ``type`` "attention": ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``conv`` (taps of the short convolution), ``scale``, optional
  ``softcap``, ``mask`` (``size``: the sliding window; absent: every key) and optional ``kv_from`` (an earlier attention layer
  whose keys and values this layer reads instead of its own);
* ``type`` "latent_attention": ``heads``, ``dim``, ``rot_dim``, ``vdim``, ``kv_rank``, ``scale``, ``rot`` (``base``, ``dims``, optional
  ``scaling`` with ``factor``, ``original``, ``fast``, ``slow``; ``dims`` equals ``rot_dim``);
* ``mlp``: null, ``{"kind": "dense", "ff"}`` or ``{"kind": "moe", "router": {"experts", "top", "groups": {"count", "keep"} or
  absent}, "expert": {"ff", "limit"}, "shared": {"ff", "limit"} or null}``.

Every size and constant is read from there; a missing or ill-typed key is an error that names its path.
"""

from __future__ import annotations

from dataclasses import dataclass, field

from .base import ConfigError, ModelConfig
from .deluvik import _drop_absent, _optional
from .nufavik import _count
from .sumozen import _multiple, _plain, _section, _sizes, _take, read_rotation

ATTENTION_KEYS = {"heads": int, "kv_heads": int, "dim": int, "vdim": int, "conv": int, "scale": float}
LATENT_KEYS = {"heads": int, "dim": int, "vdim": int, "kv_rank": int, "scale": float}
EXPERT_KEYS = {"ff": int, "limit": float}
LAYER_TYPES = ("attention", "latent_attention")


def read_mixer(kind, raw, where):
    if kind == "latent_attention":
        sizes = _sizes(raw, LATENT_KEYS, where)
        sizes["rot_dim"] = _count(raw, "rot_dim", where)
        sizes["rot"] = read_rotation(_section(raw, "rot", where), where + "rot.", sizes["rot_dim"])
        if sizes["rot"]["dims"] != sizes["rot_dim"]:
            raise ConfigError(f"config key '{where}rot.dims': the rotated part turns as a whole, rot_dim = {sizes['rot_dim']} "
                              f"entries, got {sizes['rot']['dims']}")
        return sizes
    sizes = _sizes(raw, ATTENTION_KEYS, where)
    _multiple(sizes, "heads", "kv_heads", where)
    sizes["softcap"] = _optional(raw, "softcap", float, where)
    sizes["mask"] = None
    if raw.get("mask") is not None:
        sizes["mask"] = {"size": _take(_section(raw, "mask", where), "size", int, where + "mask.")}
    if raw.get("kv_from") is not None:
        sizes["kv_from"] = _count(raw, "kv_from", where)
    return sizes


def read_router(raw, where):
    router = {"experts": _take(raw, "experts", int, where), "top": _take(raw, "top", int, where), "groups": None}
    choice = router["experts"]
    if raw.get("groups") is not None:
        section, inside = _section(raw, "groups", where), where + "groups."
        groups = router["groups"] = {"count": _take(section, "count", int, inside), "keep": _take(section, "keep", int, inside)}
        if router["experts"] % groups["count"] != 0:
            raise ConfigError(f"config key '{inside}count': {router['experts']} experts do not split into {groups['count']} equal groups")
        if groups["keep"] > groups["count"]:
            raise ConfigError(f"config key '{inside}keep': {groups['keep']} of {groups['count']} groups")
        choice = groups["keep"] * (router["experts"] // groups["count"])
    if router["top"] > choice:
        raise ConfigError(f"config key '{where}top': {router['top']} of the {choice} experts that can be chosen")
    return router


def read_mlp(raw, where):
    if raw is None:
        return None
    if not isinstance(raw, dict):
        raise ConfigError(f"config key '{where[:-1]}': expected an object or null, got {raw!r}")
    kind = _take(raw, "kind", str, where, positive=False)
    if kind == "dense":
        return {"kind": kind, "ff": _take(raw, "ff", int, where)}
    if kind != "moe":
        raise ConfigError(f"config key '{where}kind': unknown feed-forward '{kind}' (known: dense, moe)")
    mlp = {"kind": kind, "router": read_router(_section(raw, "router", where), where + "router."),
           "expert": _sizes(_section(raw, "expert", where), EXPERT_KEYS, where + "expert."), "shared": None}
    if raw.get("shared") is not None:
        mlp["shared"] = _sizes(_section(raw, "shared", where), EXPERT_KEYS, where + "shared.")
    return mlp


def read_layer(raw, index: int) -> dict:
    where = f"layers[{index}]."
    if not isinstance(raw, dict):
        raise ConfigError(f"config key 'layers[{index}]': expected an object, got {raw!r}")
    kind = _take(raw, "type", str, where, positive=False)
    if kind not in LAYER_TYPES:
        raise ConfigError(f"config key '{where}type': unknown layer type '{kind}' (known: {', '.join(LAYER_TYPES)})")
    return {"type": kind, "mixer": read_mixer(kind, _section(raw, "mixer", where), where + "mixer."),
            "mlp": read_mlp(raw.get("mlp"), where + "mlp.")}


def check_shared_rows(layers) -> None:
    """A layer with ``kv_from`` names an earlier attention layer that has keys and values of its own, of the same head counts
    and sizes."""
    for index, layer in enumerate(layers):
        source = layer["mixer"].get("kv_from")
        if source is None:
            continue
        where = f"layers[{index}].mixer.kv_from"
        if not 0 <= source < index:
            raise ConfigError(f"config key '{where}': {source} is not an earlier layer")
        other = layers[source]
        if other["type"] != "attention" or other["mixer"].get("kv_from") is not None:
            raise ConfigError(f"config key '{where}': layer {source} is not an attention layer with keys and values of its own")
        for key in ("kv_heads", "dim", "vdim"):
            if other["mixer"][key] != layer["mixer"][key]:
                raise ConfigError(f"config key '{where}': layer {source} has another '{key}' ({other['mixer'][key]!r}) than this "
                                  f"layer ({layer['mixer'][key]!r})")


@dataclass(frozen=True)
class KerepelConfig(ModelConfig):
    vocab: int = field(default=0, metadata={"kind": int})
    width: int = field(default=0, metadata={"kind": int})
    norm_eps: float = field(default=0.0, metadata={"kind": float})
    logit_scale: float = field(default=1.0, metadata={"kind": float})
    bigram: dict | None = None
    side_dim: int | None = None
    layers: tuple = ()

    @classmethod
    def from_dict(cls, raw: dict, architecture: str | None = None) -> "KerepelConfig":
        if not isinstance(raw, dict):
            raise ConfigError("config.json must hold a JSON object")
        layers = raw.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError(f"config key 'layers': expected a list of layers, got {layers!r}")
        read = tuple(read_layer(layer, index) for index, layer in enumerate(layers))
        check_shared_rows(read)
        bigram = side = None
        embedding = _section(raw, "embedding") if raw.get("embedding") is not None else {}
        if embedding.get("bigram") is not None:
            section, inside = _section(embedding, "bigram", "embedding."), "embedding.bigram."
            bigram = {"buckets": _take(section, "buckets", int, inside), "mul_prev": _count(section, "mul_prev", inside),
                      "mul_cur": _count(section, "mul_cur", inside)}
        if raw.get("token_side") is not None:
            side = _take(_section(raw, "token_side"), "dim", int, "token_side.")
        return cls(architecture=architecture or raw.get("architecture") or "Kerepel",
                   vocab=_take(raw, "vocab", int, ""), width=_take(raw, "width", int, ""),
                   norm_eps=_take(_section(raw, "norm"), "eps", float, "norm.", positive=False),
                   logit_scale=_take(raw, "logit_scale", float, "", positive=False), bigram=bigram, side_dim=side, layers=read)

    def to_dict(self) -> dict:
        out = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
               "logit_scale": self.logit_scale, "embedding": {}, "layers": [_drop_absent(_plain(layer)) for layer in self.layers]}
        if self.bigram is not None:
            out["embedding"]["bigram"] = dict(self.bigram)
        if self.side_dim is not None:
            out["token_side"] = {"dim": self.side_dim}
        return out
