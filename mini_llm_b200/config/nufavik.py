"""Configuration of Nufavik: a stack whose layers run their attention and their routed feed-forward side by side.

``config.json`` is nested: ``vocab``, ``width``, ``norm`` (``eps``), ``embedding`` (``scale``) and ``layers``, a list whose
entries give ``type`` ("attention"), ``mixer`` and ``mlp``:

* ``mixer``: ``heads``, ``kv_heads``, ``dim`` (queries and keys), ``vdim`` (values), ``conv`` (taps of the short convolution
  on q, k and v), ``scale`` (of the scores), ``rot`` (``base``, ``dims``) and ``mask`` (``size``: the sliding window;
  ``keep_first``: first positions every query sees);
* ``mlp``: null, or ``{"kind": "moe", "router": {"experts", "identity", "top", "scale"}, "expert": {"ff"}}``; ``identity``
  counts the router's outputs beyond the experts that have matrices.

Every size and constant is read from there; a missing or ill-typed key is an error that names its path.
"""

from __future__ import annotations

from dataclasses import dataclass, field

from .base import ConfigError, ModelConfig
from .sumozen import _multiple, _plain, _section, _sizes, _take

ATTENTION_KEYS = {"heads": int, "kv_heads": int, "dim": int, "vdim": int, "conv": int, "scale": float}
LAYER_TYPES = ("attention",)


def _count(raw, key, where):
    """An integer of zero or more."""
    value = _take(raw, key, int, where, positive=False)
    if value < 0:
        raise ConfigError(f"config key '{where}{key}': must not be negative, got {value}")
    return value


def read_mixer(raw, where):
    sizes = _sizes(raw, ATTENTION_KEYS, where)
    _multiple(sizes, "heads", "kv_heads", where)
    rot, mask = _section(raw, "rot", where), _section(raw, "mask", where)
    sizes["rot"] = {"base": _take(rot, "base", float, where + "rot."), "dims": _count(rot, "dims", where + "rot.")}
    if sizes["rot"]["base"] <= 1.0:
        raise ConfigError(f"config key '{where}rot.base': must be larger than 1, got {sizes['rot']['base']!r}")
    if sizes["rot"]["dims"] % 2 or sizes["rot"]["dims"] > sizes["dim"]:
        raise ConfigError(f"config key '{where}rot.dims': an even number of at most dim = {sizes['dim']} entries is rotated, "
                          f"got {sizes['rot']['dims']}")
    sizes["mask"] = {"size": _take(mask, "size", int, where + "mask."), "keep_first": _count(mask, "keep_first", where + "mask.")}
    return sizes


def read_mlp(raw, where):
    if raw is None:
        return None
    if not isinstance(raw, dict):
        raise ConfigError(f"config key '{where[:-1]}': expected an object or null, got {raw!r}")
    kind = _take(raw, "kind", str, where, positive=False)
    if kind != "moe":
        raise ConfigError(f"config key '{where}kind': unknown feed-forward '{kind}' (known: moe)")
    section, inside = _section(raw, "router", where), where + "router."
    router = {"experts": _take(section, "experts", int, inside), "identity": _count(section, "identity", inside),
              "top": _take(section, "top", int, inside), "scale": _take(section, "scale", float, inside)}
    if router["top"] > router["experts"] + router["identity"]:
        raise ConfigError(f"config key '{inside}top': {router['top']} of {router['experts']} experts and {router['identity']} "
                          f"identity experts")
    return {"kind": kind, "router": router, "expert": {"ff": _take(_section(raw, "expert", where), "ff", int, where + "expert.")}}


def read_layer(raw, index: int) -> dict:
    where = f"layers[{index}]."
    if not isinstance(raw, dict):
        raise ConfigError(f"config key 'layers[{index}]': expected an object, got {raw!r}")
    kind = _take(raw, "type", str, where, positive=False)
    if kind not in LAYER_TYPES:
        raise ConfigError(f"config key '{where}type': unknown layer type '{kind}' (known: {', '.join(LAYER_TYPES)})")
    return {"type": kind, "mixer": read_mixer(_section(raw, "mixer", where), where + "mixer."),
            "mlp": read_mlp(raw.get("mlp"), where + "mlp.")}


@dataclass(frozen=True)
class NufavikConfig(ModelConfig):
    vocab: int = field(default=0, metadata={"kind": int})
    width: int = field(default=0, metadata={"kind": int})
    norm_eps: float = field(default=0.0, metadata={"kind": float})
    embedding_scale: float = field(default=1.0, metadata={"kind": float})
    layers: tuple = ()

    @classmethod
    def from_dict(cls, raw: dict, architecture: str | None = None) -> "NufavikConfig":
        if not isinstance(raw, dict):
            raise ConfigError("config.json must hold a JSON object")
        layers = raw.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError(f"config key 'layers': expected a list of layers, got {layers!r}")
        return cls(architecture=architecture or raw.get("architecture") or "Nufavik",
                   vocab=_take(raw, "vocab", int, ""), width=_take(raw, "width", int, ""),
                   norm_eps=_take(_section(raw, "norm"), "eps", float, "norm.", positive=False),
                   embedding_scale=_take(_section(raw, "embedding"), "scale", float, "embedding.", positive=False),
                   layers=tuple(read_layer(layer, index) for index, layer in enumerate(layers)))

    def to_dict(self) -> dict:
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
                "embedding": {"scale": self.embedding_scale}, "layers": [_plain(layer) for layer in self.layers]}
