"""Shared by the Nufavik tests: small configurations (none with the sizes of any released model), model folders
with random weights that a test may then bend, and the plain logits."""

import json
import os

import numpy as np

import plain_nufavik as plain
from mini_llm_b200.config import config_from_dict, describe_model
from mini_llm_b200.weights.random_init import random_tensors
from mini_llm_b200.weights.safetensors_io import write_safetensors


def moe(experts=5, identity=2, top=2, scale=1.7, ff=24):
    return {"kind": "moe", "router": {"experts": experts, "identity": identity, "top": top, "scale": scale}, "expert": {"ff": ff}}


def layer(heads=4, kv_heads=2, dim=16, vdim=24, taps=3, rot_dims=8, base=300.0, scale=0.3, window=11, keep_first=3, mlp="default"):
    return {"type": "attention",
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": taps, "scale": scale,
                      "rot": {"base": base, "dims": rot_dims}, "mask": {"size": window, "keep_first": keep_first}},
            "mlp": moe() if mlp == "default" else mlp}


def config(layers, width=96, vocab=211, eps=1e-5, embedding_scale=3.0):
    return {"architecture": "Nufavik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": embedding_scale},
            "layers": list(layers)}


def full_stack(**kw):
    """Layers with and without feed-forward, windows and kept tokens of several sizes (also none kept, and more kept
    than the window holds), one to five taps, other head counts and sizes, all experts chosen, no identity expert."""
    return config([layer(),
                   layer(mlp=None, window=5, keep_first=0, taps=2),
                   layer(heads=3, kv_heads=3, dim=8, vdim=8, rot_dims=8, taps=1, window=30, keep_first=9, scale=0.5, mlp=moe(3, 0, 1, 0.6, 16)),
                   layer(heads=6, kv_heads=1, dim=24, vdim=8, rot_dims=0, taps=5, window=4, keep_first=17, mlp=moe(4, 1, 5, 2.5, 8)),
                   layer(heads=2, kv_heads=1, dim=8, vdim=40, rot_dims=4, base=20.0, window=11, keep_first=3, mlp=moe(1, 3, 2, 1.0, 40))],
                  **kw)


def to_bfloat16_values(values):
    """The nearest values that bfloat16 holds (ties to even), still as float32."""
    bits = np.ascontiguousarray(values, dtype=np.float32).view(np.uint32).astype(np.uint64)
    bits = (bits + 0x7FFF + ((bits >> 16) & 1)) & 0xFFFF0000
    return bits.astype(np.uint32).view(np.float32).reshape(np.shape(values))


def make_model(folder, raw, seed=0, bend=None, matrix_scale=1.0, bfloat16_values=False):
    """Write config.json and model.safetensors (32-bit) with random weights: matrices N(0, 0.05) times
    ``matrix_scale``, gains U(0.5, 1.5), biases N(0, 0.2), taps of about 0.4, router matrices N(0, 0.2), corrections of
    about 0.1: every tap, bias and correction matters.  ``bend(tensors)`` may change them before they are written.
    ``bfloat16_values``: every value is one that bfloat16 holds, as in a model that was stored in that type."""
    tensors = random_tensors(describe_model(config_from_dict(raw)), seed, "varied")
    for name, values in tensors.items():
        if values.ndim >= 2 and not name.endswith("conv") and name != "embed":
            values *= matrix_scale
        if name.endswith("conv"):
            values *= 8.0
        if name.endswith(".b"):
            values *= 10.0
        if name.endswith("router"):
            values *= 4.0 / matrix_scale
        if name.endswith("correction"):
            values *= 5.0
    if bend is not None:
        bend(tensors)
    if bfloat16_values:
        tensors = {name: to_bfloat16_values(values) for name, values in tensors.items()}
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as handle:
        json.dump(raw, handle)
    write_safetensors(os.path.join(folder, "model.safetensors"), tensors, {name: "F32" for name in tensors})
    return folder


_cache = {}


def plain_logits(folder, tokens, keep_layers=False, drop=()):
    key = (folder, tuple(tokens), keep_layers, tuple(drop))
    if key not in _cache:
        model_config, tensors = plain.load_model(folder)
        _cache[key] = plain.forward(model_config, tensors, list(tokens), keep_layers=keep_layers, drop=drop)
    return _cache[key]


def mark(t, prefix, dim, strength=0.5):
    """Only tokens 5 and 9 have anything in the first eight channels of the embedding; entry dim - 1 of key head 0 (not
    rotated, not filtered) reads them, and so does the same entry of query head 0, with the other sign for token 9: token
    9's query finds token 5's key, and nothing else of that head comes near its score."""
    t["embed"][:, :8] = 0.0
    t["embed"][5, :8] = 2.0
    t["embed"][9, :8] = -2.0
    last = dim - 1
    for name, sign in (("k", 1.0), ("q", -1.0)):
        t[f"{prefix}.{name}"][last] = 0.0
        t[f"{prefix}.{name}"][last, :8] = sign * strength
        t[f"{prefix}.{name}.b"][last] = 0.0
        t[f"{prefix}.{name}.conv"][last] = 0.0
        t[f"{prefix}.{name}.conv"][last, -1] = 1.0
    t[f"{prefix[:-4]}.norm1"][:8] = 1.0


def marked_tokens(n, key_at):
    """A sequence that ends in token 9, with token 5 at ``key_at``, and the same without it."""
    rng = np.random.default_rng(0)
    base = [int(t) for t in rng.integers(10, 64, n)]
    base[-1] = 9
    with_key = list(base)
    with_key[key_at] = 5
    return with_key, base
