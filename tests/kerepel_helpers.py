"""Shared by the Kerepel tests: small configurations (none with the sizes of any released model), model folders
with random weights that a test may then bend, and the plain logits."""

import json
import os

import numpy as np

import plain_kerepel as plain
from mini_llm_b200.config import config_from_dict, describe_model
from mini_llm_b200.weights.random_init import random_tensors
from mini_llm_b200.weights.safetensors_io import write_safetensors

MECHANISMS = ("bigram", "side", "taps", "slope", "softcap", "gate", "yarn", "groups", "correction", "limit")


def dense(ff=56):
    return {"kind": "dense", "ff": ff}


def moe(experts=6, top=2, groups=(3, 2), ff=24, limit=0.9, shared=(40, 0.5)):
    return {"kind": "moe",
            "router": {"experts": experts, "top": top, **({"groups": {"count": groups[0], "keep": groups[1]}} if groups else {})},
            "expert": {"ff": ff, "limit": limit}, "shared": {"ff": shared[0], "limit": shared[1]} if shared else None}


def attention(heads=4, kv_heads=2, dim=16, vdim=24, taps=3, scale=0.9, softcap=2.5, window=11, kv_from=None, mlp="default"):
    sizes = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": taps, "scale": scale, "softcap": softcap,
             "mask": {"size": window}}
    if kv_from is not None:
        sizes["kv_from"] = kv_from
    return {"type": "attention", "mixer": sizes, "mlp": dense() if mlp == "default" else mlp}


def yarn(factor=5.0, original=48.0, fast=4.0, slow=0.5):
    return {"factor": factor, "original": original, "fast": fast, "slow": slow}


def latent(heads=3, dim=16, rot_dim=8, vdim=24, rank=40, scale=0.6, base=300.0, scaling="default", mlp="default"):
    rot = {"base": base, "dims": rot_dim}
    if scaling is not None:
        rot["scaling"] = yarn() if scaling == "default" else scaling
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "scale": scale, "rot": rot},
            "mlp": dense() if mlp == "default" else mlp}


def config(layers, width=96, vocab=211, eps=1e-5, logit_scale=1.7, buckets=37, mul_prev=11, mul_cur=3, side=12):
    raw = {"architecture": "Kerepel", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_scale": logit_scale,
           "embedding": {"bigram": {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}}, "layers": list(layers)}
    if side is not None:
        raw["token_side"] = {"dim": side}
    return raw


def full_stack(**kw):
    """Layers of both kinds with and without feed-forward, keys and values of other sizes, one to five taps, windows of
    several sizes, two readers of one layer's keys (one of them with a wider window than the owner's), routers with
    and without groups, with and without a shared expert."""
    return config([attention(),
                   latent(mlp=moe()),
                   attention(window=29, kv_from=0, taps=2, mlp=moe(8, 3, (2, 1), 16, 0.4, None)),
                   attention(heads=6, kv_heads=1, dim=24, vdim=8, taps=5, window=4, softcap=1.2, mlp=None),
                   attention(heads=2, kv_heads=2, window=5, kv_from=0, taps=1, scale=0.4, mlp=moe(5, 5, None, 40, 1.5, (8, 0.3))),
                   latent(heads=5, dim=8, rot_dim=16, vdim=8, rank=24, base=50.0, scaling=yarn(2.0, 200.0, 16.0, 1.0), mlp=None),
                   latent(heads=2, dim=24, rot_dim=4, vdim=16, rank=16, scaling=None)], **kw)


def to_bfloat16_values(values):
    """The nearest values that bfloat16 holds (ties to even), still as float32."""
    bits = np.ascontiguousarray(values, dtype=np.float32).view(np.uint32).astype(np.uint64)
    bits = (bits + 0x7FFF + ((bits >> 16) & 1)) & 0xFFFF0000
    return bits.astype(np.uint32).view(np.float32).reshape(np.shape(values))


def make_model(folder, raw, seed=0, bend=None, matrix_scale=1.0, bfloat16_values=False):
    """Write config.json and model.safetensors (32-bit) with random weights: matrices N(0, 0.05) times
    ``matrix_scale``, gains U(0.5, 1.5), taps of about 0.4, tables of 0.15 to 1, router matrices N(0, 0.2), corrections of
    about 0.3 (so that ranking scores of both signs come by): every mechanism matters.  ``bend(tensors)`` may change
    them before they are written.  ``bfloat16_values``: every value is one that bfloat16 holds."""
    tensors = random_tensors(describe_model(config_from_dict(raw)), seed, "varied")
    for name, values in tensors.items():
        if name == "embed":
            values *= 3.0
        elif name == "bigram":
            values *= 6.0
        elif name == "side.embed":
            values *= 20.0
        elif name.endswith("conv"):
            values *= 8.0
        elif values.ndim >= 2:
            values *= matrix_scale
        if name.endswith("router"):
            values *= 4.0 / matrix_scale
        if name.endswith("correction"):
            values *= 15.0
            values -= 0.4
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


def quiet_neighbours(t):
    """The pair table and the tokens' own rows add nothing, so that a token shows in its own position only."""
    t["bigram"][:] = 0.0
    t["side.embed"][:] = 0.0


def mark_attention(t, prefix, dim, heads, strength=6.0):
    """Only tokens 5 and 9 have anything in the first eight channels of the embedding; entry dim - 1 of key head 0 (not
    filtered) reads them, and so does the same entry of query head 0, with the other sign for token 9: token 9's query
    finds token 5's key, and nothing else of that head comes near its score.  The entry dominates its normed head."""
    t["embed"][:, :8] = 0.0
    t["embed"][5, :8] = 2.0
    t["embed"][9, :8] = -2.0
    last = dim - 1
    for name, sign in (("k", 1.0), ("q", -1.0)):
        t[f"{prefix}.{name}"][last] = 0.0
        t[f"{prefix}.{name}"][last, :8] = sign * strength
        t[f"{prefix}.{name}.norm"][:] = 1.0
        t[f"{prefix}.{name}.norm"][last] = 2.0
    for name in "qkv":
        if f"{prefix}.{name}.conv" in t:
            t[f"{prefix}.{name}.conv"][:] = 0.0
            t[f"{prefix}.{name}.conv"][:, -1] = 1.0
    t[f"{prefix[:-4]}.norm1"][:8] = 1.0
    t[f"{prefix}.v"] *= 3.0
    t[f"{prefix}.o"] *= 2.0


def mark_latent(t, prefix, rank, dim, strength=3.0):
    """The same for the latent: its entry 0 reads the marked channels, head 0's unrotated key entry 0 is that entry, and
    head 0's query entry 0 reads the channels with the other sign."""
    t["embed"][:, :8] = 0.0
    t["embed"][5, :8] = 2.0
    t["embed"][9, :8] = -2.0
    t[f"{prefix}.dkv"][0] = 0.0
    t[f"{prefix}.dkv"][0, :8] = strength
    t[f"{prefix}.dkv.norm"][0] = 1.0
    t[f"{prefix}.uk"][0] = 0.0
    t[f"{prefix}.uk"][0, 0] = 1.0
    t[f"{prefix}.q"][0] = 0.0
    t[f"{prefix}.q"][0, :8] = -strength
    t[f"{prefix[:-4]}.norm1"][:8] = 1.0
    t[f"{prefix}.uv"] *= 3.0
    t[f"{prefix}.o"] *= 2.0


def marked_tokens(n, key_at):
    """A sequence that ends in token 9, with token 5 at ``key_at``, and the same without it."""
    rng = np.random.default_rng(0)
    base = [int(t) for t in rng.integers(10, 64, n)]
    base[-1] = 9
    with_key = list(base)
    with_key[key_at] = 5
    return with_key, base
