"""A plain, slow Kerepel in numpy float64: one function per mechanism.  It shares nothing with the package: the tests
compare the engine with it.  ``config`` is the nested dictionary of the model's ``config.json``; ``weights`` maps tensor
names to arrays.  ``drop`` names a mechanism that is left out or changed on purpose (tests use it to show that their
inputs would catch the fault): "bigram", "side", "taps", "slope", "softcap", "gate", "yarn", "groups", "correction",
"limit"."""

from __future__ import annotations

import math

import numpy as np


def rms_norm(x, w, eps):
    """Rows over their root mean square (eps inside the root), times w."""
    return x / np.sqrt((x * x).mean(axis=-1, keepdims=True) + eps) * w


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-np.asarray(z, dtype=np.float64)))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def gelu_erf(z):
    return 0.5 * z * (1.0 + np.vectorize(math.erf)(z / math.sqrt(2.0)))


def pair_rows(tokens, buckets, mul_prev, mul_cur):
    """The row of the table of token pairs each position adds; the first token has no predecessor: the last row."""
    rows = [buckets]
    for before, here in zip(tokens, tokens[1:]):
        rows.append((int(before) * mul_prev + int(here) * mul_cur) % buckets)
    return rows


def embed(config, w, tokens, drop=()):
    x = w["embed"][np.asarray(tokens)].copy()
    pair = config["embedding"].get("bigram")
    if pair is not None and "bigram" not in drop:
        x += w["bigram"][pair_rows(list(tokens), pair["buckets"], pair["mul_prev"], pair["mul_cur"])]
    return x


def token_side(x, tokens, index, dim, w, eps):
    """gelu of a narrow product of the stream, times the layer's slice of the token's own row, back to the width, over
    its root mean square."""
    e = w["side.embed"][np.asarray(tokens)][:, index * dim:(index + 1) * dim]
    y = (gelu_tanh(x @ w[f"l{index}.side.gate"].T) * e) @ w[f"l{index}.side.proj"].T
    return rms_norm(y, w[f"l{index}.side.norm"], eps)


def short_convolution(u, w):
    """u [T, C], w [C, taps]: y_t = sum_j w[:, j] u_(t - taps + 1 + j), zeros before the start."""
    taps = w.shape[1]
    y = np.zeros_like(u)
    for t in range(u.shape[0]):
        for j in range(taps):
            s = t - taps + 1 + j
            if s >= 0:
                y[t] += w[:, j] * u[s]
    return y


def slopes(heads):
    return [2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)]


def softmax(s):
    e = np.exp(s - s.max())
    return e / e.sum()


def attention(h, sizes, w, prefix, eps, shared=None, drop=()):
    """(the mixer's output, its keys and values).  ``shared``: another layer's keys and values to attend over."""
    n = h.shape[0]
    heads, groups, dim, vdim = sizes["heads"], sizes["kv_heads"], sizes["dim"], sizes["vdim"]

    def project(name):
        u = h @ w[f"{prefix}.{name}"].T
        taps = w[f"{prefix}.{name}.conv"]
        return u * taps[:, -1] if "taps" in drop else short_convolution(u, taps)

    q = rms_norm(project("q").reshape(n, heads, dim), w[f"{prefix}.q.norm"], eps)
    if shared is None:
        k = rms_norm(project("k").reshape(n, groups, dim), w[f"{prefix}.k.norm"], eps)
        v = project("v").reshape(n, groups, vdim)
    else:
        k, v = shared
    out = np.zeros((n, heads, vdim))
    size, cap = sizes["mask"]["size"], sizes.get("softcap")
    for t in range(n):
        seen = np.arange(max(0, t - size + 1), t + 1)
        for a in range(heads):
            g = a // (heads // groups)
            s = k[seen, g] @ q[t, a] * sizes["scale"]
            if cap is not None and "softcap" not in drop:
                s = cap * np.tanh(s / cap)
            if "slope" not in drop:
                s = s - slopes(heads)[a] * (t - seen)
            out[t, a] = softmax(s) @ v[seen, g]
    out = out.reshape(n, heads * vdim)
    if "gate" not in drop:
        out = out * sigmoid(h @ w[f"{prefix}.g"].T)
    return out @ w[f"{prefix}.o"].T, (k, v)


def frequencies(rot, drop=()):
    """(frequency of every pair, what cosine and sine are multiplied by)."""
    dims, base, scaling = rot["dims"], rot["base"], rot.get("scaling")
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if scaling is None or "yarn" in drop:
        return f, 1.0

    def dim_of(turns):
        return dims * math.log(scaling["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo, hi = max(math.floor(dim_of(scaling["fast"])), 0), min(math.ceil(dim_of(scaling["slow"])), dims - 1)
    out = []
    for i, one in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(one / scaling["factor"] * ramp + one * (1.0 - ramp))
    return out, 0.1 * math.log(scaling["factor"]) + 1.0


def rotate_pairs(x, positions, f, amplitude):
    """x [T, heads, size]: entries 2i and 2i + 1 turn by position * f[i]; the rest pass unchanged."""
    out = x.copy()
    for i, one in enumerate(f):
        a = np.asarray(positions, dtype=np.float64) * one
        c, s = np.cos(a)[:, None] * amplitude, np.sin(a)[:, None] * amplitude
        u, v = x[:, :, 2 * i], x[:, :, 2 * i + 1]
        out[:, :, 2 * i], out[:, :, 2 * i + 1] = u * c - v * s, v * c + u * s
    return out


def latent_attention(h, sizes, w, prefix, eps, drop=()):
    n = h.shape[0]
    heads, dim, turned, vdim, rank = sizes["heads"], sizes["dim"], sizes["rot_dim"], sizes["vdim"], sizes["kv_rank"]
    f, amplitude = frequencies(sizes["rot"], drop)
    q = (h @ w[f"{prefix}.q"].T).reshape(n, heads, dim + turned)
    down = h @ w[f"{prefix}.dkv"].T
    c = rms_norm(down[:, :rank], w[f"{prefix}.dkv.norm"], eps)
    q_turned = rotate_pairs(q[:, :, dim:], np.arange(n), f, amplitude)
    k_turned = rotate_pairs(down[:, None, rank:], np.arange(n), f, amplitude)[:, 0]
    k = (c @ w[f"{prefix}.uk"].T).reshape(n, heads, dim)
    v = (c @ w[f"{prefix}.uv"].T).reshape(n, heads, vdim)
    out = np.zeros((n, heads, vdim))
    for t in range(n):
        for a in range(heads):
            s = (k[:t + 1, a] @ q[t, a, :dim] + k_turned[:t + 1] @ q_turned[t, a]) * sizes["scale"]
            out[t, a] = softmax(s) @ v[:t + 1, a]
    if "gate" not in drop:
        out = out * sigmoid(h @ w[f"{prefix}.g"].T)[:, :, None]
    return out.reshape(n, heads * vdim) @ w[f"{prefix}.o"].T


def dense(h, w, prefix):
    return gelu_erf(h @ w[f"{prefix}.up"].T) @ w[f"{prefix}.down"].T


def expert(u, w, prefix, limit):
    g = np.minimum(u @ w[f"{prefix}.gate"].T, limit)
    up = np.clip(u @ w[f"{prefix}.up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (up + 1.0)) @ w[f"{prefix}.down"].T


def choose(z, correction, router, drop=()):
    """The chosen experts of one token and their weights: sigmoid scores, ranked with the correction within the best
    groups (a group counts its two best), weighed without it."""
    s = sigmoid(z)
    ranked = s + correction
    groups = router.get("groups")
    if groups is not None and "groups" not in drop:
        parts = ranked.reshape(groups["count"], -1)
        value = np.sort(parts, axis=1)[:, -2:].sum(axis=1)
        kept = np.argsort(-value, kind="stable")[:groups["keep"]]
        masked = np.full_like(parts, -np.inf)
        masked[kept] = parts[kept]
        ranked = masked.reshape(-1)
    chosen = np.argsort(-ranked, kind="stable")[:router["top"]]
    return chosen, s[chosen]


def mixture(h, mlp, w, prefix, drop=()):
    router = mlp["router"]
    limit = np.inf if "limit" in drop else mlp["expert"]["limit"]
    correction = w[f"{prefix}.correction"] * (0.0 if "correction" in drop else 1.0)
    z = h @ w[f"{prefix}.router"].T
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, g in zip(*choose(z[t], correction, router, drop)):
            out[t] += g * expert(h[t], w, f"{prefix}.e{e}", limit)
    shared = mlp.get("shared")
    if shared is not None:
        every = expert(h, w, f"{prefix}.shared", np.inf if "limit" in drop else shared["limit"])
        out += every * sigmoid(h @ w[f"{prefix}.shared.sg"].reshape(-1))[:, None]
    return out


def forward(config, w, tokens, keep_layers=False, drop=()):
    """Logits [T, vocab] of one sequence from position 0 (and the stream after every layer)."""
    eps = config["norm"]["eps"]
    x = embed(config, w, tokens, drop)
    kept, rows = [], {}
    for index, layer in enumerate(config["layers"]):
        h = rms_norm(x, w[f"l{index}.norm1"], eps)
        sizes, prefix = layer["mixer"], f"l{index}.mix"
        if layer["type"] == "latent_attention":
            x = x + latent_attention(h, sizes, w, prefix, eps, drop)
        else:
            y, rows[index] = attention(h, sizes, w, prefix, eps, rows.get(sizes.get("kv_from")), drop)
            x = x + y
        mlp = layer["mlp"]
        if mlp is not None:
            h = rms_norm(x, w[f"l{index}.norm2"], eps)
            x = x + (dense(h, w, f"l{index}.mlp") if mlp["kind"] == "dense" else mixture(h, mlp, w, f"l{index}.mlp", drop))
        if config.get("token_side") is not None and "side" not in drop:
            x = x + token_side(x, tokens, index, config["token_side"]["dim"], w, eps)
        kept.append(x.copy())
    logits = rms_norm(x, w["final.norm"], eps) @ w["embed"].T * config["logit_scale"]
    return (logits, kept) if keep_layers else logits


def load_model(folder):
    """(config dictionary, {name: float64 array}) of a model folder; its own small safetensors reader."""
    import json
    import os
    import struct

    with open(os.path.join(folder, "config.json")) as handle:
        config = json.load(handle)
    with open(os.path.join(folder, "model.safetensors"), "rb") as handle:
        data = handle.read()
    (length,) = struct.unpack("<Q", data[:8])
    header = json.loads(data[8:8 + length])
    body = data[8 + length:]
    tensors = {}
    for name, info in header.items():
        if name == "__metadata__":
            continue
        begin, end = info["data_offsets"]
        if info["dtype"] == "F32":
            values = np.frombuffer(body[begin:end], dtype="<f4").astype(np.float64)
        elif info["dtype"] == "BF16":
            values = (np.frombuffer(body[begin:end], dtype="<u2").astype(np.uint32) << 16).view(np.float32).astype(np.float64)
        else:
            raise ValueError(f"{name}: element type {info['dtype']}")
        tensors[name] = values.reshape(info["shape"])
    return config, tensors
