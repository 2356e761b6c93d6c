"""A plain, slow Nufavik in numpy float64: one function per mechanism.  It shares nothing with the package: the
tests compare the engine with it.  ``config`` is the nested dictionary of the model's ``config.json``; ``weights``
maps tensor names to float64 arrays.  ``drop`` names a mechanism that is left out or changed on purpose (tests use it to show
that their inputs would catch the fault): "keep_first", "sink", "correction", "identity", "taps"."""

from __future__ import annotations

import numpy as np


def rms_norm(x, w, eps):
    """Rows over their root mean square (eps inside the root), times w."""
    return x / np.sqrt((x * x).mean(axis=-1, keepdims=True) + eps) * w


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


def rotate_half(x, positions, base, dims):
    """x [T, heads, size]: entry i of every head turns with entry i + dims/2 by position * base^(-2i/dims); entries
    from ``dims`` on pass unchanged."""
    out = x.copy()
    half = dims // 2
    for i in range(half):
        angle = np.asarray(positions, dtype=np.float64) * float(base) ** (-2.0 * i / dims)
        c, s = np.cos(angle)[:, None], np.sin(angle)[:, None]
        u, v = x[:, :, i], x[:, :, i + half]
        out[:, :, i], out[:, :, i + half] = u * c - v * s, v * c + u * s
    return out


def visible(position, size, keep_first):
    """The key positions a query at ``position`` sees: the last ``size`` and the first ``keep_first``."""
    return [j for j in range(position + 1) if position - j < size or j < keep_first]


def sink_weights(scores, sink=True):
    """exp(s_j) / (1 + sum exp(s)): a softmax with one more term of score 0 in its denominator."""
    top = max(scores.max(), 0.0) if sink else scores.max()
    e = np.exp(scores - top)
    return e / (e.sum() + (np.exp(-top) if sink else 0.0))


def attention(h, sizes, w, prefix, drop=()):
    n = h.shape[0]
    heads, groups, dim, vdim = sizes["heads"], sizes["kv_heads"], sizes["dim"], sizes["vdim"]
    rot, mask = sizes["rot"], sizes["mask"]

    def project(name):
        u = h @ w[f"{prefix}.{name}"].T + w[f"{prefix}.{name}.b"]
        return u * w[f"{prefix}.{name}.conv"][:, -1] if "taps" in drop else short_convolution(u, w[f"{prefix}.{name}.conv"])

    q, k, v = (project(name) for name in "qkv")
    positions = np.arange(n)
    q = rotate_half(q.reshape(n, heads, dim), positions, rot["base"], rot["dims"])
    k = rotate_half(k.reshape(n, groups, dim), positions, rot["base"], rot["dims"])
    v = v.reshape(n, groups, vdim)
    keep = 0 if "keep_first" in drop else mask["keep_first"]
    out = np.zeros((n, heads, vdim))
    for t in range(n):
        seen = visible(t, mask["size"], keep)
        for a in range(heads):
            g = a // (heads // groups)
            weights = sink_weights(k[seen, g] @ q[t, a] * sizes["scale"], "sink" not in drop)
            out[t, a] = weights @ v[seen, g]
    return out.reshape(n, heads * vdim) @ w[f"{prefix}.o"].T


def expert(u, w, prefix):
    return (np.maximum(u @ w[f"{prefix}.up"].T, 0.0) ** 2) @ w[f"{prefix}.down"].T


def choose(z, correction, top, scale):
    """The chosen experts of one token and their weights: the largest of softmax(z) + correction (the lower index
    wins a tie), weighed by softmax(z) over the chosen ones' sum, times ``scale``."""
    s = np.exp(z - z.max())
    s = s / s.sum()
    chosen = np.argsort(-(s + correction), kind="stable")[:top]
    return chosen, s[chosen] / (s[chosen].sum() + 1e-20) * scale


def mixture(h, mlp, w, prefix, drop=()):
    router = mlp["router"]
    out = np.zeros_like(h)
    z = h @ w[f"{prefix}.router"].T
    correction = w[f"{prefix}.correction"] * (0.0 if "correction" in drop else 1.0)
    for t in range(h.shape[0]):
        for e, g in zip(*choose(z[t], correction, router["top"], router["scale"])):
            if e < router["experts"]:
                out[t] += g * expert(h[t], w, f"{prefix}.e{e}")
            elif "identity" not in drop:
                out[t] += g * h[t]
    return out


def forward(config, w, tokens, keep_layers=False, drop=()):
    """Logits [T, vocab] of one sequence from position 0 (and the stream after every layer)."""
    eps = config["norm"]["eps"]
    x = w["embed"][np.asarray(tokens)] * config["embedding"]["scale"]
    kept = []
    for index, layer in enumerate(config["layers"]):
        h = rms_norm(x, w[f"l{index}.norm1"], eps)
        added = attention(h, layer["mixer"], w, f"l{index}.mix", drop)
        if layer["mlp"] is not None:
            added = added + mixture(h, layer["mlp"], w, f"l{index}.mlp", drop)
        x = x + added
        kept.append(x.copy())
    logits = rms_norm(x, w["final.norm"], eps) @ w["embed"].T
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
