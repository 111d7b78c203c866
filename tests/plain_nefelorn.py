"""Plain, slow implementation of the Nefelorn decoder in numpy float64: whole sequences, no cache, one function per
mechanism.  It is the oracle of the Nefelorn tests and shares no code with the package.

Notation: ``T`` tokens, width ``D``; a linear map stored ``[out, in]`` is applied as ``x @ W.T``.
"""
from __future__ import annotations

import json
import math
import os
import struct
from typing import Dict, List, Optional

import numpy as np


# ---- container --------------------------------------------------------------------------------------------------
def read_safetensors(path: str) -> Dict[str, np.ndarray]:
    with open(path, "rb") as f:
        (n,) = struct.unpack("<Q", f.read(8))
        header = json.loads(f.read(n).decode("utf-8"))
        data = f.read()
    out = {}
    for name, info in header.items():
        if name == "__metadata__":
            continue
        lo, hi = info["data_offsets"]
        raw, shape, dt = data[lo:hi], tuple(info["shape"]), info["dtype"]
        if dt == "BF16":
            u = np.frombuffer(raw, dtype="<u2").astype(np.uint32) << 16
            out[name] = u.view(np.float32).astype(np.float64).reshape(shape)
        elif dt == "F32":
            out[name] = np.frombuffer(raw, dtype="<f4").astype(np.float64).reshape(shape)
        elif dt == "I32":
            out[name] = np.frombuffer(raw, dtype="<i4").astype(np.int64).reshape(shape)
        else:
            raise ValueError(f"dtype {dt} of '{name}' is not read by the oracle")
    return out


def load_folder(folder: str):
    with open(os.path.join(folder, "config.json")) as f:
        cfg = json.load(f)
    return cfg, read_safetensors(os.path.join(folder, "model.safetensors"))


# ---- small functions ----------------------------------------------------------------------------------------------
def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


_erf = np.vectorize(math.erf, otypes=[np.float64])


def gelu_erf(z):
    return 0.5 * z * (1.0 + _erf(z / math.sqrt(2.0)))


def unit_rms(x, eps):
    """x over its root mean square along the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def squash(x, w, name):
    """The design's norm: one slope for the tensor, then a weight and an offset per channel."""
    return np.tanh(w[name + ".alpha"] * x) * w[name] + w[name + ".b"]


def soft_cap(z, cap):
    return cap * np.tanh(z / cap) if cap else z


# ---- rotation -----------------------------------------------------------------------------------------------------
def rotation(dims, base, scaling=None):
    """(frequencies [dims/2], factor on cos and sin) of a rotation, interpolated by YaRN when ``scaling`` is given."""
    f = np.array([base ** (-2.0 * i / dims) for i in range(dims // 2)])
    if not scaling:
        return f, 1.0

    def place(turns):
        return dims * math.log(scaling["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(place(scaling["fast"])), 0)
    hi = min(math.ceil(place(scaling["slow"])), dims - 1)
    ramp = np.clip((np.arange(dims // 2) - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / scaling["factor"] * ramp + f * (1.0 - ramp), 0.1 * math.log(scaling["factor"]) + 1.0


def rotate_halves(x, positions, rot):
    """x [T, heads, d]: number i turns with number i + dims/2 (i < dims/2) by position * frequency_i."""
    if not rot or not rot["dims"]:
        return x
    half = rot["dims"] // 2
    f, factor = rotation(rot["dims"], rot["base"], rot.get("scaling"))
    ang = np.asarray(positions, dtype=np.float64)[:, None] * f[None, :]
    c, s = (np.cos(ang) * factor)[:, None, :], (np.sin(ang) * factor)[:, None, :]
    u, v = x[..., :half], x[..., half:2 * half]
    return np.concatenate([u * c - v * s, v * c + u * s, x[..., 2 * half:]], axis=-1)


# ---- masks --------------------------------------------------------------------------------------------------------
def chunk_mask(T, size):
    """[query, key]: earlier or equal, and in the same run of ``size`` tokens counted from the sequence's start."""
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    return (j <= i) & (i // size == j // size)


def window_mask(T, size, keep_first):
    """[query, key]: earlier or equal, and less than ``size`` tokens back or among the first ``keep_first``."""
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    return (j <= i) & ((i - j < size) | (j < keep_first))


# ---- attention ----------------------------------------------------------------------------------------------------
def softmax_attention(q, k, v, scale, visible):
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H, dv]; query head h reads key head h // (H / G)."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    for h in range(H):
        g = h // (H // G)
        s = np.where(visible, (q[:, h] @ k[:, g].T) * scale, -np.inf)
        e = np.exp(s - s.max(axis=1, keepdims=True))
        out[:, h] = (e / e.sum(axis=1, keepdims=True)) @ v[:, g]
    return out


def heads(x, n):
    return x.reshape(x.shape[0], n, -1)


def chunked_attention(h, w, p, m, eps, positions, shared=None):
    """Queries and keys normed over the whole projection, then turned; chunks; a gate per head.  ``shared``: (keys, values) of
    another layer, used as they are.  Returns (output, keys, values)."""
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q = heads(unit_rms(h @ w[p + "q"].T, eps) * w[p + "q.norm"], H)
    q = rotate_halves(q, positions, m["rot"])
    if shared is None:
        k = heads(unit_rms(h @ w[p + "k"].T, eps) * w[p + "k.norm"], G)
        k, v = rotate_halves(k, positions, m["rot"]), heads(h @ w[p + "v"].T, G)
    else:
        k, v = shared
    o = softmax_attention(q, k, v, m["scale"], chunk_mask(T, m["mask"]["size"]))
    o = o * sigmoid(h @ w[p + "g"].T)[:, :, None]
    return o.reshape(T, -1) @ w[p + "o"].T, k, v


def window_attention(h, w, p, m, eps, positions, shared=None):
    """Queries and keys turned, then brought to unit root mean square per head; a window and the first tokens."""
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q = unit_rms(rotate_halves(heads(h @ w[p + "q"].T, H), positions, m["rot"]), eps)
    if shared is None:
        k = unit_rms(rotate_halves(heads(h @ w[p + "k"].T, G), positions, m["rot"]), eps)
        v = heads(h @ w[p + "v"].T, G)
    else:
        k, v = shared
    o = softmax_attention(q, k, v, m["scale"], window_mask(T, m["mask"]["size"], m["mask"].get("keep_first", 0)))
    return o.reshape(T, -1) @ w[p + "o"].T, k, v


# ---- feed-forward -------------------------------------------------------------------------------------------------
def dense(h, w, p):
    return gelu_erf(h @ w[p + "up"].T) @ w[p + "down"].T


def expert(h, w, stem):
    z = h @ w[stem + ".gate"].T
    return (z * sigmoid(z) * (h @ w[stem + ".up"].T)) @ w[stem + ".down"].T


def router_choice(h, w_router, top, scale):
    """(experts [T, top], weights [T, top]): logistic scores, the largest ``top`` of them over their sum, times ``scale``."""
    s = sigmoid(h @ w_router.T)
    idx = np.argsort(-s, axis=-1, kind="stable")[:, :top]
    c = np.take_along_axis(s, idx, axis=-1)
    return idx, c / (c.sum(axis=-1, keepdims=True) + 1e-20) * scale


def experts_feed_forward(h, w, p, f):
    idx, wts = router_choice(h, w[p + "router"], f["router"]["top"], f["router"].get("scale", 1.0))
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, s in zip(idx[t], wts[t]):
            out[t] += s * expert(h[t:t + 1], w, p + f"e{int(e)}")[0]
    return out


# ---- the model ----------------------------------------------------------------------------------------------------
def forward(cfg, w, tokens, positions=None, collect: Optional[List[np.ndarray]] = None):
    """Logits [T, vocab] of one sequence; ``collect`` receives the stream after every layer."""
    eps = cfg["norm"]["eps"]
    positions = list(range(len(tokens))) if positions is None else positions
    x = w["embed"][np.asarray(tokens)] * cfg.get("embedding", {}).get("scale", 1.0)
    kept = []
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        mixer = {"attention": chunked_attention, "attention_2": window_attention}[layer["type"]]
        shared = kept[m["kv_from"]] if m.get("kv_from") is not None else None
        y, k, v = mixer(squash(x, w, p + "norm1"), w, p + "mix.", m, eps, positions, shared)
        kept.append((k, v))
        x = x + squash(y, w, p + "norm1b")
        f = layer.get("mlp")
        if f is not None:
            h = squash(x, w, p + "norm2")
            y = dense(h, w, p + "mlp.") if f["kind"] == "dense" else experts_feed_forward(h, w, p + "mlp.", f)
            x = x + squash(y, w, p + "norm2b")
        if collect is not None:
            collect.append(x.copy())
    return soft_cap(squash(x, w, "final.norm") @ w["head"].T, cfg.get("logit_softcap"))
