"""Plain, slow implementation of the Segorax decoder in numpy float64: whole sequences, no cache, one function per
mechanism, keys and values of every head made in full.  It is the oracle of the Segorax tests and shares no code with the
package.

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


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


_erf = np.vectorize(math.erf, otypes=[np.float64])


def gelu_erf(z):
    return 0.5 * z * (1.0 + _erf(z / math.sqrt(2.0)))


def rms_norm(x, w, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * w


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


def rotate_pairs(x, positions, dims, base, scaling=None):
    """x [T, ..., d]: numbers 2i and 2i + 1 (i < dims/2) turn together by position * frequency_i."""
    f, factor = rotation(dims, base, scaling)
    ang = np.asarray(positions, dtype=np.float64)[:, None] * f[None, :]
    shape = (len(positions),) + (1,) * (x.ndim - 2) + (dims // 2,)
    c, s = (np.cos(ang) * factor).reshape(shape), (np.sin(ang) * factor).reshape(shape)
    out = x.copy()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * c - v * s
    out[..., 1:dims:2] = v * c + u * s
    return out


# ---- attention ----------------------------------------------------------------------------------------------------
def softmax_attention(q, k, v, scale, sink=None):
    """q, k [T, H, d], v [T, H, dv]: causal; with ``sink`` [H] every head's denominator also holds exp(sink_h)."""
    T, H, _ = q.shape
    out = np.zeros((T, H, v.shape[2]))
    later = np.triu(np.ones((T, T), dtype=bool), 1)
    for h in range(H):
        s = (q[:, h] @ k[:, h].T) * scale
        s[later] = -np.inf
        m = s.max(axis=1, keepdims=True)
        if sink is not None:
            m = np.maximum(m, sink[h])
        e = np.exp(s - m)
        den = e.sum(axis=1, keepdims=True)
        if sink is not None:
            den = den + np.exp(sink[h] - m)
        out[:, h] = (e / den) @ v[:, h]
    return out


def latent_attention(h, w, p, m, eps, positions, low_rank_q, with_sink):
    """Keys and values of all heads from one normed latent per token and one turned key part that the heads share; queries
    straight from h, or through a normed latent of their own."""
    T = h.shape[0]
    H, dk, dr, dv, r = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    if low_rank_q:
        q = rms_norm(h @ w[p + "dq"].T, w[p + "dq.norm"], eps) @ w[p + "uq"].T
    else:
        q = h @ w[p + "q"].T
    q = q.reshape(T, H, dk + dr)
    down = h @ w[p + "dkv"].T
    c = rms_norm(down[:, :r], w[p + "dkv.norm"], eps)
    k_plain = (c @ w[p + "uk"].T).reshape(T, H, dk)
    v = (c @ w[p + "uv"].T).reshape(T, H, dv)
    rot = m["rot"]
    k_turned = rotate_pairs(down[:, r:], positions, rot["dims"], rot["base"], rot.get("scaling"))
    q_turned = rotate_pairs(q[..., dk:], positions, rot["dims"], rot["base"], rot.get("scaling"))
    q = np.concatenate([q[..., :dk], q_turned], axis=-1)
    k = np.concatenate([k_plain, np.repeat(k_turned[:, None, :], H, axis=1)], axis=-1)
    o = softmax_attention(q, k, v, m["scale"], w[p + "sink"] if with_sink else None)
    return o.reshape(T, H * dv) @ w[p + "o"].T


# ---- feed-forward -------------------------------------------------------------------------------------------------
def dense(h, w, p):
    return (gelu_tanh(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def expert(h, w, stem):
    return gelu_erf(h @ w[stem + ".up"].T) @ w[stem + ".down"].T


def router_choice(h, w_router, correction, top, groups):
    """(experts [T, top], their scores [T, top]).  Scores are logistic; the choice goes by score + correction; ``groups``
    (count, keep) or None: only experts of the ``keep`` groups whose two best choice scores add up to most are eligible."""
    s = sigmoid(h @ w_router.T)
    T, E = s.shape
    choice = s + correction[None, :]
    idx = np.zeros((T, top), dtype=np.int64)
    for t in range(T):
        c = choice[t].copy()
        if groups is not None:
            count, keep = groups
            size = E // count
            total = [np.sort(c[g * size:(g + 1) * size])[::-1][:2].sum() for g in range(count)]
            best = np.argsort(-np.array(total), kind="stable")[:keep]
            for g in range(count):
                if g not in best:
                    c[g * size:(g + 1) * size] = -np.inf
        idx[t] = np.argsort(-c, kind="stable")[:top]
    return idx, np.take_along_axis(s, idx, axis=-1)


def experts_feed_forward(h, w, p, f):
    g = f["router"].get("groups")
    idx, wts = router_choice(h, w[p + "router"], w[p + "correction"], f["router"]["top"], (g["count"], g["keep"]) if g else None)
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, s in zip(idx[t], wts[t]):
            out[t] += s * expert(h[t:t + 1], w, p + f"e{int(e)}")[0]
    if f.get("shared"):
        out += sigmoid(h @ w[p + "shared.sg"].T) * expert(h, w, p + "shared")
    return out


# ---- the model ----------------------------------------------------------------------------------------------------
def forward(cfg, w, tokens, positions=None, collect: Optional[List[np.ndarray]] = None):
    """Logits [T, vocab] of one sequence; ``collect`` receives the stream after every layer."""
    eps, m = cfg["norm"]["eps"], cfg.get("residual_mult", 1.0)
    positions = list(range(len(tokens))) if positions is None else positions
    x = w["embed"][np.asarray(tokens)] * cfg.get("embedding", {}).get("scale", 1.0)
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        low, sink = {"latent_attention": (True, True), "latent_attention_2": (False, False)}[layer["type"]]
        y = latent_attention(x, w, p + "mix.", layer["mixer"], eps, positions, low, sink)
        x = x + m * rms_norm(y, w[p + "norm1"], eps)
        f = layer.get("mlp")
        if f is not None:
            y = dense(x, w, p + "mlp.") if f["kind"] == "dense" else experts_feed_forward(x, w, p + "mlp.", f)
            x = x + m * rms_norm(y, w[p + "norm2"], eps)
        if collect is not None:
            collect.append(x.copy())
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T * cfg.get("logit_scale", 1.0)
