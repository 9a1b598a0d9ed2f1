"""Plain, slow, whole-sequence statement of the Sezopel design, one function per mechanism.

A decoder-only model whose embedding rows are scaled and whose sublayers read the stream as it is: only what they give
back is normed, x <- x + norm1(mixer(x)), x <- x + norm2(ff(x)).  Behind the feed-forward every layer takes in a vector
that belongs to the token and the layer: x <- x + norm(P (gelu(G x) * e)).  A mixer is softmax attention (normed, partly
rotated queries and keys, capped scores, one sigmoid gate per head, possibly another layer's keys and values) or retention
(linear attention with a fixed decay per head on rotated queries and keys).  The feed-forward is two matrices with a
squared relu between them.  The logits are capped.

Everything is numpy in one floating type (float64 by default), no cache, no batching; the recurrence is walked token by
token.  Shares no code with the package.
"""

from __future__ import annotations

import json
import struct

import numpy as np


# ---- model folder ---------------------------------------------------------------------------

def read_safetensors(path: str, dtype=np.float64) -> dict:
    with open(path, "rb") as f:
        (n,) = struct.unpack("<Q", f.read(8))
        header = json.loads(f.read(n))
        blob = f.read()
    out = {}
    for name, meta in header.items():
        if name == "__metadata__":
            continue
        lo, hi = meta["data_offsets"]
        raw = blob[lo:hi]
        if meta["dtype"] == "BF16":
            arr = (np.frombuffer(raw, dtype="<u2").astype(np.uint32) << 16).view(np.float32).astype(dtype)
        elif meta["dtype"] == "F32":
            arr = np.frombuffer(raw, dtype="<f4").astype(dtype)
        elif meta["dtype"] == "I32":
            arr = np.frombuffer(raw, dtype="<i4")
        else:
            raise ValueError(f"{name}: dtype {meta['dtype']}")
        out[name] = arr.reshape(meta["shape"]).copy()
    return out


def load_model(model_dir: str, dtype=np.float64):
    with open(f"{model_dir}/config.json") as f:
        cfg = json.load(f)
    return cfg, read_safetensors(f"{model_dir}/model.safetensors", dtype)


# ---- small pieces ---------------------------------------------------------------------------

def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def unit_rms(x, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def norm(x, w, eps):
    return unit_rms(x, eps) * w


def cap(z, limit):
    """Values bent into (-limit, limit); no limit leaves them."""
    return z if limit is None else limit * np.tanh(z / limit)


def rotate(x, positions, rot):
    """x [T, heads, d]: channel i of each head with channel i + dims/2, for the first ``dims`` channels; the rest pass."""
    if rot is None:
        return x
    dims = int(rot["dims"])
    half = dims // 2
    f = float(rot["base"]) ** (-2.0 * np.arange(half, dtype=np.float64) / dims)
    ang = np.asarray(positions, dtype=np.float64)[:, None] * f[None, :]
    c, s = np.cos(ang)[:, None, :], np.sin(ang)[:, None, :]
    out = x.copy()
    u, v = x[..., :half], x[..., half:dims]
    out[..., :half] = u * c - v * s
    out[..., half:dims] = v * c + u * s
    return out


# ---- mixers -----------------------------------------------------------------------------------

def keys_values(h, w, p, m, eps):
    """What a layer with projections of its own leaves for itself and for layers that borrow: rotated, normed keys
    [T, G, dim] and values [T, G, vdim]."""
    T = h.shape[0]
    G, d, dv = m["kv_heads"], m["dim"], m["vdim"]
    k = rotate((h @ w[p + "k"].T).reshape(T, G, d), np.arange(T), m.get("rot"))
    return unit_rms(k, eps), (h @ w[p + "v"].T).reshape(T, G, dv)


def attention(h, w, p, m, eps, kv):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    k, v = kv
    q = unit_rms(rotate((h @ w[p + "q"].T).reshape(T, H, d), np.arange(T), m.get("rot")), eps)
    gate = sigmoid(h @ w[p + "g"].T)                                           # [T, H]
    out = np.zeros((T, H, dv), h.dtype)
    for n in range(H):
        kh, vh = k[:, n // (H // G)], v[:, n // (H // G)]
        s = cap((q[:, n] @ kh.T) * m["scale"], m.get("softcap"))
        s = np.where(np.tril(np.ones((T, T), bool)), s, -np.inf)
        e = np.exp(s - s.max(-1, keepdims=True))
        out[:, n] = (e / e.sum(-1, keepdims=True)) @ vh * gate[:, n:n + 1]
    return out.reshape(T, H * dv) @ w[p + "o"].T


def retention(h, w, p, m, eps):
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    pos = np.arange(T)
    q = rotate((h @ w[p + "q"].T).reshape(T, H, d), pos, m.get("rot"))
    k = rotate((h @ w[p + "k"].T).reshape(T, H, d), pos, m.get("rot")) * d ** -0.5
    v = (h @ w[p + "v"].T).reshape(T, H, dv)
    decay = np.asarray(m["decay"], dtype=h.dtype)
    S = np.zeros((H, d, dv), h.dtype)
    o = np.zeros((T, H, dv), h.dtype)
    for t in range(T):
        S = S * decay[:, None, None] + k[t][:, :, None] * v[t][:, None, :]
        o[t] = np.einsum("hij,hi->hj", S, q[t])
    return (unit_rms(o, eps).reshape(T, H * dv) * silu(h @ w[p + "g"].T)) @ w[p + "o"].T


# ---- the layer's other terms --------------------------------------------------------------------

def feed_forward(h, w, p):
    return np.maximum(h @ w[p + "up"].T, 0.0) ** 2 @ w[p + "down"].T


def token_side(h, ids, w, layer, dim, eps):
    """The term of the token's own vector for this layer, normed."""
    p = f"l{layer}.side."
    e = w["side.embed"][np.asarray(ids)][:, layer * dim:(layer + 1) * dim]
    return norm((gelu_tanh(h @ w[p + "gate"].T) * e) @ w[p + "proj"].T, w[p + "norm"], eps)


# ---- the model ------------------------------------------------------------------------------------

def forward(ids, cfg, w, streams=None):
    """Logits [T, vocab] of one whole sequence.  ``streams`` (a list) receives the stream after every layer."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][np.asarray(ids)] * cfg["embedding"]["scale"]
    kept = {}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        if layer["type"] == "attention":
            src = m.get("kv_from")
            if src is None:
                kept[i] = keys_values(x, w, p + "mix.", m, eps)
            y = attention(x, w, p + "mix.", m, eps, kept[i if src is None else src])
        else:
            y = retention(x, w, p + "mix.", m, eps)
        x = x + norm(y, w[p + "norm1"], eps)
        if layer["mlp"] is not None:
            x = x + norm(feed_forward(x, w, p + "mlp."), w[p + "norm2"], eps)
        if cfg.get("token_side") is not None:
            x = x + token_side(x, ids, w, i, cfg["token_side"]["dim"], eps)
        if streams is not None:
            streams.append(x.copy())
    return cap(norm(x, w["final.norm"], eps) @ w["head"].T, cfg.get("logit_softcap"))
