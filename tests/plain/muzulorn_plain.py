"""Plain, slow, whole-sequence statement of the Muzulorn design, one function per mechanism.

A decoder-only model whose embedding takes in a row that belongs to the pair (token before, token), and whose stream is
several copies that every sublayer mixes anew (hyper-connections).  A mixer is softmax attention without rotation (norms over
the whole query and key projections, a query factor that grows with the position, capped scores, a learned bias by bucketed
distance; possibly another layer's keys and values), latent attention (queries through a latent of their own, one rotated key
part for all heads, a sliding window, a sink, a gate per output channel), or a state-space recurrence with one decay per token
and head (Mamba-2).  The feed-forward, if any, is dense with the exact gelu or a mixture of gated experts beside a gated
shared one.

Everything is numpy in one floating type (float64 by default), no cache, no batching; the recurrence is walked token by
token.  Shares no code with the package.
"""

from __future__ import annotations

import json
import math
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


_erf = np.vectorize(math.erf, otypes=[np.float64])


def gelu(z):
    return (0.5 * z * (1.0 + _erf(z / math.sqrt(2.0)))).astype(z.dtype)


def softplus(z):
    return np.logaddexp(0.0, z)


def unit_rms(x, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def norm_around_zero(x, w, eps):
    """The stored weight is what the gain has beyond one."""
    return unit_rms(x, eps) * (1.0 + w)


def norm(x, w, eps):
    return unit_rms(x, eps) * w


def softmax(s, sink=None):
    """Over the last axis; ``sink``: one more term exp(sink) in the denominator."""
    top = s.max(-1, keepdims=True) if sink is None else np.maximum(s.max(-1, keepdims=True), sink)
    e = np.exp(s - top)
    return e / (e.sum(-1, keepdims=True) + (0.0 if sink is None else np.exp(sink - top)))


def rotate_pairs(x, positions, rot):
    """x [T, heads, d]: channel 2i of each head with channel 2i + 1, for the first ``dims`` channels; the rest pass."""
    if rot is None or not rot["dims"]:
        return x
    dims = int(rot["dims"])
    f = float(rot["base"]) ** (-2.0 * np.arange(dims // 2, dtype=np.float64) / dims)
    ang = np.asarray(positions, dtype=np.float64)[:, None] * f[None, :]
    c, s = np.cos(ang)[:, None, :], np.sin(ang)[:, None, :]
    out = x.copy()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * c - v * s
    out[..., 1:dims:2] = v * c + u * s
    return out


# ---- embedding ----------------------------------------------------------------------------------

def embedding(ids, cfg, w):
    x = w["embed"][np.asarray(ids)]
    bg = (cfg.get("embedding") or {}).get("bigram")
    if bg is None:
        return x.copy()
    rows = [bg["buckets"]] + [(int(a) * bg["mul_prev"] + int(b) * bg["mul_cur"]) % bg["buckets"] for a, b in zip(ids[:-1], ids[1:])]
    return x + w["bigram"][np.asarray(rows)]


# ---- mixers -----------------------------------------------------------------------------------

def distance_bucket(n: int, buckets: int, limit: int) -> int:
    """Small distances have buckets of their own, larger ones share buckets that widen with the logarithm."""
    half = buckets // 2
    if n < half:
        return n
    return min(buckets - 1, half + math.floor(math.log(n / half) / math.log(limit / half) * (buckets - half)))


def query_factor(positions, q_temp):
    p = np.asarray(positions, dtype=np.float64)
    return 1.0 + q_temp["coef"] * np.log(np.floor((p + 1.0) / q_temp["every"]) + 1.0)


def keys_values(h, w, p, m, eps):
    """What an attention layer with projections of its own leaves for itself and for layers that borrow: keys [T, G, dim]
    (normed over the whole projection) and values [T, G, vdim]."""
    T, G = h.shape[0], m["kv_heads"]
    k = norm(h @ w[p + "k"].T + w[p + "k.b"], w[p + "k.norm"], eps)
    v = h @ w[p + "v"].T + w[p + "v.b"]
    return k.reshape(T, G, m["dim"]), v.reshape(T, G, m["vdim"])


def attention(h, w, p, m, eps, kv):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    k, v = kv
    q = norm(h @ w[p + "q"].T + w[p + "q.b"], w[p + "q.norm"], eps)
    if m.get("q_temp") is not None:
        q = q * query_factor(np.arange(T), m["q_temp"])[:, None]
    q = q.reshape(T, H, d)
    rel = w[p + "rel"]
    by_distance = rel[[distance_bucket(n, rel.shape[0], m["bias_max"]) for n in range(T)]]       # [T, H]
    dist = np.arange(T)[:, None] - np.arange(T)[None, :]
    out = np.zeros((T, H, dv), h.dtype)
    for n in range(H):
        s = (q[:, n] @ k[:, n // (H // G)].T) * m["scale"]
        if m.get("softcap") is not None:
            s = m["softcap"] * np.tanh(s / m["softcap"])
        s = s + by_distance[np.maximum(dist, 0), n]
        out[:, n] = softmax(np.where(dist >= 0, s, -np.inf)) @ v[:, n // (H // G)]
    return out.reshape(T, H * dv) @ w[p + "o"].T + w[p + "o.b"]


def latent_attention(h, w, p, m, eps):
    T = h.shape[0]
    H, d, r, dv, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = np.arange(T)
    q = (norm(h @ w[p + "dq"].T, w[p + "dq.norm"], eps) @ w[p + "uq"].T).reshape(T, H, d + r)
    qn, qr = q[..., :d], rotate_pairs(q[..., d:], pos, m.get("rot"))
    down = h @ w[p + "dkv"].T
    c = norm(down[:, :rank], w[p + "dkv.norm"], eps)
    kr = rotate_pairs(down[:, None, rank:], pos, m.get("rot"))[:, 0]
    kn = (c @ w[p + "uk"].T).reshape(T, H, d)
    v = (c @ w[p + "uv"].T).reshape(T, H, dv)
    dist = pos[:, None] - pos[None, :]
    seen = (dist >= 0) & (dist < m["mask"]["size"]) if m.get("mask") is not None else dist >= 0
    out = np.zeros((T, H, dv), h.dtype)
    for n in range(H):
        s = (qn[:, n] @ kn[:, n].T + qr[:, n] @ kr.T) * m["scale"]
        out[:, n] = softmax(np.where(seen, s, -np.inf), w[p + "sink"][n]) @ v[:, n]
    return (out.reshape(T, H * dv) * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def causal_convolution(x, taps_w, bias):
    """x [T, C]: per channel sum_j w[:, j] x_(t - (taps-1) + j) + bias, zeros before the start."""
    T, C = x.shape
    taps = taps_w.shape[1]
    padded = np.concatenate([np.zeros((taps - 1, C), x.dtype), x], axis=0)
    return sum(padded[j:j + T] * taps_w[:, j] for j in range(taps)) + bias


def state_space(xs, B, C, dt, a_log, D):
    """xs [T, H, dv], B and C [T, H, N], dt [T, H] step sizes: S <- exp(-exp(a_log) dt) S + dt B x^T, y = S^T C + D x."""
    T, H, dv = xs.shape
    S = np.zeros((H, B.shape[2], dv), xs.dtype)
    y = np.zeros_like(xs)
    for t in range(T):
        S = np.exp(-np.exp(a_log) * dt[t])[:, None, None] * S + (dt[t][:, None] * B[t])[:, :, None] * xs[t][:, None, :]
        y[t] = np.einsum("hij,hi->hj", S, C[t]) + D[:, None] * xs[t]
    return y


def mamba2(h, w, p, m, eps):
    T = h.shape[0]
    H, dv, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * dv
    z, xbc, dt = np.split(h @ w[p + "in"].T, [inner, 2 * inner + 2 * G * N], axis=1)
    xbc = silu(causal_convolution(xbc, w[p + "conv"], w[p + "conv.b"]))
    xs, B, C = np.split(xbc, [inner, inner + G * N], axis=1)
    spread = np.arange(H) // (H // G)
    y = state_space(xs.reshape(T, H, dv), B.reshape(T, G, N)[:, spread], C.reshape(T, G, N)[:, spread],
                    softplus(dt + w[p + "dt_bias"]), w[p + "A_log"], w[p + "D"])
    y = y.reshape(T, inner) * silu(z)
    parts = m["norm_groups"]
    y = unit_rms(y.reshape(T, parts, inner // parts), eps).reshape(T, inner) * w[p + "norm"]
    return y @ w[p + "o"].T


# ---- feed-forward -----------------------------------------------------------------------------------

def gated_unit(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def experts(h, w, p, mlp, margins=None):
    """``margins`` (a list) receives, per token, the gap between the last chosen expert's logit and the best one left out, relative to
    the logits' spread."""
    z = h @ w[p + "router"].T + w[p + "router.b"]
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        won = np.argsort(-z[t], kind="stable")[:mlp["router"]["top"]]
        for e, weight in zip(won, softmax(z[t][won])):
            out[t] += weight * gated_unit(h[t:t + 1], w, f"{p}e{e}.")[0]
    if mlp.get("shared") is not None:
        out = out + gated_unit(h, w, p + "shared.") * sigmoid(h @ w[p + "shared.sg"].T)
    top = mlp["router"]["top"]
    if margins is not None and top < z.shape[1]:
        s = -np.sort(-z, axis=1)
        margins.append((s[:, top - 1] - s[:, top]) / np.sqrt((z * z).mean(-1)))
    return out


def feed_forward(h, w, p, mlp, margins=None):
    if mlp["kind"] == "dense":
        return gelu(h @ w[p + "up"].T) @ w[p + "down"].T
    return experts(h, w, p, mlp, margins)


# ---- the streams --------------------------------------------------------------------------------------

def connect(streams, w, p, mult, sublayer):
    """streams [s, T, W]: the sublayer reads a weighted sum of them; each new stream is a mix of the old ones (the mix
    matrix's rows are the old streams) plus its share of the sublayer's output."""
    u = np.einsum("s,stw->tw", w[p + "in"], streams)
    y = sublayer(u)
    return np.einsum("stw,sr->rtw", streams, w[p + "mix"]) + mult * w[p + "out"][:, None, None] * y[None]


# ---- the model ------------------------------------------------------------------------------------

def forward(ids, cfg, w, after_layers=None, margins=None):
    """Logits [T, vocab] of one whole sequence.  ``after_layers`` (a list) receives the sum of the streams after every layer,
    ``margins`` what `experts` says of every router."""
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    x = embedding(list(ids), cfg, w)
    streams = np.repeat(x[None], cfg["streams"], axis=0)
    kept = {}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]

        def mixer(u):
            h = norm_around_zero(u, w[p + "norm1"], eps)
            if layer["type"] == "latent_attention":
                return latent_attention(h, w, p + "mix.", m, eps)
            if layer["type"] == "mamba2":
                return mamba2(h, w, p + "mix.", m, eps)
            src = m.get("kv_from")
            if src is None:
                kept[i] = keys_values(h, w, p + "mix.", m, eps)
            return attention(h, w, p + "mix.", m, eps, kept[i if src is None else src])
        streams = connect(streams, w, p + "hc1.", mult, mixer)
        if layer["mlp"] is not None:
            streams = connect(streams, w, p + "hc2.", mult, lambda u: feed_forward(norm_around_zero(u, w[p + "norm2"], eps), w, p + "mlp.", layer["mlp"], margins))
        if after_layers is not None:
            after_layers.append(streams.sum(0))
    return norm_around_zero(streams.sum(0), w["final.norm"], eps) @ w["head"].T
