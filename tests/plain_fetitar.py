"""A plain, slow implementation of the Fetitar decoder in float64 numpy: one function per mechanism, whole sequences, no cache.
It shares no code with the package; the tests hold the package to it.  ``cfg`` is the model's config.json as a dict, ``w`` maps
tensor names to float64 arrays.  ``rms`` is x over the root of its mean square plus eps."""
from __future__ import annotations

import math

import numpy as np


# ------------------------------------------------------------------ small functions
def sigmoid(z):
    return 0.5 * (1.0 + np.tanh(0.5 * z))


def silu(z):
    return z * sigmoid(z)


def rms(x, eps):
    """x divided by its root mean square over the last axis, eps inside the root."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def centred_norm(x, gain, eps):
    """A norm whose gain is kept around zero."""
    return rms(x, eps) * (1.0 + gain)


# ------------------------------------------------------------------ embedding
def bigram_rows(tokens, buckets, mul_prev, mul_cur):
    """The pair table's row of every token: a hash of (token before, token), the last row for a sequence's first token."""
    rows = []
    for t, cur in enumerate(tokens):
        rows.append(buckets if t == 0 else (int(tokens[t - 1]) * mul_prev + int(cur) * mul_cur) % buckets)
    return rows


def embed(cfg, w, tokens):
    e = cfg["embedding"]
    x = w["embed"][np.asarray(tokens)] * float(e.get("scale", 1.0))
    if e.get("bigram"):
        b = e["bigram"]
        x = x + w["bigram"][bigram_rows(tokens, int(b["buckets"]), int(b["mul_prev"]), int(b["mul_cur"]))]
    return x


# ------------------------------------------------------------------ positions
def yarn_frequencies(dims, base, scaling=None):
    """(frequency of every pair, factor on cosine and sine)."""
    f = np.array([float(base) ** (-2.0 * i / dims) for i in range(dims // 2)])
    if not scaling:
        return f, 1.0
    factor, original = float(scaling["factor"]), float(scaling["original"])

    def index(turns):
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(float(base)))

    lo = max(math.floor(index(float(scaling["fast"]))), 0)
    hi = min(math.ceil(index(float(scaling["slow"]))), dims - 1)
    out = np.zeros_like(f)
    for i in range(dims // 2):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out[i] = f[i] / factor * ramp + f[i] * (1.0 - ramp)
    return out, 0.1 * math.log(factor) + 1.0


def rotate_halves(x, positions, dims, base, scaling=None):
    """x [T, heads, d]: channels i and i + dims/2 of a head's first ``dims`` turn by position * f_i."""
    if not dims:
        return x
    f, grow = yarn_frequencies(dims, base, scaling)
    angle = np.asarray(positions, dtype=np.float64)[:, None] * f[None, :]
    c, s = (np.cos(angle) * grow)[:, None, :], (np.sin(angle) * grow)[:, None, :]
    out = x.copy()
    a, b = x[..., :dims // 2], x[..., dims // 2:dims]
    out[..., :dims // 2] = a * c - b * s
    out[..., dims // 2:dims] = b * c + a * s
    return out


def distance_slopes(heads):
    return [2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)]


# ------------------------------------------------------------------ attention
def softmax_attention(q, k, v, scale, window=None, slopes=None):
    """q [T, H, d], k [T, G, d], v [T, G, vd] of one sequence from position 0; query i sees key j when 0 <= i - j < window (None:
    every j <= i).  ``slopes`` [H]: slope_h (i - j) is taken off the scaled score."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    for h in range(H):
        g = h // (H // G)
        for i in range(T):
            j0 = 0 if window is None else max(0, i - window + 1)
            s = (k[j0:i + 1, g] @ q[i, h]) * scale
            if slopes is not None:
                s = s - slopes[h] * (i - np.arange(j0, i + 1))
            e = np.exp(s - s.max())
            out[i, h] = (e / e.sum()) @ v[j0:i + 1, g]
    return out


def window_of(m):
    return (m.get("mask") or {}).get("size")


def mixed_values(v, first, weight):
    """(1 - weight) v + weight first: a layer's values mixed with the first mixing layer's of the same token."""
    return (1.0 - weight) * v + weight * first


def sloped_attention(m, w, p, h, eps, first=None):
    """Grouped heads; biases; one norm over all query and one over all key channels of a token; a penalty per distance; values
    mixed with ``first``.  Returns (output, this layer's own values before any mixing)."""
    H, G, d, vd, T = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), len(h)
    q = rms(h @ w[p + "q"].T + w[p + "q.b"], eps) * w[p + "q.norm"]
    k = rms(h @ w[p + "k"].T + w[p + "k.b"], eps) * w[p + "k.norm"]
    own = h @ w[p + "v"].T + w[p + "v.b"]
    v = own if first is None else mixed_values(own, first, float(w[p + "vmix"]))
    o = softmax_attention(q.reshape(T, H, d), k.reshape(T, G, d), v.reshape(T, G, vd), float(m["scale"]), window_of(m), distance_slopes(H))
    return o.reshape(T, -1) @ w[p + "o"].T + w[p + "o.b"], own


def latent_attention(m, w, p, h, positions, eps):
    """Keys and values expanded from a latent per token, one rotated key part shared by the heads, a gate per head."""
    H, d, rd, vd, r = int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["kv_rank"])
    T, rot = len(h), m["rot"]
    turn = lambda x: rotate_halves(x, positions, int(rot["dims"]), float(rot["base"]), rot.get("scaling"))
    cq = rms(h @ w[p + "dq"].T, eps) * w[p + "dq.norm"]
    q = (cq @ w[p + "uq"].T).reshape(T, H, d + rd)
    down = h @ w[p + "dkv"].T
    c = rms(down[:, :r], eps) * w[p + "dkv.norm"]
    k = np.concatenate([(c @ w[p + "uk"].T).reshape(T, H, d), np.repeat(turn(down[:, None, r:]), H, axis=1)], axis=-1)
    v = (c @ w[p + "uv"].T).reshape(T, H, vd)
    o = softmax_attention(np.concatenate([q[..., :d], turn(q[..., d:])], axis=-1), k, v, float(m["scale"]), window_of(m))
    o = o * sigmoid(h @ w[p + "g"].T)[:, :, None]
    return o.reshape(T, H * vd) @ w[p + "o"].T


# ------------------------------------------------------------------ the model
def feed_forward(w, p, x):
    return (silu(x @ w[p + "gate"].T + w[p + "gate.b"]) * (x @ w[p + "up"].T + w[p + "up.b"])) @ w[p + "down"].T + w[p + "down.b"]


def forward(cfg, w, tokens):
    """Logits [T, vocab] of one sequence, and the stream after every layer [layers, T, width]."""
    eps = float(cfg["norm"]["eps"])
    positions = np.arange(len(tokens))
    x = embed(cfg, w, tokens)
    after, first = [], None
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = centred_norm(x, w[p + "norm1"], eps)
        if layer["type"] == "latent_attention":
            y = latent_attention(m, w, p + "mix.", h, positions, eps)
        else:
            y, own = sloped_attention(m, w, p + "mix.", h, eps, first if m.get("v_mix") else None)
            if m.get("v_mix") and first is None:
                first = own
        x = x + centred_norm(y, w[p + "norm1b"], eps)
        if layer.get("mlp"):
            x = x + centred_norm(feed_forward(w, p + "mlp.", centred_norm(x, w[p + "norm2"], eps)), w[p + "norm2b"], eps)
        after.append(x.copy())
    return centred_norm(x, w["final.norm"], eps) @ w["head"].T, np.stack(after)
