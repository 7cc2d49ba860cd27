"""A plain, slow implementation of the Semanex decoder in float64 numpy: one function per mechanism, whole sequences,
token by token where a recurrence runs.  It shares no code with the package; the tests hold the package to it.  ``cfg`` is
the model's config.json as a dict, ``w`` maps tensor names to float64 arrays."""
from __future__ import annotations

import math

import numpy as np


# ------------------------------------------------------------------ small functions
def sigmoid(z):
    return 0.5 * (1.0 + np.tanh(0.5 * z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.log1p(np.exp(-np.abs(z))) + np.maximum(z, 0.0)


_erf = np.vectorize(math.erf, otypes=[np.float64])


def gelu_exact(z):
    return 0.5 * z * (1.0 + _erf(z / math.sqrt(2.0)))


def rms(x, eps):
    """x divided by its root mean square over the last axis, eps inside the root."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def causal_convolution(x, taps):
    """x [T, C], taps [C, K]: per channel, the last column meets the current token, zeros before the sequence's start."""
    T, C = x.shape
    K = taps.shape[1]
    out = np.zeros((T, C))
    for t in range(T):
        for j in range(K):
            src = t - (K - 1) + j
            if src >= 0:
                out[t] += taps[:, j] * x[src]
    return out


# ------------------------------------------------------------------ positions
def rotate_interleaved(x, positions, dims, base):
    """x [T, heads, d]: channels 2i and 2i+1 of a head's first ``dims`` turn by position * base^(-2i/dims)."""
    f = base ** (-2.0 * np.arange(dims // 2, dtype=np.float64) / dims) if dims else np.zeros(0)
    angle = np.asarray(positions, dtype=np.float64)[:, None] * f[None, :]
    c, s = np.cos(angle)[:, None, :], np.sin(angle)[:, None, :]
    out = x.copy()
    a, b = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = a * c - b * s
    out[..., 1:dims:2] = b * c + a * s
    return out


# ------------------------------------------------------------------ attention
def softmax_attention(q, k, v, scale, softcap=None, sink=None):
    """q [T, H, d], k [T, G, d], v [T, G, vd] of one sequence from position 0; query i sees every key j <= i.  A ``softcap``
    c turns a scaled score s into c tanh(s / c).  ``sink`` [H]: one more term exp(sink_h) in head h's denominator, without a
    value."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    for h in range(H):
        g = h // (H // G)
        for i in range(T):
            s = (k[:i + 1, g] @ q[i, h]) * scale
            if softcap:
                s = softcap * np.tanh(s / softcap)
            m = s.max() if sink is None else max(s.max(), sink[h])
            e = np.exp(s - m)
            den = e.sum() + (0.0 if sink is None else math.exp(sink[h] - m))
            out[i, h] = (e / den) @ v[:i + 1, g]
    return out


def capped_attention(m, w, p, h, eps):
    """Grouped heads, an RMS norm per query and key head, capped scores, no positions, a gate per output channel."""
    H, G, d, vd = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q = rms((h @ w[p + "q"].T).reshape(-1, H, d), eps) * w[p + "q.norm"]
    k = rms((h @ w[p + "k"].T).reshape(-1, G, d), eps) * w[p + "k.norm"]
    v = (h @ w[p + "v"].T).reshape(-1, G, vd)
    o = softmax_attention(q, k, v, float(m["scale"]), m.get("softcap"))
    return (o.reshape(len(h), -1) * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def latent_attention(m, w, p, h, positions, eps):
    """Keys and values expanded from a latent per token, one rotated key part shared by the heads, a sink, a gate per channel."""
    H, d, rd, vd, r = int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["kv_rank"])
    T, rot = len(h), m["rot"]
    cq = rms(h @ w[p + "dq"].T, eps) * w[p + "dq.norm"]
    q = (cq @ w[p + "uq"].T).reshape(T, H, d + rd)
    q_rot = rotate_interleaved(q[..., d:], positions, int(rot["dims"]), float(rot["base"]))
    down = h @ w[p + "dkv"].T
    c = rms(down[:, :r], eps) * w[p + "dkv.norm"]
    k_rot = rotate_interleaved(down[:, None, r:], positions, int(rot["dims"]), float(rot["base"]))
    k = np.concatenate([(c @ w[p + "uk"].T).reshape(T, H, d), np.repeat(k_rot, H, axis=1)], axis=-1)
    v = (c @ w[p + "uv"].T).reshape(T, H, vd)
    o = softmax_attention(np.concatenate([q[..., :d], q_rot], axis=-1), k, v, float(m["scale"]), None, w[p + "sink"])
    return (o.reshape(T, H * vd) * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


# ------------------------------------------------------------------ the state-space recurrence
def state_space_scan(x, B, C, dt, rate, D):
    """x [T, H, P], B, C [T, G, N], dt [T, H] (positive), rate [H] (positive), D [H]: per head
    S <- exp(-rate dt) S + dt B x^T,  y = S^T C + D x.  Returns y [T, H, P]."""
    T, H, P = x.shape
    G, N = B.shape[1], B.shape[2]
    S = np.zeros((H, N, P))
    y = np.zeros((T, H, P))
    for t in range(T):
        for h in range(H):
            g = h // (H // G)
            S[h] = math.exp(-rate[h] * dt[t, h]) * S[h] + dt[t, h] * np.outer(B[t, g], x[t, h])
            y[t, h] = S[h].T @ C[t, g] + D[h] * x[t, h]
    return y


def state_space_mixer(m, w, p, h, eps):
    H, P, N, G = int(m["heads"]), int(m["vdim"]), int(m["state"]), int(m["groups"])
    inner, T = H * P, len(h)
    proj = h @ w[p + "in"].T
    z, xbc, dt = proj[:, :inner], proj[:, inner:2 * inner + 2 * G * N], proj[:, 2 * inner + 2 * G * N:]
    xbc = silu(causal_convolution(xbc, w[p + "conv"]) + w[p + "conv.b"])
    x, B, C = xbc[:, :inner], xbc[:, inner:inner + G * N], xbc[:, inner + G * N:]
    y = state_space_scan(x.reshape(T, H, P), B.reshape(T, G, N), C.reshape(T, G, N), softplus(dt + w[p + "dt_bias"]),
                         np.exp(w[p + "A_log"]), w[p + "D"]).reshape(T, inner)
    y = y * silu(z)
    parts = int(m["norm_groups"])
    y = rms(y.reshape(T, parts, inner // parts), eps).reshape(T, inner) * w[p + "norm"]
    return y @ w[p + "o"].T


def parallel_mixer(m, w, p, h, eps):
    return float(m["left_scale"]) * capped_attention(m["left"], w, p + "left.", h, eps) + \
        float(m["right_scale"]) * state_space_mixer(m["right"], w, p + "right.", h, eps)


# ------------------------------------------------------------------ the model
def feed_forward(w, p, x):
    return gelu_exact(x @ w[p + "up"].T) @ w[p + "down"].T


def forward(cfg, w, tokens):
    """Logits [T, vocab] of one sequence, and the stream after every layer [layers, T, width]."""
    eps, alpha = float(cfg["norm"]["eps"]), float(cfg["postln_alpha"])
    positions = np.arange(len(tokens))
    x = w["embed"][np.asarray(tokens)] * float(cfg["embedding"]["scale"])
    after = []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        h = x + causal_convolution(x, w[p + "canon1"])
        if layer["type"] == "parallel":
            y = parallel_mixer(layer["mixer"], w, p + "mix.", h, eps)
        else:
            y = latent_attention(layer["mixer"], w, p + "mix.", h, positions, eps)
        x = rms(alpha * x + y, eps) * w[p + "norm1"]
        if layer.get("mlp"):
            x = rms(alpha * x + feed_forward(w, p + "mlp.", x), eps) * w[p + "norm2"]
        after.append(x.copy())
    return (rms(x, eps) * w["final.norm"]) @ w["head"].T, np.stack(after)
