"""Plain, slow restatement of the Metapel decoder in numpy (test infrastructure only).

One function per mechanism, written from the design's equations, float64 throughout unless a caller
passes another dtype. A sequence is always computed whole, from its first token: there is no cache, no
state and no batch, so nothing here can share a fault with the incremental product path. ``config`` is the
dictionary of a ``config.json``; ``weights`` maps tensor names to arrays.
"""
from __future__ import annotations

import numpy as np


def sigmoid(x):
    return np.where(x >= 0, 1.0 / (1.0 + np.exp(-np.abs(x))), np.exp(-np.abs(x)) / (1.0 + np.exp(-np.abs(x))))


def silu(x):
    return x * sigmoid(x)


def gelu_tanh(x):
    return 0.5 * x * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (x + 0.044715 * x ** 3)))


def rms_norm(x, w, eps):
    """Rows of x over their root mean square (eps under the root), times the gain."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * w


def linear(x, w):
    return x @ w.T


def causal_conv(h, w):
    """Per-channel causal convolution over time. h [T, C], w [C, taps]; the last tap meets the current row."""
    taps = w.shape[1]
    out = np.zeros_like(h)
    for j in range(taps):
        lag = taps - 1 - j
        if lag < len(h):
            out[lag:] += w[:, j] * h[:len(h) - lag]
    return out


def rotate_interleaved(x, positions, base, dims):
    """Rotary positions on the first ``dims`` entries of the last axis, neighbours (2i, 2i + 1) paired.
    x [T, ..., D]."""
    x = x.copy()
    for i in range(dims // 2):
        ang = positions * base ** (-2.0 * i / dims)
        ang = ang.reshape((-1,) + (1,) * (x.ndim - 2))
        c, s = np.cos(ang), np.sin(ang)
        u, v = x[..., 2 * i].copy(), x[..., 2 * i + 1].copy()
        x[..., 2 * i] = u * c - v * s
        x[..., 2 * i + 1] = v * c + u * s
    return x


def window_mask(T, size):
    """mask[i, j]: position i sees position j, itself and the size - 1 before it (size None: all before it)."""
    d = np.arange(T)[:, None] - np.arange(T)[None, :]
    return (d >= 0) & ((d < size) if size is not None else True)


def softmax_masked(scores, mask):
    s = np.where(mask, scores, -np.inf)
    e = np.exp(s - s.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def min_gru_gates(h, w):
    """Update gate and candidate of every row: both read the current row only."""
    z = sigmoid(linear(h, w["z"]) + w["z.b"])
    u = linear(h, w["x"]) + w["x.b"]
    return z, np.where(u >= 0, u + 0.5, sigmoid(u))


def min_gru_scan(z, cand, start=None):
    s = np.zeros(z.shape[1], z.dtype) if start is None else start
    out = np.empty_like(z)
    for t in range(len(z)):
        s = (1.0 - z[t]) * s + z[t] * cand[t]
        out[t] = s
    return out


def min_gru(h, w, m):
    z, cand = min_gru_gates(h, w)
    return linear(min_gru_scan(z, cand) * silu(linear(h, w["g"])), w["o"])


def latent_attention(h, w, m, eps):
    T, H, D, R, V, C = len(h), m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = np.arange(T)
    rot = m["rot"]
    q = linear(h, w["q"]).reshape(T, H, D + R)
    q_rot = rotate_interleaved(q[:, :, D:], pos, rot["base"], rot["dims"])
    dkv = linear(h, w["dkv"])
    c = rms_norm(dkv[:, :C], w["dkv.norm"], eps)
    k_rot = rotate_interleaved(dkv[:, C:], pos, rot["base"], rot["dims"])
    k = linear(c, w["uk"]).reshape(T, H, D)
    v = linear(c, w["uv"]).reshape(T, H, V)
    mask = window_mask(T, (m.get("mask") or {}).get("size"))
    out = np.empty((T, H, V), h.dtype)
    for a in range(H):
        scores = (q[:, a, :D] @ k[:, a].T + q_rot[:, a] @ k_rot.T) * m["scale"]
        out[:, a] = softmax_masked(scores, mask) @ v[:, a]
    return linear(out.reshape(T, H * V) * sigmoid(linear(h, w["g"])), w["o"])


def dense_mlp(h, w):
    return linear(gelu_tanh(linear(h, w["up"])), w["down"])


def _sub(weights, prefix, dtype):
    return {k[len(prefix):]: np.asarray(v, dtype) for k, v in weights.items() if k.startswith(prefix)}


def layer(x, i, config, weights):
    """x plus mixer and feed-forward, which read the same norm through a convolution each."""
    spec, eps, dt = config["layers"][i], config["norm"]["eps"], x.dtype
    w = _sub(weights, f"l{i}.", dt)
    h = rms_norm(x, w["norm1"], eps)
    hm = h + causal_conv(h, w["canon1"])
    mix = _sub(w, "mix.", dt)
    if spec["type"] == "mingru":
        out = min_gru(hm, mix, spec["mixer"])
    elif spec["type"] == "latent_attention":
        out = latent_attention(hm, mix, spec["mixer"], eps)
    else:
        raise ValueError(spec["type"])
    if spec["mlp"] is not None:
        out = out + dense_mlp(h + causal_conv(h, w["canon2"]), _sub(w, "mlp.", dt))
    return x + out


def forward(tokens, config, weights, dtype=np.float64, keep_layers=False):
    """Logits of every position [T, vocab] (and the residual stream after every layer)."""
    embed = np.asarray(weights["embed"], dtype)
    x = embed[np.asarray(tokens)]
    streams = []
    for i in range(len(config["layers"])):
        x = layer(x, i, config, weights)
        streams.append(x)
    logits = linear(rms_norm(x, np.asarray(weights["final.norm"], dtype), config["norm"]["eps"]), embed)
    return (logits, streams) if keep_layers else logits
