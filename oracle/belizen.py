"""Plain, slow restatement of the Belizen decoder in numpy (test infrastructure only).

One function per mechanism, float64 throughout unless a caller passes another dtype. As in ``oracle/metapel.py``, a
sequence is always computed whole, from its first token: no cache, no state slots, no chunks, no sorting of tokens by expert.
``config`` is the dictionary of a ``config.json``; ``weights`` maps tensor names to arrays.
"""
from __future__ import annotations

import numpy as np

from .metapel import _sub, gelu_tanh, linear, rms_norm, sigmoid, silu, softmax_masked


def softcap(x, cap):
    return x if not cap else cap * np.tanh(x / cap)


def layer_runs(config):
    """(layer, pass) in the order in which they run; the pass is None outside the loop."""
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    return ([(i, None) for i in range(a)] + [(i, t) for t in range(loop["times"]) for i in range(a, b)] + [(i, None) for i in range(b, n)])


# ---- attention -------------------------------------------------------------------------------------

def kept_window_mask(T, size, keep):
    """mask[i, j]: position i sees itself, the size - 1 positions before it and the first ``keep`` positions."""
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    return (j <= i) & (((i - j < size) | (j < keep)) if size is not None else True)


def yarn_frequencies(rot):
    """Angle per position of every rotated pair, and the factor on cosine and sine."""
    dims, base, s = rot["dims"], rot["base"], rot.get("scaling")
    f = base ** (-2.0 * np.arange(dims // 2) / dims)
    if not s:
        return f, 1.0

    def dim_of(turns):  # the dimension that makes this many turns within the original length
        return dims * np.log(s["original"] / (2 * np.pi * turns)) / (2 * np.log(base))

    lo, hi = max(np.floor(dim_of(s["fast"])), 0), min(np.ceil(dim_of(s["slow"])), dims - 1)
    ramp = np.clip((np.arange(dims // 2) - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / s["factor"] * ramp + f * (1.0 - ramp), 0.1 * np.log(s["factor"]) + 1.0


def rotate_halves(x, positions, freq, mult):
    """x [T, heads, D]: entry i turned together with entry i + len(freq), the entries beyond left alone."""
    n = len(freq)
    ang = positions[:, None, None] * freq
    c, s = np.cos(ang) * mult, np.sin(ang) * mult
    u, v = x[..., :n], x[..., n:2 * n]
    return np.concatenate([u * c - v * s, v * c + u * s, x[..., 2 * n:]], axis=-1)


def attention(h, w, m, eps):
    T, H, G, D, V = len(h), m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (linear(h, w["q"]) + w["q.b"]).reshape(T, H, D)
    k = (linear(h, w["k"]) + w["k.b"]).reshape(T, G, D)
    v = (linear(h, w["v"]) + w["v.b"]).reshape(T, G, V)
    freq, mult = yarn_frequencies(m["rot"])
    q, k = (rotate_halves(rms_norm(x, w[n], eps), np.arange(T), freq, mult) for x, n in ((q, "q.norm"), (k, "k.norm")))
    mask = m.get("mask") or {}
    mask = kept_window_mask(T, mask.get("size"), mask.get("keep_first", 0))
    out = np.empty((T, H, V), h.dtype)
    for a in range(H):
        b = a // (H // G)
        out[:, a] = softmax_masked(softcap(q[:, a] @ k[:, b].T * m["scale"], m.get("softcap")), mask) @ v[:, b]
    return linear(out.reshape(T, H * V) * sigmoid(linear(h, w["g"])), w["o"])


# ---- gated linear attention --------------------------------------------------------------------------

def decays(h, w, tau):
    """Factor per key channel and row."""
    return sigmoid(linear(linear(h, w["a1"]), w["a2"]) + w["a2.b"]) ** (1.0 / tau)


def gla_scan(q, k, v, alpha):
    """q, k, alpha [T, dim], v [T, vdim] of one head: the state's rows decay, the new pair is added, the query reads it."""
    S, out = np.zeros((k.shape[1], v.shape[1]), k.dtype), np.empty_like(v)
    for t in range(len(q)):
        S = alpha[t][:, None] * S + np.outer(k[t], v[t])
        out[t] = S.T @ q[t]
    return out


def gla(h, w, m, eps):
    T, H, D, V = len(h), m["heads"], m["dim"], m["vdim"]
    q = (linear(h, w["q"]) * D ** -0.5).reshape(T, H, D)
    k, v = linear(h, w["k"]).reshape(T, H, D), linear(h, w["v"]).reshape(T, H, V)
    alpha = decays(h, w, m["tau"]).reshape(T, H, D)
    out = np.stack([gla_scan(q[:, a], k[:, a], v[:, a], alpha[:, a]) for a in range(H)], axis=1)
    return linear(rms_norm(out, w["norm"], eps).reshape(T, H * V) * silu(linear(h, w["g"])), w["o"])


# ---- feed-forward ---------------------------------------------------------------------------------------

def dense_geglu(h, w):
    return linear(gelu_tanh(linear(h, w["gate"])) * linear(h, w["up"]), w["down"])


def clamped_expert(h, w, name, limit):
    g = np.minimum(linear(h, w[name + ".gate"]), limit)
    u = np.clip(linear(h, w[name + ".up"]), -limit, limit)
    return linear(g * sigmoid(1.702 * g) * (u + 1.0), w[name + ".down"])


def route(h, w, top):
    """The chosen outputs of the router and their weights: the correction takes part in the choice only."""
    z = linear(h, w["router"])
    e = np.exp(z - z.max(axis=-1, keepdims=True))
    s = e / e.sum(axis=-1, keepdims=True)
    chosen = np.argsort(-(s + w["correction"]), axis=-1, kind="stable")[:, :top]
    return chosen, np.take_along_axis(s, chosen, axis=-1)


def mixture(h, w, mlp):
    """The weighted sum of a row's experts (those past the last one return the row itself) plus the shared expert."""
    n, limit, shared = mlp["router"]["experts"], mlp["expert"]["limit"], mlp.get("shared")
    chosen, weight = route(h, w, mlp["router"]["top"])
    out = clamped_expert(h, w, "shared", shared["limit"]) if shared else np.zeros_like(h)
    for t in range(len(h)):
        for e, s in zip(chosen[t], weight[t]):
            out[t] += s * (clamped_expert(h[t:t + 1], w, f"e{e}", limit)[0] if e < n else h[t])
    return out


# ---- the model --------------------------------------------------------------------------------------------

def layer(x, i, config, weights):
    spec, eps, mult = config["layers"][i], config["norm"]["eps"], config["residual_mult"]
    w = _sub(weights, f"l{i}.", x.dtype)
    x = x + mult * {"attention": attention, "gla": gla}[spec["type"]](rms_norm(x, w["norm1"], eps), _sub(w, "mix.", x.dtype), spec["mixer"], eps)
    if spec["mlp"] is not None:
        h, mlp = rms_norm(x, w["norm2"], eps), _sub(w, "mlp.", x.dtype)
        x = x + mult * (dense_geglu(h, mlp) if spec["mlp"]["kind"] == "dense" else mixture(h, mlp, spec["mlp"]))
    return x


def before_pass(x, start, t, step):
    """What joins the stream ahead of pass t: what the layers started from (not the first time), and the pass's own vector."""
    return x + (start if t > 0 else 0.0) + step[t]


def forward(tokens, config, weights, dtype=np.float64, keep_layers=False):
    """Logits of every position [T, vocab] (and the residual stream after every layer run)."""
    embed = np.asarray(weights["embed"], dtype)
    start = x = embed[np.asarray(tokens)] * config["embedding"]["scale"]
    streams = []
    for i, t in layer_runs(config):
        if t is not None and i == config["loop"]["start"]:
            x = before_pass(x, start, t, np.asarray(weights["loop.step"], dtype))
        x = layer(x, i, config, weights)
        streams.append(x)
    logits = linear(rms_norm(x, np.asarray(weights["final.norm"], dtype), config["norm"]["eps"]), embed)
    logits = softcap(logits, config.get("logit_softcap"))
    return (logits, streams) if keep_layers else logits
