"""Plain, slow restatement of the Zulozen decoder in numpy (test infrastructure only).

One function per mechanism, float64 throughout unless a caller passes another dtype. As in ``oracle/metapel.py``, a
sequence is always computed whole, from its first token: no cache, no batch, no sorting of tokens by expert.
``config`` is the dictionary of a ``config.json``; ``weights`` maps tensor names to arrays.
"""
from __future__ import annotations

import numpy as np

from .metapel import _sub, linear, rms_norm, rotate_interleaved, sigmoid, silu


def chunk_mask(T, size):
    """mask[i, j]: position i sees position j, itself or before it, of the same chunk of ``size`` positions counted
    from the sequence's start (size None: everything before it)."""
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    return (j <= i) & ((i // size == j // size) if size is not None else True)


def softmax_with_sink(scores, mask, sink):
    """Weights over the visible keys; the denominator also holds exp(sink)."""
    s = np.where(mask, scores, -np.inf)
    top = np.maximum(s.max(axis=-1, keepdims=True), sink)
    e = np.exp(s - top)
    return e / (e.sum(axis=-1, keepdims=True) + np.exp(sink - top))


def attention(h, w, m, eps):
    T, H, G, D, V = len(h), m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos, rot = np.arange(T), m["rot"]
    # one norm over all heads together, then the heads are cut and rotated
    q = rms_norm(linear(h, w["q"]), w["q.norm"], eps).reshape(T, H, D)
    k = rms_norm(linear(h, w["k"]), w["k.norm"], eps).reshape(T, G, D)
    q, k = (rotate_interleaved(x, pos, rot["base"], rot["dims"]) for x in (q, k))
    v = linear(h, w["v"]).reshape(T, G, V)
    gate = sigmoid(linear(h, w["g"]))
    mask = chunk_mask(T, (m.get("mask") or {}).get("size"))
    out = np.empty((T, H, V), h.dtype)
    for a in range(H):
        b = a // (H // G)
        p = softmax_with_sink(q[:, a] @ k[:, b].T * m["scale"], mask, w["sink"][a])
        out[:, a] = gate[:, a:a + 1] * (p @ v[:, b])
    return linear(out.reshape(T, H * V), w["o"])


def dense_relu2(h, w):
    return linear(np.maximum(linear(h, w["up"]) + w["up.b"], 0.0) ** 2, w["down"]) + w["down.b"]


def expert(h, w, name):
    return linear(silu(linear(h, w[name + ".gate"])) * linear(h, w[name + ".up"]), w[name + ".down"])


def route(h, router, top):
    """The chosen experts of every row, best first, and their scores."""
    s = sigmoid(linear(h, router))
    chosen = np.argsort(-s, axis=-1, kind="stable")[:, :top]
    return chosen, np.take_along_axis(s, chosen, axis=-1)


def mixture(h, w, mlp):
    """Every row through its experts, which read the row times its score, and through the shared expert."""
    chosen, score = route(h, w["router"], mlp["router"]["top"])
    out = expert(h, w, "shared") if mlp.get("shared") else np.zeros_like(h)
    for t in range(len(h)):
        for e, s in zip(chosen[t], score[t]):
            out[t] += expert(s * h[t:t + 1], w, f"e{e}")[0]
    return out


def layer(x, i, config, weights):
    """Two sublayers, each between a norm of its input and a norm of its output."""
    spec, eps, mult = config["layers"][i], config["norm"]["eps"], config["residual_mult"]
    w = _sub(weights, f"l{i}.", x.dtype)
    if spec["type"] != "attention":
        raise ValueError(spec["type"])
    y = attention(rms_norm(x, w["norm1"], eps), _sub(w, "mix.", x.dtype), spec["mixer"], eps)
    x = x + mult * rms_norm(y, w["norm1b"], eps)
    if spec["mlp"] is not None:
        h, mlp = rms_norm(x, w["norm2"], eps), _sub(w, "mlp.", x.dtype)
        y = dense_relu2(h, mlp) if spec["mlp"]["kind"] == "dense" else mixture(h, mlp, spec["mlp"])
        x = x + mult * rms_norm(y, w["norm2b"], eps)
    return x


def forward(tokens, config, weights, dtype=np.float64, keep_layers=False):
    """Logits of every position [T, vocab] (and the residual stream after every layer)."""
    x = np.asarray(weights["embed"], dtype)[np.asarray(tokens)]
    streams = []
    for i in range(len(config["layers"])):
        x = layer(x, i, config, weights)
        streams.append(x)
    logits = linear(rms_norm(x, np.asarray(weights["final.norm"], dtype), config["norm"]["eps"]), np.asarray(weights["head"], dtype))
    return (logits, streams) if keep_layers else logits
