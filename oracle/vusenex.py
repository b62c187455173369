"""Plain, slow restatement of the Vusenex decoder in numpy (test infrastructure only).

One function per mechanism, float64 throughout unless a caller passes another dtype. As in ``oracle/metapel.py``, a
sequence is always computed whole, from its first token: no cache, no batch, no sorting of tokens by expert.
``config`` is the dictionary of a ``config.json``; ``weights`` maps tensor names to arrays.
"""
from __future__ import annotations

import math

import numpy as np

from .metapel import _sub, linear, rms_norm, sigmoid, softmax_masked

ERF = np.vectorize(math.erf, otypes=[np.float64])


def gelu(x):
    """The exact form: x times the normal distribution function."""
    return (0.5 * x * (1.0 + ERF(x / math.sqrt(2.0)))).astype(x.dtype)


# ---- embedding ---------------------------------------------------------------------------------------

def bigram_rows(tokens, bigram):
    """Row of the bigram table for every token: hashed from it and its predecessor; the last row for the first token."""
    n = bigram["buckets"]
    return [n if i == 0 else (tokens[i - 1] * bigram["mul_prev"] + t * bigram["mul_cur"]) % n for i, t in enumerate(tokens)]


def embedding(tokens, config, weights, dtype):
    tokens = [int(t) for t in tokens]
    table, pairs, places = (np.asarray(weights[n], dtype) for n in ("embed", "bigram", "pos"))
    return table[tokens] + pairs[bigram_rows(tokens, config["embedding"]["bigram"])] + places[:len(tokens)]


# ---- attention -----------------------------------------------------------------------------------------

def query_factor(T, temp):
    """Factor of the query at every position: grows by steps with the logarithm of the position."""
    if not temp:
        return np.ones(T)
    return 1.0 + temp["coef"] * np.log(np.floor((np.arange(T) + 1) / temp["every"]) + 1.0)


def distance_bias(T, r1, r2):
    """What is taken off the score of position i for position j; only j <= i is ever looked at."""
    d = np.maximum(np.arange(T)[:, None] - np.arange(T)[None, :], 0)
    return r1 * np.log(1.0 + r2 * d)


def softmax_plus_one(scores, mask):
    """Weights over the visible keys; the denominator also holds one."""
    s = np.where(mask, scores, -np.inf)
    top = np.maximum(s.max(axis=-1, keepdims=True), 0.0)
    e = np.exp(s - top)
    return e / (e.sum(axis=-1, keepdims=True) + np.exp(-top))


def causal(T):
    return np.tril(np.ones((T, T), bool))


def attention(h, w, m, eps):
    T, H, G, D = len(h), m["heads"], m["kv_heads"], m["dim"]
    q, k = linear(h, w["q"]) + w["q.b"], linear(h, w["k"]) + w["k.b"]
    v = k.reshape(T, G, D)  # the values: the keys before their norm
    q = rms_norm(q, w["q.norm"], eps).reshape(T, H, D) * query_factor(T, m.get("q_temp"))[:, None, None]
    k = rms_norm(k, w["k.norm"], eps).reshape(T, G, D)
    out = np.empty((T, H, D), h.dtype)
    for a in range(H):
        b = a // (H // G)
        s = q[:, a] @ k[:, b].T * m["scale"] - distance_bias(T, w["r1"][a], w["r2"][a])
        out[:, a] = softmax_plus_one(s, causal(T)) @ v[:, b]
    return linear(out.reshape(T, H * D), w["o"])


def latent_attention(h, w, m, eps):
    T, H, D, V = len(h), m["heads"], m["dim"], m["vdim"]
    q = linear(h, w["q"]).reshape(T, H, D)
    c = rms_norm(linear(h, w["dkv"]), w["dkv.norm"], eps)
    k, v = linear(c, w["uk"]).reshape(T, H, D), linear(c, w["uv"]).reshape(T, H, V)
    out = np.empty((T, H, V), h.dtype)
    for a in range(H):
        out[:, a] = softmax_masked(q[:, a] @ k[:, a].T * m["scale"], causal(T)) @ v[:, a]
    return linear(out.reshape(T, H * V), w["o"])


# ---- feed-forward --------------------------------------------------------------------------------------

def expert(h, w, name):
    return linear(gelu(linear(h, w[name + ".up"])), w[name + ".down"])


def eligible(s, groups):
    """Which experts may be chosen: those of the ``keep`` groups whose largest scores are largest."""
    if not groups:
        return np.ones(s.shape, bool)
    best = s.reshape(len(s), groups["count"], -1).max(axis=-1)
    kept = np.zeros(best.shape, bool)
    np.put_along_axis(kept, np.argsort(-best, axis=-1, kind="stable")[:, :groups["keep"]], True, axis=-1)
    return np.repeat(kept, s.shape[1] // groups["count"], axis=1)


def route(h, matrix, router):
    """The chosen experts of every row, best first, and their weights, which add up to one."""
    z = linear(h, matrix)
    e = np.exp(z - z.max(axis=-1, keepdims=True))
    s = e / e.sum(axis=-1, keepdims=True)
    chosen = np.argsort(-np.where(eligible(s, router.get("groups")), s, -np.inf), axis=-1, kind="stable")[:, :router["top"]]
    weight = np.take_along_axis(s, chosen, axis=-1)
    return chosen, weight / (weight.sum(axis=-1, keepdims=True) + 1e-20)


def mixture(h, w, mlp):
    """The weighted sum of a row's experts plus the shared expert."""
    chosen, weight = route(h, w["router"], mlp["router"])
    out = expert(h, w, "shared") if mlp.get("shared") else np.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        rows, place = np.nonzero(chosen == e)
        if len(rows):
            out[rows] += weight[rows, place][:, None] * expert(h[rows], w, f"e{e}")
    return out


# ---- the model -------------------------------------------------------------------------------------------

def gated(y, h, matrix, bias):
    """A sublayer's result, every element times a gate formed from what the sublayer read."""
    return y * sigmoid(linear(h, matrix) + bias)


def layer(x, i, config, weights):
    """Two sublayers that read the stream itself; their gated results are normalised and added."""
    spec, eps = config["layers"][i], config["norm"]["eps"]
    w = _sub(weights, f"l{i}.", x.dtype)
    mixer = {"attention": attention, "latent_attention": latent_attention}[spec["type"]]
    x = x + rms_norm(gated(mixer(x, _sub(w, "mix.", x.dtype), spec["mixer"], eps), x, w["rg1"], w["rg1.b"]), w["norm1"], eps)
    if spec["mlp"] is not None:
        y = mixture(x, _sub(w, "mlp.", x.dtype), spec["mlp"])
        x = x + rms_norm(gated(y, x, w["rg2"], w["rg2.b"]), w["norm2"], eps)
    return x


def forward(tokens, config, weights, dtype=np.float64, keep_layers=False):
    """Logits of every position [T, vocab] (and the residual stream after every layer)."""
    x = embedding(tokens, config, weights, dtype)
    streams = []
    for i in range(len(config["layers"])):
        x = layer(x, i, config, weights)
        streams.append(x)
    logits = linear(rms_norm(x, np.asarray(weights["final.norm"], dtype), config["norm"]["eps"]), np.asarray(weights["head"], dtype))
    return (logits, streams) if keep_layers else logits
