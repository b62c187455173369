"""Small Zulozen configurations with random weights for the tests (the harness that feeds a device model is in
``metapel_models``)."""
import numpy as np

from oracle import binding


def attn(heads, kv_heads, dim, vdim, chunk, mlp=None, base=10000.0, scale=None, rot_dims=None):
    return {"type": "attention",
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": chunk} if chunk else None,
                      "rot": {"base": base, "dims": dim // 2 // 2 * 2 if rot_dims is None else rot_dims},
                      "scale": dim ** -0.5 if scale is None else scale},
            "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, shared=None):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}, "shared": {"ff": shared} if shared else None}


def config(width, vocab, layers, eps=1e-5, mult=0.4):
    return {"architecture": "Zulozen", "width": width, "vocab": vocab, "norm": {"eps": eps}, "residual_mult": mult, "layers": layers}


def tensor_shapes(cfg):
    H = cfg["width"]
    t = {"embed": (cfg["vocab"], H), "final.norm": (H,), "head": (cfg["vocab"], H)}
    for i, e in enumerate(cfg["layers"]):
        m, p, mlp = e["mixer"], f"l{i}.", e["mlp"]
        q, k, v = m["heads"] * m["dim"], m["kv_heads"] * m["dim"], m["kv_heads"] * m["vdim"]
        t[p + "norm1"] = t[p + "norm1b"] = (H,)
        t[p + "mix.q"], t[p + "mix.k"], t[p + "mix.v"] = (q, H), (k, H), (v, H)
        t[p + "mix.q.norm"], t[p + "mix.k.norm"], t[p + "mix.sink"] = (q,), (k,), (m["heads"],)
        t[p + "mix.g"], t[p + "mix.o"] = (m["heads"], H), (H, m["heads"] * m["vdim"])
        if mlp is None:
            continue
        t[p + "norm2"] = t[p + "norm2b"] = (H,)
        if mlp["kind"] == "dense":
            t[p + "mlp.up"], t[p + "mlp.up.b"] = (mlp["ff"], H), (mlp["ff"],)
            t[p + "mlp.down"], t[p + "mlp.down.b"] = (H, mlp["ff"]), (H,)
            continue
        t[p + "mlp.router"] = (mlp["router"]["experts"], H)
        parts = [(f"e{j}", mlp["expert"]["ff"]) for j in range(mlp["router"]["experts"])]
        for name, ff in parts + ([("shared", mlp["shared"]["ff"])] if mlp["shared"] else []):
            t[f"{p}mlp.{name}.gate"] = t[f"{p}mlp.{name}.up"] = (ff, H)
            t[f"{p}mlp.{name}.down"] = (H, ff)
    return t


def bf16(x):
    return binding.round_to_bf16(np.ascontiguousarray(x, np.float32))


def random_weights(cfg, seed=0, gain=1.5, decisive=True):
    """Matrices of gain / sqrt(inputs), gains around one, biases and sinks of visible size; bf16 values. ``decisive``: routers
    whose choices, different from token to token, are far from a close call, so that rounding does not change an expert."""
    rng = np.random.default_rng(seed)
    w = {}
    for name, shape in tensor_shapes(cfg).items():
        x = rng.standard_normal(shape)
        if ".norm" in name or name == "final.norm":
            x = 1.0 + 0.2 * x
        elif name.endswith(".b"):
            x = 2.0 * x
        elif name.endswith(".sink"):
            x = 1.0 + 1.5 * x
        elif name == "embed":
            x = 3.0 * x
        else:
            x = gain * x / np.sqrt(shape[1])
        w[name] = bf16(x)
    if decisive:
        h = w["embed"].astype(np.float64)
        h /= np.sqrt((h ** 2).mean(axis=1, keepdims=True))
        for i, e in enumerate(cfg["layers"]):
            if e["mlp"] is None or e["mlp"]["kind"] != "moe":
                continue
            n, top = e["mlp"]["router"]["experts"], e["mlp"]["router"]["top"]
            logits = np.full((cfg["vocab"], n), -2.2)
            for row in logits:
                row[rng.permutation(n)[:top]] = rng.uniform(0.2, 1.4, top)
            w[f"l{i}.mlp.router"] = bf16((np.linalg.pinv(h) @ logits).T / w[f"l{i}.norm2"])
    return w


# Sizes that no single kernel variant covers together: widths that are no multiple of 4 or 8, odd head counts and sizes, chunks
# of a few tokens, keys rotated in part, wholly or not at all, layers without a feed-forward, experts of odd width.
ODD = config(50, 24, [attn(3, 1, 10, 7, 5, dense(26), rot_dims=4), attn(4, 2, 6, 9, 11, moe(5, 2, 13, 9), rot_dims=6), attn(1, 1, 4, 5, 1),
                      attn(6, 3, 8, 3, 64, moe(3, 3, 7), rot_dims=0)], mult=0.25)
# Heads that pad to 64, more than eight query heads to a key head, many experts, no shared expert.
TUNED = config(128, 30, [attn(4, 2, 32, 48, 40, dense(192), base=500.0), attn(11, 1, 64, 16, 70, moe(40, 4, 64, 72), rot_dims=64),
                         attn(2, 2, 64, 64, 100, moe(8, 3, 128), scale=0.3)], eps=1e-3, mult=0.6)
# Heads that pad to 128 in keys, values or both; every token seen; one expert of all.
WIDE = config(192, 100, [attn(9, 3, 128, 64, None, dense(512), base=50000.0), attn(20, 2, 64, 128, 150, moe(6, 1, 192, 136)),
                         attn(3, 1, 80, 112, 33, moe(2, 2, 64, 64), rot_dims=14)], mult=0.8)
# Heads beyond 128.
BROAD = config(96, 50, [attn(2, 1, 144, 32, 90, dense(40), rot_dims=20), attn(2, 2, 24, 256, 60, moe(9, 2, 80, 64))])
CONFIGS = {"odd": ODD, "tuned": TUNED, "wide": WIDE, "broad": BROAD}
