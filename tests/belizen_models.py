"""Small Belizen configurations with random weights for the tests (the harness that feeds a device model is in
``metapel_models``)."""
import numpy as np

from oracle import binding


def gla(heads, dim, vdim, tau, rank, mlp=None):
    """``rank`` is a size that no configuration gives; it stands in the list of tensors only."""
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}, "mlp": mlp, "rank": rank}


def attn(heads, kv_heads, dim, vdim, window, keep=0, mlp=None, base=10000.0, scale=None, rot_dims=None, yarn=None, cap=20.0):
    return {"type": "attention",
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "softcap": cap,
                      "mask": {"size": window, "keep_first": keep} if window else None,
                      "rot": {"base": base, "dims": dim // 4 * 2 if rot_dims is None else rot_dims, "scaling": yarn},
                      "scale": dim ** -0.5 if scale is None else scale},
            "mlp": mlp}


def yarn(factor, original, fast, slow):
    return {"factor": factor, "original": original, "fast": fast, "slow": slow}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, identity, top, ff, limit, shared=None, shared_limit=None):
    return {"kind": "moe", "router": {"experts": experts, "identity": identity, "top": top}, "expert": {"ff": ff, "limit": limit},
            "shared": {"ff": shared, "limit": shared_limit or limit} if shared else None}


def config(width, vocab, layers, eps=1e-5, mult=0.4, scale=2.0, loop=None, cap=30.0):
    return {"architecture": "Belizen", "width": width, "vocab": vocab, "norm": {"eps": eps}, "residual_mult": mult,
            "embedding": {"scale": scale}, "logit_softcap": cap, "loop": dict(zip(("start", "stop", "times"), loop)) if loop else None,
            "layers": layers}


def tensor_shapes(cfg):
    H = cfg["width"]
    t = {"embed": (cfg["vocab"], H), "final.norm": (H,)}
    if cfg["loop"]:
        t["loop.step"] = (cfg["loop"]["times"], H)
    for i, e in enumerate(cfg["layers"]):
        m, p, mlp = e["mixer"], f"l{i}.", e["mlp"]
        t[p + "norm1"] = (H,)
        if e["type"] == "gla":
            k, v, r = m["heads"] * m["dim"], m["heads"] * m["vdim"], e["rank"]
            t[p + "mix.q"], t[p + "mix.k"], t[p + "mix.v"], t[p + "mix.g"] = (k, H), (k, H), (v, H), (v, H)
            t[p + "mix.a1"], t[p + "mix.a2"], t[p + "mix.a2.b"] = (r, H), (k, r), (k,)
            t[p + "mix.norm"], t[p + "mix.o"] = (m["vdim"],), (H, v)
        else:
            q, k, v = m["heads"] * m["dim"], m["kv_heads"] * m["dim"], m["kv_heads"] * m["vdim"]
            for n, rows in (("q", q), ("k", k), ("v", v)):
                t[f"{p}mix.{n}"], t[f"{p}mix.{n}.b"] = (rows, H), (rows,)
            t[p + "mix.q.norm"] = t[p + "mix.k.norm"] = (m["dim"],)
            t[p + "mix.g"], t[p + "mix.o"] = (m["heads"] * m["vdim"], H), (H, m["heads"] * m["vdim"])
        if mlp is None:
            continue
        t[p + "norm2"] = (H,)
        if mlp["kind"] == "dense":
            t[p + "mlp.gate"] = t[p + "mlp.up"] = (mlp["ff"], H)
            t[p + "mlp.down"] = (H, mlp["ff"])
            continue
        n = mlp["router"]["experts"] + mlp["router"]["identity"]
        t[p + "mlp.router"], t[p + "mlp.correction"] = (n, H), (n,)
        parts = [(f"e{j}", mlp["expert"]["ff"]) for j in range(mlp["router"]["experts"])]
        for name, ff in parts + ([("shared", mlp["shared"]["ff"])] if mlp["shared"] else []):
            t[f"{p}mlp.{name}.gate"] = t[f"{p}mlp.{name}.up"] = (ff, H)
            t[f"{p}mlp.{name}.down"] = (H, ff)
    return t


def bf16(x):
    return binding.round_to_bf16(np.ascontiguousarray(x, np.float32))


PATTERNS = 12  # kinds of tokens that the decisive routers tell apart, by as many dimensions of the stream


def random_weights(cfg, seed=0, gain=1.5, decisive=True):
    """Matrices of gain / sqrt(inputs), gains around one, biases of visible size, decays from quick to slow; bf16 values.
    ``decisive``: routers read a few dimensions into which only the embedding writes, so that their choices, different from token to token
    and not always those of the largest scores, are far from a close call and rounding does not change an expert."""
    rng = np.random.default_rng(seed)
    w = {}
    for name, shape in tensor_shapes(cfg).items():
        x = rng.standard_normal(shape)
        if name.endswith("q.norm") or name.endswith("k.norm"):
            x = 1.6 + 0.3 * x
        elif ".norm" in name or name == "final.norm":
            x = 1.0 + 0.2 * x
        elif name.endswith(".a2.b"):
            x = 1.0 + 2.5 * x
        elif name.endswith(".b"):
            x = 0.7 * x
        elif name.endswith(".correction"):
            x = 0.25 * x
        elif name.endswith("loop.step"):
            x = 1.5 * x
        elif name.endswith(".o") or name.endswith(".down"):
            x = 2 * gain * x / np.sqrt(shape[1])
        elif name != "embed":
            x = gain * x / np.sqrt(shape[1])
        w[name] = bf16(x)
    if decisive:
        P, kind = PATTERNS, rng.permutation(cfg["vocab"]) % PATTERNS
        w["embed"][:, :P] = 3.0 * np.eye(P)[kind]
        for name in w:
            if name.endswith(".o") or name.endswith(".down"):
                w[name][:P] = 0.0
            elif name.endswith("loop.step"):
                w[name][:, :P] = 0.0
            elif name.endswith("norm2"):
                w[name][:P] = 1.0
            elif name.endswith("mlp.router"):
                i = int(name[1:name.index(".")])
                corr = w[f"l{i}.mlp.correction"].astype(np.float64)
                logits = [_clear_choice(rng, corr, cfg["layers"][i]["mlp"]["router"]["top"]) for _ in range(P)]
                w[name][:, P:] = 0.0
                w[name][:, :P] = bf16(np.stack(logits, axis=1) / 2.0)  # what the norm leaves of the embedding's 3
    return w


def _clear_choice(rng, correction, top):
    """Logits whose choice has a wide gap, in scores with the correction added, also when they come out smaller or larger."""
    n = len(correction)
    if top == n:
        return rng.standard_normal(n)
    best, at = None, -1.0
    for _ in range(200):
        z = rng.standard_normal(n) * 0.5 - 2.0
        z[rng.permutation(n)[:top]] = rng.uniform(0.5, 1.5, top)
        gap = 1.0
        for f in (0.7, 1.0, 1.4):
            s = np.exp(f * z) / np.exp(f * z).sum() + correction
            order = np.sort(s)
            gap = min(gap, order[-top] - order[-top - 1])
        if gap > at:
            best, at = z, gap
        if gap > 0.06 and rng.random() < 0.3:
            break
    return best


# Sizes that no single kernel variant covers together: widths that are no multiple of 4 or 8, odd head counts and sizes, windows of a
# few tokens, keys rotated in part, wholly or not at all, layers without a feed-forward, experts of odd width, a loop from the first layer.
ODD = config(50, 24, [gla(3, 5, 7, 2.0, 3, dense(26)), attn(3, 1, 10, 7, 5, 2, moe(5, 2, 2, 13, 0.8, 9, 1.1), rot_dims=4, yarn=yarn(3.0, 64, 8.0, 0.5)),
                      gla(1, 12, 6, 0.4, 5), attn(4, 2, 6, 9, 11, 0, moe(3, 1, 3, 7, 1.4), rot_dims=6, cap=3.0)], mult=0.25, loop=(0, 2, 3), cap=8.0)
# The chunked form of linear attention with heads padded to 16, attention heads that pad to 64, more than eight query heads to a key
# head, many experts, no shared expert, decays that are steep within a few rows.
TUNED = config(128, 30, [gla(2, 32, 48, 16.0, 16, moe(9, 3, 2, 64, 1.5, 72, 2.5)), attn(11, 1, 64, 16, 70, 20, dense(192), rot_dims=64, yarn=yarn(8.0, 128, 16.0, 1.0)),
                         gla(5, 20, 36, 0.3, 7, moe(20, 4, 3, 72, 0.9)), attn(4, 2, 32, 48, 40, 3, None, base=500.0), gla(1, 64, 16, 4.0, 8)],
               eps=1e-3, mult=0.3, loop=(1, 3, 2))
# Heads that pad to 128, every token seen, one expert per token, the last layers looped.
WIDE = config(192, 100, [attn(9, 3, 128, 64, None, 0, dense(512), base=50000.0, scale=0.05), gla(2, 128, 128, 16.0, 16, moe(6, 1, 1, 192, 1.7, 136)),
                         attn(8, 1, 80, 112, 33, 17, moe(4, 2, 2, 64, 0.7, 64), rot_dims=16, yarn=yarn(2.0, 32, 4.0, 1.0), cap=0.0)], mult=0.5, loop=(1, 3, 2), cap=0.0)
# Heads beyond 128, linear attention with key heads of 144 and 272 values, no loop.
BROAD = config(104, 50, [attn(2, 1, 144, 32, 90, 40, dense(40), rot_dims=20), gla(2, 144, 40, 8.0, 4, moe(2, 2, 2, 80, 2.0, 64)), gla(1, 272, 24, 16.0, 24),
                         attn(6, 2, 24, 256, 60, 1, moe(9, 0, 2, 80, 1.0))])
CONFIGS = {"odd": ODD, "tuned": TUNED, "wide": WIDE, "broad": BROAD}
