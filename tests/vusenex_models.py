"""Small Vusenex configurations with random weights for the tests (the harness that feeds a device model is in
``metapel_models``)."""
import numpy as np

from oracle import binding


def attn(heads, kv_heads, dim, mlp=None, temp=(0.4, 20), scale=None):
    return {"type": "attention",
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": dim ** -0.5 if scale is None else scale,
                      "q_temp": dict(zip(("coef", "every"), temp)) if temp else None},
            "mlp": mlp}


def latent(heads, dim, vdim, rank, mlp=None, scale=None):
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": rank, "scale": dim ** -0.5 if scale is None else scale}, "mlp": mlp}


def moe(experts, groups, keep, top, ff, shared=None):
    return {"kind": "moe", "router": {"experts": experts, "top": top, "groups": {"count": groups, "keep": keep} if groups else None},
            "expert": {"ff": ff}, "shared": {"ff": shared} if shared else None}


def config(width, vocab, layers, eps=1e-5, pairs=(37, 5, 11), positions=900):
    return {"architecture": "Vusenex", "width": width, "vocab": vocab, "norm": {"eps": eps}, "max_positions": positions,
            "embedding": {"bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), pairs))}, "layers": layers}


def tensor_shapes(cfg):
    H = cfg["width"]
    t = {"embed": (cfg["vocab"], H), "bigram": (cfg["embedding"]["bigram"]["buckets"] + 1, H), "pos": (cfg["max_positions"], H),
         "final.norm": (), "head": (cfg["vocab"], H)}
    for i, e in enumerate(cfg["layers"]):
        m, p, mlp = e["mixer"], f"l{i}.", e["mlp"]
        t[p + "norm1"], t[p + "rg1"], t[p + "rg1.b"] = (), (H, H), (H,)
        q = m["heads"] * m["dim"]
        t[p + "mix.q"], t[p + "mix.o"] = (q, H), (H, m["heads"] * m["vdim"])
        if e["type"] == "attention":
            k = m["kv_heads"] * m["dim"]
            t[p + "mix.k"], t[p + "mix.q.b"], t[p + "mix.k.b"], t[p + "mix.q.norm"], t[p + "mix.k.norm"] = (k, H), (q,), (k,), (q,), (k,)
            t[p + "mix.r1"] = t[p + "mix.r2"] = (m["heads"],)
        else:
            t[p + "mix.dkv"], t[p + "mix.dkv.norm"] = (m["kv_rank"], H), (m["kv_rank"],)
            t[p + "mix.uk"], t[p + "mix.uv"] = (q, m["kv_rank"]), (m["heads"] * m["vdim"], m["kv_rank"])
        if mlp is None:
            continue
        t[p + "norm2"], t[p + "rg2"], t[p + "rg2.b"], t[p + "mlp.router"] = (), (H, H), (H,), (mlp["router"]["experts"], H)
        parts = [(f"e{j}", mlp["expert"]["ff"]) for j in range(mlp["router"]["experts"])]
        for name, ff in parts + ([("shared", mlp["shared"]["ff"])] if mlp["shared"] else []):
            t[f"{p}mlp.{name}.up"], t[f"{p}mlp.{name}.down"] = (ff, H), (H, ff)
    return t


def bf16(x):
    x = np.asarray(x, np.float32)
    return binding.round_to_bf16(np.ascontiguousarray(x)).reshape(x.shape)


PATTERNS = 12  # kinds of tokens that the decisive routers tell apart, by as many dimensions of the stream


def random_weights(cfg, seed=0, gain=1.2, decisive=True):
    """Matrices of gain / sqrt(inputs), gains around one, biases of visible size, distance terms from flat to steep; bf16 values.
    ``decisive``: routers read a few dimensions into which only the embedding writes, so that their choices, different from token to token,
    are far from a close call and rounding does not change an expert."""
    rng = np.random.default_rng(seed)
    w = {}
    for name, shape in tensor_shapes(cfg).items():
        x = rng.standard_normal(shape)
        if name.endswith("q.norm") or name.endswith("k.norm"):
            x = 1.1 + 0.3 * x
        elif "norm" in name:
            x = 1.0 + 0.2 * x
        elif name.endswith(".r1"):
            x = 0.2 + np.abs(x)
        elif name.endswith(".r2"):
            x = 0.05 + 0.3 * np.abs(x)
        elif name.endswith(".b"):
            x = 0.7 * x
        elif name == "pos":
            x = 0.6 * x
        elif name not in ("embed", "bigram"):
            x = gain * x / np.sqrt(shape[-1])
        w[name] = bf16(x)
    if decisive:
        P, kind = PATTERNS, rng.permutation(cfg["vocab"]) % PATTERNS
        w["embed"][:, :P] = 3.0 * np.eye(P)[kind]
        w["bigram"][:, :P] = w["pos"][:, :P] = 0.0
        for name in w:
            if name.endswith(".o") or name.endswith(".down"):
                w[name][:P] = 0.0
            elif name.endswith("mlp.router"):
                router = cfg["layers"][int(name[1:name.index(".")])]["mlp"]["router"]
                w[name][:, P:] = 0.0
                w[name][:, :P] = bf16(np.stack([_clear_choice(rng, router) for _ in range(P)], axis=1) / 3.0)
    return w


def gaps(z, router):
    """How clear a choice is: the smallest difference of logits between what is taken and what is not, among groups and among experts."""
    n, top, groups = len(z), router["top"], router["groups"]
    gap, open_ = np.inf, np.ones(n, bool)
    if groups:
        best = np.sort(z.reshape(groups["count"], -1).max(axis=1))
        if groups["keep"] < groups["count"]:
            gap = best[-groups["keep"]] - best[-groups["keep"] - 1]
            open_ = np.repeat(z.reshape(groups["count"], -1).max(axis=1) >= best[-groups["keep"]], n // groups["count"])
    s = np.sort(z[open_])
    return min(gap, s[-top] - s[-top - 1]) if top < len(s) else gap


def _clear_choice(rng, router):
    best, at = None, -1.0
    for _ in range(400):
        z = rng.standard_normal(router["experts"]) * 1.2
        gap = gaps(z, router)
        if gap > at:
            best, at = z, gap
        if gap > 0.4:
            break
    return best


# Sizes that no single kernel variant covers together: widths that are no multiple of 4 or 8, odd head counts and sizes, one head, layers
# without a feed-forward or without a shared expert, experts of odd width, groups of one expert, no groups, one group.
ODD = config(50, 24, [latent(3, 5, 7, 10, moe(6, 3, 2, 3, 33, 29)), attn(3, 1, 10, moe(5, 5, 3, 2, 37), temp=(1.2, 7)), latent(2, 12, 7, 6, scale=0.1),
                      attn(4, 2, 7, moe(4, 1, 1, 4, 31, 26), temp=None), attn(1, 1, 9, moe(3, 0, 0, 1, 35, 43), temp=(0.35, 1), scale=0.15)], pairs=(23, 1, 1), positions=300)
# Attention heads that pad to 64, more than eight query heads to a key head, tuned latent sizes, many experts.
TUNED = config(128, 30, [attn(11, 1, 64, moe(8, 4, 2, 3, 64, 72)), latent(5, 32, 48, 64), attn(6, 3, 48, moe(20, 5, 3, 4, 72), temp=(0.9, 33)),
                         latent(12, 16, 32, 96, moe(9, 3, 1, 2, 136, 64))], eps=1e-3, pairs=(101, 1000003, 7919))
# Heads that pad to 128, long latents, one expert per token.
WIDE = config(192, 100, [attn(9, 3, 128, moe(6, 2, 1, 1, 192, 136), scale=0.05), latent(20, 64, 64, 192, moe(4, 2, 2, 2, 64, 64)), attn(8, 1, 80)],
              pairs=(500, 3, 17))
# Heads beyond 128, values unequal to keys, the longest latents that the tuned kernels take.
BROAD = config(104, 50, [attn(2, 1, 144, moe(12, 6, 2, 3, 80)), latent(2, 32, 144, 128, moe(2, 2, 1, 1, 80, 64)), attn(6, 2, 24),
                         latent(3, 80, 256, 512, scale=0.07)], pairs=(64, 31, 2))
CONFIGS = {"odd": ODD, "tuned": TUNED, "wide": WIDE, "broad": BROAD}
