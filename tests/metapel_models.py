"""Small Metapel configurations with random weights for the tests, and a harness that feeds token portions to a
device model through the framework's cache manager and state slots."""
import numpy as np

from oracle import binding


def mingru(width, ff=0):
    return {"type": "mingru", "mixer": {"width": width}, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def latent(heads, dim, rot, vdim, rank, window, ff=0, base=10000.0, scale=None, rot_dims=None):
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "mask": {"size": window},
                      "rot": {"base": base, "dims": rot if rot_dims is None else rot_dims},
                      "scale": (dim + rot) ** -0.5 if scale is None else scale},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(width, vocab, layers, taps=4, eps=1e-5):
    return {"architecture": "Metapel", "width": width, "vocab": vocab, "norm": {"eps": eps}, "canon": {"taps": taps}, "layers": layers}


def tensor_shapes(cfg):
    H = cfg["width"]
    t = {"embed": (cfg["vocab"], H), "final.norm": (H,)}
    for i, e in enumerate(cfg["layers"]):
        m, p = e["mixer"], f"l{i}."
        t[p + "norm1"] = (H,)
        t[p + "canon1"] = (H, cfg["canon"]["taps"])
        if e["type"] == "mingru":
            W = m["width"]
            for n in "zxg":
                t[f"{p}mix.{n}"] = (W, H)
            t[p + "mix.z.b"], t[p + "mix.x.b"], t[p + "mix.o"] = (W,), (W,), (H, W)
        else:
            h, r = m["heads"], m["kv_rank"]
            t[p + "mix.q"] = (h * (m["dim"] + m["rot_dim"]), H)
            t[p + "mix.dkv"], t[p + "mix.dkv.norm"] = (r + m["rot_dim"], H), (r,)
            t[p + "mix.uk"], t[p + "mix.uv"] = (h * m["dim"], r), (h * m["vdim"], r)
            t[p + "mix.g"], t[p + "mix.o"] = (h * m["vdim"], H), (H, h * m["vdim"])
        if e["mlp"] is not None:
            t[p + "canon2"] = (H, cfg["canon"]["taps"])
            t[p + "mlp.up"], t[p + "mlp.down"] = (e["mlp"]["ff"], H), (H, e["mlp"]["ff"])
    return t


def random_weights(cfg, seed=0, gain=1.5):
    """Matrices of gain / sqrt(inputs), gains around one, biases and filters of visible size; bf16 values."""
    rng = np.random.default_rng(seed)
    w = {}
    for name, shape in tensor_shapes(cfg).items():
        x = rng.standard_normal(shape)
        if name.endswith("norm") or name.endswith("norm1"):
            x = 1.0 + 0.2 * x
        elif name.endswith(".b"):
            x = 0.7 * x
        elif ".canon" in name:
            x = 0.4 * x
        elif name != "embed":
            x = gain * x / np.sqrt(shape[1])
        w[name] = binding.round_to_bf16(x.astype(np.float32))
    return w


# Sizes that no single kernel variant covers together: widths that are no multiple of 4 or 8, odd head counts,
# one tap, a window of one token, partly rotated keys, layers without a feed-forward, unequal layers.
ODD = config(50, 61, [mingru(22, 30), latent(3, 10, 6, 7, 18, 5, 26, rot_dims=4), mingru(36), latent(1, 4, 2, 5, 9, 1, 12)], taps=3)
ONE_TAP = config(64, 96, [latent(2, 16, 16, 24, 32, 9, 64), mingru(48, 40)], taps=1, eps=1e-3)
TUNED = config(128, 192, [mingru(160, 192), latent(5, 32, 16, 48, 64, 40, 128), latent(12, 16, 32, 32, 96, 17, 0, base=500.0),
                          mingru(64, 320)], taps=4)
WIDE = config(256, 320, [latent(20, 64, 32, 64, 192, 150, 512, base=50000.0), mingru(384, 0),
                         latent(3, 48, 64, 80, 512, 77, 64, scale=0.05)], taps=5)
BROAD_VALUES = config(96, 128, [latent(2, 32, 0, 144, 128, 100, 64), latent(3, 80, 16, 256, 64, 30)], taps=2)
CONFIGS = {"broad_values": BROAD_VALUES, "odd": ODD, "one_tap": ONE_TAP, "tuned": TUNED, "wide": WIDE}


def make_model(pkg, backend, cfg, weights, dtype, blocks=64, tokens=1024, seqs=8):
    meta = pkg.LayeredMetadata.from_config(cfg, "test", {n: x.shape for n, x in weights.items()})
    return pkg.CudaLayeredModel.new(meta, weights, blocks, 16, backend, compute_dtype=dtype, max_batch_tokens=tokens,
                                    max_batch_sequences=seqs)


class Feeder:
    """Live sequences of a model. ``step`` runs one batch of portions and collects the logits of every row."""

    def __init__(self, pkg, model):
        from orionserve_rs_b200.trace import TraceRunner

        self.runner, self.logits = TraceRunner(model), {}

    def step(self, portions, end=()):
        entries = [{"id": n, "tokens": [int(x) for x in t], "want": list(range(len(t)))} for n, t in portions]
        out = self.runner.step(entries, end)
        at = 0
        for n, t in portions:
            self.logits.setdefault(n, []).append(out[at:at + len(t)])
            at += len(t)

    def run(self, name, tokens, sizes):
        """Feeds one sequence in portions of these sizes (the last one repeated), alone, and ends it."""
        at, k = 0, 0
        while at < len(tokens):
            n = sizes[min(k, len(sizes) - 1)]
            self.step([(name, tokens[at:at + n])], [name] if at + n >= len(tokens) else [])
            at, k = at + n, k + 1
        return self.all(name)

    def all(self, name):
        return np.concatenate(self.logits[name])


def worst_error(got, exp):
    """Largest over the rows of: rms of the difference (mean taken off) over the rms of all expected logits."""
    d = got.astype(np.float64) - exp
    d -= d.mean(axis=1, keepdims=True)
    return float(np.sqrt((d ** 2).mean(axis=1)).max() / np.sqrt((exp ** 2).mean()))
