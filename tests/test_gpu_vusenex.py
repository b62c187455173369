"""Vusenex on the device against the plain implementation in ``oracle/vusenex.py``: every mechanism alone, whole prompts,
portions, decoding, mixed batches, reuse of pages, far keys and keys at page borders, the first tokens, pairs of tokens across steps, and
generation through the engine. ``tol`` is the bar on the rms error of a row of logits over the rms of the logits: 3e-5 in the f32 build; 3e-2
in the bf16 build, whose weights are the same values and whose activations are rounded."""
import dataclasses
import json

import numpy as np
import pytest

from metapel_models import Feeder, make_model, worst_error
from oracle import vusenex
from vusenex_models import CONFIGS, attn, bf16, config, latent, moe, random_weights

pytestmark = pytest.mark.gpu
TOL = {"F32": 3e-5, "BF16": 3e-2}


@pytest.fixture(scope="module")
def backend(pkg):
    if not pkg.is_available():
        pytest.fail("no CUDA device: the model has no CPU fallback")
    return pkg.CudaBackend(0)


@pytest.fixture(params=["F32", "BF16"])
def dtype(request, pkg):
    return getattr(pkg.DType, request.param)


def tol(dtype):
    return TOL[dtype.name]


class Case:
    """One configuration: weights, expected logits of a few sequences."""
    cache = {}

    def __init__(self, name):
        self.cfg = CONFIGS[name]
        self.weights = random_weights(self.cfg, seed=len(name))
        rng = np.random.default_rng(17)
        self.tokens = {n: rng.integers(0, self.cfg["vocab"], size).tolist()
                       for n, size in (("a", 230), ("b", 97), ("c", 33), ("d", 1), ("e", 161))}
        self.expected = {n: vusenex.forward(t, self.cfg, self.weights) for n, t in self.tokens.items()}

    @classmethod
    def get(cls, name):
        if name not in cls.cache:
            cls.cache[name] = cls(name)
        return cls.cache[name]


@pytest.fixture(params=sorted(CONFIGS))
def case(request):
    return Case.get(request.param)


def test_whole_prompts(pkg, backend, case, dtype):
    f = Feeder(pkg, make_model(pkg, backend, case.cfg, case.weights, dtype))
    for n, t in case.tokens.items():
        assert worst_error(f.run(n, t, [len(t)]), case.expected[n]) < tol(dtype), n


def test_token_by_token_equals_the_prompt(pkg, backend, case, dtype):
    f = Feeder(pkg, make_model(pkg, backend, case.cfg, case.weights, dtype))
    assert worst_error(f.run("b", case.tokens["b"], [1]), case.expected["b"]) < tol(dtype)
    # long decoding after a prompt
    assert worst_error(f.run("a", case.tokens["a"], [50, 1]), case.expected["a"]) < tol(dtype)


@pytest.mark.parametrize("sizes", [[2], [3], [7], [8], [9], [16], [17], [64], [1, 2, 63, 5, 33, 1, 1, 12, 100], [15, 1, 1, 15, 9, 7, 16]])
def test_portions(pkg, backend, case, dtype, sizes):
    f = Feeder(pkg, make_model(pkg, backend, case.cfg, case.weights, dtype))
    assert worst_error(f.run("a", case.tokens["a"], sizes), case.expected["a"]) < tol(dtype)


def test_mixed_batches_and_reuse(pkg, backend, case, dtype):
    """Unequal requests in one batch, prompts beside single tokens, on a pool that just holds the live ones, so
    that pages are used again by later requests; the order of the entries changes too."""
    f = Feeder(pkg, make_model(pkg, backend, case.cfg, case.weights, dtype, blocks=42, seqs=3))
    rng = np.random.default_rng(5)
    waiting = ["a", "b", "c", "d", "e", "b2", "a2", "d2", "e2", "c2"]
    live, at = [], {}
    while waiting or live:
        while waiting and len(live) < 3:
            live.append(waiting.pop(0))
            at[live[-1]] = 0
        part, end = [], []
        for n in rng.permutation(live):
            if len(live) > 1 and rng.random() < 0.2:
                continue  # left out of this step
            t = case.tokens[n[0]]
            k = min(int(rng.choice([1, 1, 1, 2, 4, 9, 30, 70])), len(t) - at[n])
            part.append((n, t[at[n]:at[n] + k]))
            at[n] += k
            if at[n] == len(t):
                end.append(n)
        if part:
            f.step(part, end)
        live = [n for n in live if n not in end]
    for n in at:
        assert worst_error(f.all(n), case.expected[n[0]]) < tol(dtype), n


def test_batch_composition_changes_rounding_at_most(pkg, backend, case):
    """A request alone and the same request inside a batch: in the f32 build, equal up to a few roundings."""
    alone = Feeder(pkg, make_model(pkg, backend, case.cfg, case.weights, pkg.DType.F32))
    a = alone.run("a", case.tokens["a"], [90, 1])
    f = Feeder(pkg, make_model(pkg, backend, case.cfg, case.weights, pkg.DType.F32))
    f.step([("e", case.tokens["e"][:40]), ("a", case.tokens["a"][:90]), ("c", case.tokens["c"][:5])])
    for i in range(90, 230):
        f.step([("c", case.tokens["c"][i % 33:i % 33 + 1]), ("a", case.tokens["a"][i:i + 1])])
    assert worst_error(f.all("a"), a.astype(np.float64)) < 5e-6


def test_first_tokens(pkg, backend, case, dtype):
    """Sequences of one to nine tokens, each alone and all in one batch."""
    f = Feeder(pkg, make_model(pkg, backend, case.cfg, case.weights, dtype, seqs=9))
    t = case.tokens["a"]
    names = [f"n{k}" for k in range(1, 10)]
    f.step([(n, t[:int(n[1:])]) for n in names], names)
    for n in names:
        k = int(n[1:])
        assert worst_error(f.all(n), case.expected["a"][:k]) < tol(dtype), n
        assert worst_error(f.run(n + "s", t[:k], [k]), case.expected["a"][:k]) < tol(dtype), n


def test_any_routing_in_32_bits(pkg, backend):
    """Routers that are not made to be decisive."""
    cfg = CONFIGS["tuned"]
    w = random_weights(cfg, seed=31, decisive=False)
    t = np.random.default_rng(1).integers(0, cfg["vocab"], 150).tolist()
    f = Feeder(pkg, make_model(pkg, backend, cfg, w, pkg.DType.F32))
    exp = vusenex.forward(t, cfg, w)
    assert worst_error(f.run("p", t, [150]), exp) < TOL["F32"]
    assert worst_error(f.run("q", t, [30, 2, 9, 1]), exp) < TOL["F32"]


# ---- one mechanism at a time: the other sublayers contribute nothing ---------------------------------

def silence(w, *parts):
    for n in w:
        if any(p in n for p in parts):
            w[n] = np.zeros_like(w[n])
    return w


def only(w, *norms):
    """Sublayers whose norm is not named add nothing."""
    return silence(w, *(n for n in w if n.endswith((".norm1", ".norm2")) and n not in norms))


L = latent(2, 16, 16, 16)
MECHANISMS = {
    "embedding, final norm and head": (config(72, 40, [L]), ()),
    "pairs with one bucket": (config(72, 40, [L], pairs=(1, 3, 4)), ()),
    "pairs with large factors": (config(72, 40, [L], pairs=(1009, 4294967311, 99999989)), ()),
    "embedding of a width that is no multiple of four": (config(54, 40, [latent(2, 8, 8, 16)]), ()),
    "latent attention": (config(96, 40, [latent(3, 32, 48, 64)]), ("l0.norm1",)),
    "latent attention, many heads": (config(96, 40, [latent(33, 16, 16, 80, scale=0.4)]), ("l0.norm1",)),
    "latent attention, wide values": (config(96, 40, [latent(2, 48, 256, 192)]), ("l0.norm1",)),
    "latent attention, ragged sizes": (config(90, 40, [latent(3, 19, 33, 21)]), ("l0.norm1",)),
    "latent attention, short latents": (config(96, 40, [latent(4, 32, 32, 32)]), ("l0.norm1",)),
    "attention": (config(96, 40, [attn(6, 2, 64)]), ("l0.norm1",)),
    "attention without query factors": (config(96, 40, [attn(8, 1, 128, temp=None)]), ("l0.norm1",)),
    "query factors that grow at every token": (config(96, 40, [attn(4, 4, 32, temp=(1.3, 1))]), ("l0.norm1",)),
    "query factors at fractions of a token": (config(96, 40, [attn(2, 1, 16, temp=(0.6, 2.5))]), ("l0.norm1",)),
    "attention, one head": (config(96, 40, [attn(1, 1, 48)]), ("l0.norm1",)),
    "attention, wide heads": (config(96, 40, [attn(4, 2, 200)]), ("l0.norm1",)),
    "attention, heads the tuned kernels do not take": (config(96, 40, [attn(2, 1, 272)]), ("l0.norm1",)),
    "attention, ragged sizes": (config(90, 40, [attn(3, 3, 11)]), ("l0.norm1",)),
    "attention, twenty heads to a key": (config(96, 40, [attn(20, 1, 40)]), ("l0.norm1",)),
    "mixture": (config(72, 40, [latent(2, 16, 16, 16, moe(7, 7, 3, 2, 21, 30))]), ("l0.norm2",)),
    "mixture on tensor cores": (config(128, 60, [latent(2, 16, 16, 16, moe(12, 4, 2, 3, 72, 136))]), ("l0.norm2",)),
    "every group kept": (config(128, 60, [latent(2, 16, 16, 16, moe(12, 4, 4, 5, 64))]), ("l0.norm2",)),
    "one expert": (config(128, 60, [latent(2, 16, 16, 16, moe(1, 1, 1, 1, 64, 64))]), ("l0.norm2",)),
    "many experts": (config(128, 60, [latent(2, 16, 16, 16, moe(160, 8, 3, 6, 64, 64))]), ("l0.norm2",)),
    "routed experts alone": (config(128, 60, [latent(2, 16, 16, 16, moe(16, 2, 1, 8, 64))]), ("l0.norm2",)),
}


@pytest.mark.parametrize("name", sorted(MECHANISMS))
def test_mechanism_alone(pkg, backend, dtype, name):
    cfg, audible = MECHANISMS[name]
    w = only(random_weights(cfg, seed=3), *audible)
    t = np.random.default_rng(1).integers(0, cfg["vocab"], 150).tolist()
    exp = vusenex.forward(t, cfg, w)
    f = Feeder(pkg, make_model(pkg, backend, cfg, w, dtype))
    assert worst_error(f.run("p", t, [150]), exp) < tol(dtype)
    assert worst_error(f.run("q", t, [30, 2, 9, 1]), exp) < tol(dtype)


@pytest.mark.parametrize("part", ["l0.rg1", "l0.rg2"])
def test_gates_alone(pkg, backend, dtype, part):
    """Gates that open and close whole values, one sublayer at a time."""
    cfg = config(128, 40, [attn(4, 2, 32, moe(4, 2, 1, 1, 64, 64))])
    w = only(random_weights(cfg, seed=3), "l0.norm" + part[-1])
    w[part] = bf16(6.0 * w[part])
    t = np.random.default_rng(1).integers(0, 40, 150).tolist()
    exp = vusenex.forward(t, cfg, w)
    assert worst_error(vusenex.forward(t, cfg, {**w, part: 0 * w[part]}), exp) > 0.1
    f = Feeder(pkg, make_model(pkg, backend, cfg, w, dtype))
    assert worst_error(f.run("p", t, [150]), exp) < tol(dtype)
    assert worst_error(f.run("q", t, [30, 2, 9, 1]), exp) < tol(dtype)


@pytest.mark.parametrize("rows", [5, 17, 33, 64, 65, 200, 300, 700])
@pytest.mark.parametrize("experts", [(8, 4, 2, 2, 72, 200), (16, 8, 5, 4, 64, None), (6, 3, 1, 2, 136, 64)])
def test_tiles_of_experts(pkg, backend, dtype, rows, experts):
    """Every number of rows per tile, experts with no, few and many rows, products that end inside a tile."""
    cfg = config(128, 64, [latent(1, 16, 16, 16, moe(*experts))])
    w = only(random_weights(cfg, seed=rows), "l0.norm2")
    rng = np.random.default_rng(2)
    t = np.where(rng.random(rows) < 0.7, rng.integers(0, 3, rows), rng.integers(0, 64, rows)).tolist()  # uneven use of the experts
    f = Feeder(pkg, make_model(pkg, backend, cfg, w, dtype))
    assert worst_error(f.run("p", t, [rows]), vusenex.forward(t, cfg, w)) < tol(dtype)


def test_a_dense_feed_forward_in_gated_blocks(pkg, backend, dtype):
    """Not part of the design, but of the block."""
    cfg = config(128, 40, [attn(4, 2, 32), latent(2, 16, 16, 64)])
    rng, H, F = np.random.default_rng(5), 128, 96
    w = random_weights(cfg, seed=3)
    for n, shape in (("norm2", ()), ("rg2", (H, H)), ("rg2.b", (H,)), ("mlp.up", (F, H)), ("mlp.down", (H, F))):
        w["l1." + n] = bf16(1.5 * rng.standard_normal(shape) / np.sqrt(shape[-1])) if len(shape) == 2 else bf16(rng.uniform(0.5, 1.5, shape))
    t = rng.integers(0, 40, 150).tolist()
    x = vusenex.forward(t, cfg, w, keep_layers=True)[1][-1]
    y = vusenex.linear(np.maximum(vusenex.linear(x, w["l1.mlp.up"].astype(float)), 0.0) ** 2, w["l1.mlp.down"].astype(float))
    x = x + vusenex.rms_norm(vusenex.gated(y, x, w["l1.rg2"].astype(float), w["l1.rg2.b"]), w["l1.norm2"], 1e-5)
    exp = vusenex.linear(vusenex.rms_norm(x, w["final.norm"], 1e-5), w["head"].astype(float))
    meta = pkg.LayeredMetadata.from_config(cfg)
    meta.layers[1] = dataclasses.replace(meta.layers[1], ffn_dim=F, activation="relu2")
    m = pkg.CudaLayeredModel.new(meta, w, 64, 16, backend, compute_dtype=dtype, max_batch_tokens=1024, max_batch_sequences=8)
    f = Feeder(pkg, m)
    assert worst_error(f.run("p", t, [150]), exp) < tol(dtype)
    assert worst_error(f.run("q", t, [30, 2, 9, 1]), exp) < tol(dtype)


# ---- far keys and keys at page borders: one score that stands out ----------------------------------------

def beacon_model(mixer, width=128, positions=900):
    """One layer in which token 1, as a query, is drawn to token 2 as a key, so that the value of token 2 dominates wherever it is
    visible: both have a dimension of the stream of their own, and only there do some dimensions of queries and keys look."""
    cfg = config(width, 64, [mixer], positions=positions)
    w = random_weights(cfg, seed=8)
    w["embed"][:, -2:] = w["bigram"][:, -2:] = w["pos"][:, -2:] = 0.0
    w["embed"][1, -2] = w["embed"][2, -1] = 8.0
    m, p = mixer["mixer"], "l0.mix."
    q = w[p + "q"].reshape(m["heads"], m["dim"], width)
    q[:, :, -2:] = 0.0
    if mixer["type"] == "attention":
        k, half = w[p + "k"].reshape(m["kv_heads"], m["dim"], width), m["dim"] // 2
        k[:, :, -2:] = 0.0
        q[:, half:], k[:, half:] = 0.0, 0.0
        q[:, half:, -2], k[:, half:, -1] = 1.5, 1.5
        for n in ("q", "k"):
            w[f"{p}{n}.norm"] = np.ones_like(w[f"{p}{n}.norm"])
            w[f"{p}{n}.b"].reshape(-1, m["dim"])[:, half:] = 0.0
        m["scale"] = (40.0 if m["dim"] > 16 else 20.0) / m["dim"]
    else:
        half = m["kv_rank"] // 2
        w[p + "dkv"][:, -2:] = 0.0
        w[p + "dkv"][half:] = 0.0
        w[p + "dkv"][half:, -1] = 1.5
        w[p + "dkv.norm"] = np.ones_like(w[p + "dkv.norm"])
        uk = w[p + "uk"].reshape(m["heads"], m["dim"], m["kv_rank"])
        q[:, :2], uk[:, :2] = 0.0, 0.0
        q[:, 2:] = bf16(0.3 * q[:, 2:])
        uk[:, 2:, half:] = 0.0
        q[:, :2, -2], uk[:, :2, half:] = 1.0, bf16(2.0 / half)
        m["scale"] = 1.0
    return cfg, w


BEACONS = {"attention": attn(6, 2, 64, temp=(0.2, 100)), "attention, few dimensions": attn(2, 1, 10), "attention, many dimensions": attn(8, 2, 112), "latent attention": latent(3, 32, 32, 64),
           "latent attention, few dimensions": latent(2, 6, 10, 12)}


@pytest.mark.parametrize("name", sorted(BEACONS))
def test_keys_at_page_borders(pkg, backend, dtype, name):
    """The key at the borders of pages and of the kernels' tiles, in prompts and in decoding; a key that comes only after the query."""
    cfg, w = beacon_model(json.loads(json.dumps(BEACONS[name])))
    rng = np.random.default_rng(3)
    f = Feeder(pkg, make_model(pkg, backend, cfg, w, dtype))
    runs = 0
    for key, query in [(0, 1), (0, 15), (0, 16), (15, 16), (16, 17), (15, 140), (16, 140), (63, 64), (64, 129), (127, 128), (128, 255), (0, 290), (280, 290),
                       (18, 17), (65, 64)]:
        t = rng.integers(3, 64, max(query, key) + 9)
        t[key], t[query] = 2, 1
        t = t.tolist()
        exp = vusenex.forward(t, cfg, w)
        blind = list(t)
        blind[key] = 3
        shift = worst_error(vusenex.forward(blind, cfg, w)[query:query + 1], exp[query:query + 1])
        assert (shift > 0.15) == (key < query), (key, query, shift)
        for sizes in ([len(t)], [query, 1], [max(query - 1, 1), 3], [max(query - 5, 1), 12]):
            runs += 1
            assert worst_error(f.run(f"r{runs}", t, sizes), exp) < tol(dtype), (key, query, sizes)


@pytest.mark.parametrize("name", sorted(BEACONS))
def test_a_far_key_among_hundreds(pkg, backend, dtype, name):
    cfg, w = beacon_model(json.loads(json.dumps(BEACONS[name])))
    t = np.random.default_rng(4).integers(3, 64, 760)
    t[[20, 700]] = 2
    t[[400, 619, 620, 650, 712, 759]] = 1
    t = t.tolist()
    exp = vusenex.forward(t, cfg, w)
    blind = list(t)
    blind[20] = 3
    without = vusenex.forward(blind, cfg, w)
    assert all(worst_error(without[p:p + 1], exp[p:p + 1]) > 0.15 for p in (400, 619, 620, 650))
    for sizes in ([760], [590, 1], [128], [500, 3]):
        f = Feeder(pkg, make_model(pkg, backend, cfg, w, dtype))
        assert worst_error(f.run("p", t, sizes), exp) < tol(dtype), sizes


@pytest.mark.parametrize("dim", [40, 128, 144])
@pytest.mark.parametrize("rate", [0.0, 0.002, 0.2, 5.0, 300.0])
def test_distance_terms_of_any_rate(pkg, backend, dtype, rate, dim):
    """Flat ones, ones that fall slowly, and ones that fall at the first step, with multiples of either sign, near and far."""
    cfg = config(96, 40, [attn(6, 3, dim)])
    w = random_weights(cfg, seed=3)
    w["l0.mix.r2"] = bf16(np.full(6, rate))
    w["l0.mix.r1"] = bf16(np.linspace(-0.5, 3.0, 6))
    t = np.random.default_rng(1).integers(0, 40, 620).tolist()
    exp = vusenex.forward(t, cfg, w)
    f = Feeder(pkg, make_model(pkg, backend, cfg, w, dtype))
    assert worst_error(f.run("p", t, [620]), exp) < tol(dtype)
    assert worst_error(f.run("q", t, [400, 2, 9, 150, 1]), exp) < tol(dtype)


def test_pairs_of_tokens_across_steps(pkg, backend, dtype):
    """The predecessor comes from the batch or from an earlier step, on this page or the one before; other requests in between leave it alone."""
    cfg = config(64, 200, [latent(1, 8, 8, 8)], pairs=(997, 201, 1))
    w = only(random_weights(cfg, seed=2))
    rng = np.random.default_rng(1)
    t = {n: rng.integers(0, 200, 70).tolist() for n in "ab"}
    exp = {n: vusenex.forward(t[n], cfg, w) for n in t}
    for cut in (1, 2, 15, 16, 17, 31, 32, 33):
        f = Feeder(pkg, make_model(pkg, backend, cfg, w, dtype, blocks=12))
        f.step([("a", t["a"][:cut])])
        f.step([("b", t["b"][:cut])])
        f.step([("b", t["b"][cut:cut + 1]), ("a", t["a"][cut:cut + 2])])
        f.step([("a", t["a"][cut + 2:])], ["a"])
        f.step([("b", t["b"][cut + 1:])], ["b"])
        f.step([("a2", t["a"][:cut])])  # on pages that held other tokens
        f.step([("a2", t["a"][cut:])])
        for n in ("a", "b", "a2"):
            assert worst_error(f.all(n), exp[n[0]]) < tol(dtype), (cut, n)


def test_keys_in_the_cache(pkg, backend, dtype):
    """One set of rows, the keys as projected, and the factor of their norm."""
    cfg = config(64, 40, [attn(4, 2, 20), latent(2, 12, 12, 24)])
    w = random_weights(cfg, seed=4)
    t = np.random.default_rng(1).integers(0, 40, 37).tolist()
    m = make_model(pkg, backend, cfg, w, dtype, blocks=4)
    m.forward(pkg.ForwardBatch(t, list(range(37)), [1], [37], [37], [[2, 0, 3]]))
    k, factor, c = m.read_kv()
    assert k.shape == (4, 2, 16, 20) and factor.shape == (4, 2, 16, 1) and c.shape == (4, 16, 24)
    x = vusenex.embedding(t, cfg, w, np.float64)
    keys = x @ w["l0.mix.k"].T + w["l0.mix.k.b"]
    rows = np.concatenate([k[b].transpose(1, 0, 2) for b in (2, 0, 3)])[:37]
    assert np.abs(rows.reshape(37, 40) - keys).max() < (2e-5 if dtype == pkg.DType.F32 else 8e-2)
    got = np.concatenate([factor[b, :, :, 0].T for b in (2, 0, 3)])[:37]
    assert np.allclose(got, 1 / np.sqrt((keys ** 2).mean(axis=1, keepdims=True) + 1e-5), rtol=1e-5 if dtype == pkg.DType.F32 else 2e-2)
    assert not k[1].any() and not factor[1].any()


# ---- the model inside the framework -----------------------------------------------------------------

def greedy(cfg, w, prompt, n):
    out = list(prompt)
    for _ in range(n):
        out.append(int(np.argmax(vusenex.forward(out, cfg, w)[-1])))
    return out[len(prompt):]


def follows_greedily(cfg, w, prompt, out, margin):
    """Every token is the plain implementation's best one after the tokens before it, up to `margin` logits."""
    logits = vusenex.forward(prompt + out, cfg, w)
    return all(logits[len(prompt) - 1 + i][tok] >= logits[len(prompt) - 1 + i].max() - margin for i, tok in enumerate(out))


def run_engine(pkg, model, prompts, n, blocks, **cfg):
    E = pkg.engine
    kw = dict(max_num_seqs=8, max_num_batched_tokens=64, request_timeout_secs=None)
    kw.update(cfg)
    eng = E.Engine(model, E.SchedulerConfig(**kw), blocks, 16, True)
    tokens = {}
    for p in prompts:
        tokens[eng.submit(p, E.SamplingParams(temperature=0.0, max_tokens=n))] = []
    for _ in range(2000):
        if not eng.has_work():
            break
        eng.step()
        for ev in eng.take_events():
            if ev.kind == "token":
                tokens[ev.id].append(ev.token)
    assert not eng.has_work()
    return list(tokens.values()), eng


@pytest.mark.parametrize("name", ["odd", "tuned"])
def test_generation_through_the_engine(pkg, backend, name, dtype):
    """Chunked prompts, continuous batching, the tokens of plain greedy decoding."""
    c = Case.get(name)
    rng = np.random.default_rng(6)
    prompts = [rng.integers(0, c.cfg["vocab"], k).tolist() for k in (3, 40, 90, 17, 1, 64)]
    model = make_model(pkg, backend, c.cfg, c.weights, dtype, tokens=64, seqs=8)
    assert model.num_state_slots() == 0
    out, eng = run_engine(pkg, model, prompts, 20, 64)
    for p, o in zip(prompts, out):
        assert len(o) == 20
        if dtype == pkg.DType.F32:
            assert o == greedy(c.cfg, c.weights, p, 20)
        assert follows_greedily(c.cfg, c.weights, p, o, 1e-3 if dtype == pkg.DType.F32 else 0.35)
    assert eng.scheduler().cache().stats()["free_blocks"] == 64


def test_preempted_requests_are_recomputed(pkg, backend):
    """A pool too small for all requests: some are preempted in the middle of their output, and every one still
    gets the tokens of plain greedy decoding."""
    c = Case.get("odd")
    rng = np.random.default_rng(7)
    prompts = [rng.integers(0, c.cfg["vocab"], k).tolist() for k in (30, 28, 25, 31)]
    model = make_model(pkg, backend, c.cfg, c.weights, pkg.DType.F32, blocks=12, tokens=64, seqs=4)
    out, eng = run_engine(pkg, model, prompts, 40, 12)
    assert eng.scheduler().stats()["total_preempted"] > 0
    for p, o in zip(prompts, out):
        assert o == greedy(c.cfg, c.weights, p, 40)


def test_cached_prefixes_are_skipped(pkg, backend):
    """Nothing but the cache is carried along, predecessors included, so a prompt whose first blocks are cached starts behind them."""
    c = Case.get("odd")
    head = np.random.default_rng(8).integers(0, c.cfg["vocab"], 48).tolist()
    prompts = [head + [1, 2, 3], head + [4], head]
    model = make_model(pkg, backend, c.cfg, c.weights, pkg.DType.F32, tokens=64, seqs=4)
    out, eng = run_engine(pkg, model, prompts, 6, 64, max_num_seqs=1, skip_cached_prefix=True)
    assert eng.scheduler().stats()["total_skipped_prefill_tokens"] > 48
    for p, o in zip(prompts, out):
        assert o == greedy(c.cfg, c.weights, p, 6)


def test_checkpoint_directory_through_the_registry(pkg, backend, tmp_path):
    from orionserve_rs_b200.trace import TraceRunner

    c = Case("tuned")
    (tmp_path / "config.json").write_text(json.dumps(c.cfg))
    pkg.write_safetensors(str(tmp_path / "model.safetensors"), c.weights, pkg.DType.BF16)
    assert pkg.model_class(str(tmp_path)) is pkg.CudaLayeredModel
    r = TraceRunner.from_directory(str(tmp_path), pkg.DType.F32, 256)
    got = r.step([{"id": "x", "tokens": c.tokens["b"], "want": [3, 96, 50]}], ["x"])
    assert worst_error(got, c.expected["b"][[3, 96, 50]]) < 3e-5
    del c.weights["l2.mlp.e17.up"]
    pkg.write_safetensors(str(tmp_path / "model.safetensors"), c.weights, pkg.DType.BF16)
    with pytest.raises(pkg.ModelError, match="missing tensor `l2.mlp.e17.up`"):
        pkg.load_model(str(tmp_path), 8, 16, backend)


def test_positions_with_gaps_are_refused(pkg, backend):
    c = Case.get("odd")
    m = make_model(pkg, backend, c.cfg, c.weights, pkg.DType.F32)
    with pytest.raises(pkg.InternalError, match="not consecutive"):
        m.forward(pkg.ForwardBatch([1, 1], [3, 5], [1], [2], [6], [[0]]))


def test_positions_beyond_the_table_are_refused(pkg, backend):
    c = Case.get("odd")
    m = make_model(pkg, backend, c.cfg, c.weights, pkg.DType.F32)
    with pytest.raises(pkg.InternalError, match="position 300"):
        m.forward(pkg.ForwardBatch([1], [300], [1], [1], [301], [list(range(19))]))
    eng = pkg.engine.Engine(m, pkg.engine.SchedulerConfig(max_num_batched_tokens=64, request_timeout_secs=None), 64, 16, True)
    with pytest.raises(pkg.EngineError, match="exceeds context length 300"):
        eng.submit([1] * 290, pkg.engine.SamplingParams(temperature=0.0, max_tokens=11))
    eng.submit([1] * 290, pkg.engine.SamplingParams(temperature=0.0, max_tokens=10))
    while eng.has_work():
        eng.step()
    assert sum(ev.kind == "token" for ev in eng.take_events()) == 10


def test_step_graph_replays_the_same_logits(pkg, backend):
    c = Case.get("tuned")
    m = make_model(pkg, backend, c.cfg, c.weights, pkg.DType.BF16)
    f = Feeder(pkg, m)
    t = c.tokens["a"]
    f.step([("x", t[:40]), ("y", t[:7])])
    for i in range(100):  # beyond the number of repeats after which the layout is captured
        f.step([("x", [t[40 + i]]), ("y", [t[7 + i]])])
    assert worst_error(f.all("x"), c.expected["a"][:140]) < TOL["BF16"]
    assert worst_error(f.all("y"), c.expected["a"][:107]) < TOL["BF16"]
    assert m.replay(3) > 0
    f.step([("x", [t[140]]), ("y", [t[107]])])
    assert worst_error(f.all("x"), c.expected["a"][:141]) < TOL["BF16"]
