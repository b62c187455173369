"""Belizen on the device against the plain implementation in ``oracle/belizen.py``: every mechanism alone, whole prompts,
portions, decoding, mixed batches, reuse of pages and state slots, window edges and kept tokens, far keys, long memory, and generation
through the engine. ``tol`` is the bar on the rms error of a row of logits over the rms of the logits: 3e-5 in the f32 build; 3e-2 in
the bf16 build, whose weights are the same values and whose activations are rounded."""
import json

import numpy as np
import pytest

from metapel_models import Feeder, make_model, worst_error
from oracle import belizen
from belizen_models import CONFIGS, attn, bf16, config, dense, gla, moe, random_weights, yarn

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
        self.expected = {n: belizen.forward(t, self.cfg, self.weights) for n, t in self.tokens.items()}

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
    # long decoding after a prompt: windows slide over decoded tokens
    assert worst_error(f.run("a", case.tokens["a"], [50, 1]), case.expected["a"]) < tol(dtype)


@pytest.mark.parametrize("sizes", [[2], [3], [7], [8], [9], [16], [17], [64], [1, 2, 63, 5, 33, 1, 1, 12, 100]])
def test_portions(pkg, backend, case, dtype, sizes):
    f = Feeder(pkg, make_model(pkg, backend, case.cfg, case.weights, dtype))
    assert worst_error(f.run("a", case.tokens["a"], sizes), case.expected["a"]) < tol(dtype)


def test_mixed_batches_and_reuse(pkg, backend, case, dtype):
    """Unequal requests in one batch, prompts beside single tokens, on a pool that just holds the live ones, so
    that pages and slots are used again by later requests; the order of the entries changes too."""
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
    exp = belizen.forward(t, cfg, w)
    assert worst_error(f.run("p", t, [150]), exp) < TOL["F32"]
    assert worst_error(f.run("q", t, [30, 2, 9, 1]), exp) < TOL["F32"]


# ---- one mechanism at a time: the other sublayers contribute nothing ---------------------------------

def silence(w, *parts):
    for n in w:
        if any(p in n for p in parts):
            w[n] = np.zeros_like(w[n])
    return w


G = gla(2, 16, 16, 4.0, 4)
MECHANISMS = {
    "embedding, final norm and head": (config(72, 40, [gla(2, 16, 16, 4.0, 4, dense(24))], cap=0.0), (".o", ".down")),
    "soft cap of the logits": (config(72, 40, [gla(2, 16, 16, 4.0, 4, dense(24))], cap=2.0), (".o", ".down")),
    "loop": (config(72, 40, [G, G, G], loop=(1, 2, 4)), (".o",)),
    "loop of all layers": (config(72, 40, [G, G], loop=(0, 2, 2)), (".o",)),
    "loop of one pass": (config(72, 40, [G, G], loop=(1, 2, 1)), ()),
    "gated dense feed-forward": (config(72, 40, [gla(2, 16, 16, 4.0, 4, dense(100))]), ("mix.o",)),
    "gated dense feed-forward on tensor cores": (config(128, 40, [gla(2, 16, 16, 4.0, 4, dense(328))]), ("mix.o",)),
    "mixture": (config(72, 40, [gla(2, 16, 16, 4.0, 4, moe(7, 3, 2, 21, 0.7, 30, 1.9))]), ("mix.o",)),
    "mixture on tensor cores": (config(128, 60, [gla(2, 16, 16, 4.0, 4, moe(7, 2, 2, 72, 0.8, 136, 2.1))]), ("mix.o",)),
    "routed experts alone": (config(128, 60, [gla(2, 16, 16, 4.0, 4, moe(12, 1, 3, 64, 3.0))]), ("mix.o",)),
    "identity experts alone": (config(128, 60, [gla(2, 16, 16, 4.0, 4, moe(3, 9, 4, 64, 1.0))]), ("mix.o", ".down")),
    "shared expert alone": (config(128, 60, [gla(2, 16, 16, 4.0, 4, moe(4, 0, 1, 64, 1.0, 72, 0.6))]), ("mix.o", ".e0.", ".e1.", ".e2.", ".e3.")),
    "values and windows": (config(96, 40, [attn(4, 2, 64, 64, 13, 3)]), ("mix.q", "mix.g")),
    "gates": (config(96, 40, [attn(4, 2, 64, 64, 50)]), ("mix.q",)),
    "soft cap of the scores": (config(96, 40, [attn(4, 2, 64, 64, 50, 9, scale=1.0, cap=2.5)]), ()),
    "attention": (config(96, 40, [attn(6, 2, 64, 64, 50, 7, base=30.0)]), ()),
    "stretched frequencies": (config(96, 40, [attn(6, 2, 64, 64, 100, 0, rot_dims=64, yarn=yarn(6.0, 40, 3.0, 0.7))]), ()),
    "attention over everything before": (config(96, 40, [attn(8, 1, 128, 128, None, rot_dims=128, cap=0.0)]), ()),
    "linear attention": (config(96, 40, [gla(3, 32, 64, 16.0, 16)]), ()),
    "linear attention, wide keys": (config(96, 40, [gla(1, 256, 32, 8.0, 16)]), ()),
    "linear attention, steep decays": (config(96, 40, [gla(2, 64, 64, 0.1, 8)]), ()),
    "linear attention, ragged sizes": (config(90, 40, [gla(3, 19, 33, 3.0, 5)]), ()),
}


@pytest.mark.parametrize("name", sorted(MECHANISMS))
def test_mechanism_alone(pkg, backend, dtype, name):
    cfg, silent = MECHANISMS[name]
    w = silence(random_weights(cfg, seed=3), *silent)
    t = np.random.default_rng(1).integers(0, cfg["vocab"], 150).tolist()
    exp = belizen.forward(t, cfg, w)
    f = Feeder(pkg, make_model(pkg, backend, cfg, w, dtype))
    assert worst_error(f.run("p", t, [150]), exp) < tol(dtype)
    assert worst_error(f.run("q", t, [30, 2, 9, 1]), exp) < tol(dtype)


@pytest.mark.parametrize("rows", [5, 17, 33, 64, 65, 200, 300, 700])
@pytest.mark.parametrize("experts", [(2, 1, 2, 72, 1.0, 200), (16, 4, 2, 64, 0.8, None), (3, 5, 4, 136, 2.0, 64)])
def test_tiles_of_experts(pkg, backend, dtype, rows, experts):
    """Every number of rows per tile, experts with no, few and many rows, products that end inside a tile, rows without any expert."""
    cfg = config(128, 64, [gla(1, 8, 8, 4.0, 2, moe(*experts))])
    w = silence(random_weights(cfg, seed=rows), "mix.o")  # a lone head of eight values may all but cancel, whatever computes it
    rng = np.random.default_rng(2)
    t = np.where(rng.random(rows) < 0.7, rng.integers(0, 3, rows), rng.integers(0, 64, rows)).tolist()  # uneven use of the experts
    f = Feeder(pkg, make_model(pkg, backend, cfg, w, dtype))
    exp = belizen.forward(t, cfg, w)
    assert worst_error(f.run("p", t, [rows]), exp) < tol(dtype)


# ---- linear attention: chunk borders and long memory ------------------------------------------------------

@pytest.mark.parametrize("shape", [(2, 32, 32, 16.0, 8), (1, 48, 80, 0.2, 4), (2, 128, 128, 16.0, 16), (1, 160, 24, 2.0, 6), (1, 10, 14, 5.0, 3)])
def test_portions_that_end_around_chunk_borders(pkg, backend, dtype, shape):
    cfg = config(96, 40, [gla(*shape)])
    w = random_weights(cfg, seed=9)
    t = np.random.default_rng(1).integers(0, 40, 261).tolist()
    exp = belizen.forward(t, cfg, w)
    f = Feeder(pkg, make_model(pkg, backend, cfg, w, dtype))
    for k, sizes in enumerate(([261], [63], [64], [65], [9, 128], [1, 10, 2, 64, 8, 70], [127, 1, 1, 132])):
        assert worst_error(f.run(f"r{k}", t, sizes), exp) < tol(dtype), sizes


def test_a_token_is_remembered_for_long(pkg, backend, dtype):
    """Decays close to one; a key that only one early token has, asked for by late ones: in prompts, portions and decoding."""
    cfg, w = memory_model()
    t = np.random.default_rng(4).integers(3, 64, 620)
    t[5] = 2
    t[[70, 128, 400, 555, 619]] = 1
    t = t.tolist()
    exp = belizen.forward(t, cfg, w)
    blind = list(t)
    blind[5] = 3
    assert worst_error(belizen.forward(blind, cfg, w)[619:], exp[619:]) > 0.1
    for sizes in ([620], [500, 1], [64], [300, 7, 2, 90]):
        f = Feeder(pkg, make_model(pkg, backend, cfg, w, dtype))
        assert worst_error(f.run("p", t, sizes), exp) < tol(dtype), sizes


def memory_model():
    cfg = config(128, 64, [gla(2, 32, 32, 16.0, 8)], mult=1.0)
    w = random_weights(cfg, seed=8)
    w["l0.mix.a2.b"] = bf16(np.full_like(w["l0.mix.a2.b"], 9.0))
    w["l0.mix.a2"] *= 0
    w["l0.norm1"] = np.ones_like(w["l0.norm1"])
    q, k = (w[f"l0.mix.{n}"].astype(np.float64).reshape(2, 32, 128) for n in "qk")
    w["embed"][:, 100:] = 0.0  # two dimensions that only tokens 1 and 2 have
    w["embed"][1, 126] = w["embed"][2, 127] = 6.0
    q[:, :, 126:], k[:, :, 126:] = 0.0, 0.0
    k[:, 16:] = 0.0
    q[:, 16:, 126], k[:, 16:, 127] = 3.0, 3.0
    w["l0.mix.q"], w["l0.mix.k"] = bf16(q.reshape(-1, 128)), bf16(k.reshape(-1, 128))
    return cfg, w


def test_passes_of_a_loop_keep_states_and_caches_of_their_own(pkg, backend, dtype):
    """With one cache or state for all passes, the second pass would meet what the first has left."""
    cfg = config(96, 40, [gla(2, 16, 16, 16.0, 4), attn(2, 1, 32, 32, 30, 2), gla(2, 16, 16, 16.0, 4)], loop=(0, 2, 3))
    w = random_weights(cfg, seed=2)
    t = np.random.default_rng(1).integers(0, 40, 120).tolist()
    exp = belizen.forward(t, cfg, w)
    m = make_model(pkg, backend, cfg, w, dtype)
    assert len(m.read_kv()) == 6
    f = Feeder(pkg, m)
    for k, sizes in enumerate(([120], [60, 1], [11])):
        assert worst_error(f.run(f"p{k}", t, sizes), exp) < tol(dtype), sizes


# ---- windows and far keys: one score that stands out -----------------------------------------------------

def beacon_model(window, keep, heads=2, kv_heads=1, dim=16, vdim=16, width=128):
    """One attention layer in which token 1, as a query, is drawn to token 2 as a key, so that the value of token 2
    dominates wherever it is visible; the keys of the other tokens have little in the dimensions that token 1 asks in."""
    cfg = config(width, 64, [attn(heads, kv_heads, dim, vdim, window, keep, rot_dims=4, scale=32.0 / dim, cap=25.0)], mult=1.0, cap=0.0)
    w = random_weights(cfg, seed=8)
    hq, hk = (w["embed"][i].astype(np.float64) for i in (1, 2))
    hq, hk = hq / np.sqrt((hq ** 2).mean()), hk / np.sqrt((hk ** 2).mean())
    w["l0.norm1"] = np.ones_like(w["l0.norm1"])
    for n in ("q.norm", "k.norm"):
        w[f"l0.mix.{n}"] = np.ones_like(w[f"l0.mix.{n}"])
    half, u = dim // 2, np.zeros(dim)
    u[half:] = np.where(np.arange(dim - half) % 2, 1.0, -1.0)
    q = w["l0.mix.q"].astype(np.float64).reshape(heads, dim, width)
    k = w["l0.mix.k"].astype(np.float64).reshape(kv_heads, dim, width)
    k[:, half:] = 0.0
    w["l0.mix.q.b"] *= 0
    w["l0.mix.k.b"] = bf16(np.tile(np.where(np.arange(dim) < half, 6.0, 0.0), kv_heads))  # keys are long without what is asked for
    q += 14.0 * u[None, :, None] * hq / width
    k += 14.0 * u[None, :, None] * hk / width
    w["l0.mix.q"], w["l0.mix.k"] = bf16(q.reshape(-1, width)), bf16(k.reshape(-1, width))
    return cfg, w


def edge_cases(window, keep):
    """(key, query): the key just inside or just outside the window, one of the first tokens, the last kept or the first not kept; early
    and late in the sequence."""
    pairs = set()
    for query in (window + keep + 1, 2 * window + keep + 17, 290):
        pairs |= {(query - window + 1, query), (query - window, query), (query - window - 1, query), (0, query), (keep, query), (keep + 1, query),
                  (keep - 1, query)}
    return sorted((key, query) for key, query in pairs if 0 <= key < query)


@pytest.mark.parametrize("window,keep", [(1, 0), (1, 1), (2, 3), (15, 16), (16, 1), (17, 33), (33, 5), (64, 64), (65, 20), (130, 4)])
def test_window_edges_and_kept_tokens(pkg, backend, dtype, window, keep):
    cfg, w = beacon_model(window, keep)
    rng = np.random.default_rng(3)
    f = Feeder(pkg, make_model(pkg, backend, cfg, w, dtype))
    runs = 0
    for key, query in edge_cases(window, keep):
        t = rng.integers(3, 64, query + 9)
        t[key], t[query] = 2, 1
        t = t.tolist()
        exp = belizen.forward(t, cfg, w)
        blind = list(t)
        blind[key] = 3
        shift = worst_error(belizen.forward(blind, cfg, w)[query:query + 1], exp[query:query + 1])
        assert (shift > 0.15) == (query - key < window or key < keep), (key, query, shift)  # the key shows exactly when it is seen
        for sizes in ([len(t)], [query, 1], [max(query - 1, 1), 3], [max(query - 5, 1), 12]):
            runs += 1
            assert worst_error(f.run(f"r{runs}", t, sizes), exp) < tol(dtype), (key, query, sizes)


def test_a_far_key_among_hundreds(pkg, backend, dtype):
    cfg, w = beacon_model(600, 3, heads=9, kv_heads=3, dim=64, vdim=64)
    t = np.random.default_rng(4).integers(3, 64, 760)
    t[[20, 700]] = 2
    t[[400, 619, 620, 650, 712, 759]] = 1
    t = t.tolist()
    exp = belizen.forward(t, cfg, w)
    blind = list(t)
    blind[20] = 3
    without = belizen.forward(blind, cfg, w)
    assert all((worst_error(without[p:p + 1], exp[p:p + 1]) > 0.15) == seen for p, seen in ((400, True), (619, True), (620, False)))
    for sizes in ([760], [590, 1], [128], [500, 3]):
        f = Feeder(pkg, make_model(pkg, backend, cfg, w, dtype))
        assert worst_error(f.run("p", t, sizes), exp) < tol(dtype), sizes


def test_keys_and_values_in_the_cache(pkg, backend, dtype):
    cfg = config(64, 40, [attn(4, 2, 20, 28, 9, 2, rot_dims=8, yarn=yarn(4.0, 30, 2.0, 0.5))])
    w = random_weights(cfg, seed=4)
    t = np.random.default_rng(1).integers(0, 40, 37).tolist()
    m = make_model(pkg, backend, cfg, w, dtype, blocks=4)
    m.forward(pkg.ForwardBatch(t, list(range(37)), [1], [37], [37], [[2, 0, 3]]))
    k, v = m.read_kv()
    assert k.shape == (4, 2, 16, 20) and v.shape == (4, 2, 16, 28)
    h = belizen.rms_norm(cfg["embedding"]["scale"] * w["embed"][t].astype(np.float64), w["l0.norm1"], 1e-5)
    keys = (h @ w["l0.mix.k"].T + w["l0.mix.k.b"]).reshape(37, 2, 20)
    keys = belizen.rotate_halves(belizen.rms_norm(keys, w["l0.mix.k.norm"], 1e-5), np.arange(37), *belizen.yarn_frequencies(cfg["layers"][0]["mixer"]["rot"]))
    values = (h @ w["l0.mix.v"].T + w["l0.mix.v.b"]).reshape(37, 2, 28)
    for got, exp in ((k, keys), (v, values)):
        rows = np.concatenate([got[b].transpose(1, 0, 2) for b in (2, 0, 3)])[:37]
        assert np.abs(rows - exp).max() < (2e-5 if dtype == pkg.DType.F32 else 6e-2)
    assert not k[1].any() and not v[1].any()


# ---- the model inside the framework -----------------------------------------------------------------

def greedy(cfg, w, prompt, n):
    out = list(prompt)
    for _ in range(n):
        out.append(int(np.argmax(belizen.forward(out, cfg, w)[-1])))
    return out[len(prompt):]


def follows_greedily(cfg, w, prompt, out, margin):
    """Every token is the plain implementation's best one after the tokens before it, up to `margin` logits."""
    logits = belizen.forward(prompt + out, cfg, w)
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
    """Chunked prompts, continuous batching, more requests than state slots: the tokens of plain greedy decoding."""
    c = Case.get(name)
    rng = np.random.default_rng(6)
    prompts = [rng.integers(0, c.cfg["vocab"], k).tolist() for k in (3, 40, 90, 17, 1, 64)]
    model = make_model(pkg, backend, c.cfg, c.weights, dtype, tokens=64, seqs=4)
    assert model.num_state_slots() == 4
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


def test_batches_that_do_not_continue_the_state_are_refused(pkg, backend):
    c = Case.get("odd")
    m = make_model(pkg, backend, c.cfg, c.weights, pkg.DType.F32)
    m.forward(pkg.ForwardBatch([1, 2], [0, 1], [1], [2], [2], [[0]], state_slots=[0]))
    with pytest.raises(pkg.InternalError, match="its state covers 2 tokens"):
        m.forward(pkg.ForwardBatch([1], [3], [1], [1], [4], [[0]], state_slots=[0]))
    with pytest.raises(pkg.InvalidRequest, match="state slot"):
        m.forward(pkg.ForwardBatch([1], [2], [1], [1], [3], [[0]]))


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
