"""Metapel on the device against the plain implementation in ``oracle/metapel.py``: every mechanism alone, whole
prompts, portions, decoding, mixed batches, reuse of pages and slots, window edges, and generation through the
engine. ``tol`` is the bar on the rms error of a row of logits over the rms of the logits: 3e-5 in the f32
build; 3e-2 in the bf16 build, whose weights are the same values and whose activations are rounded."""
import json

import numpy as np
import pytest

from metapel_models import CONFIGS, Feeder, config, latent, make_model, mingru, random_weights, worst_error
from oracle import binding, metapel

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
    """One configuration: weights, expected logits of a few sequences, and device models on demand."""
    cache = {}

    def __init__(self, name):
        self.cfg = CONFIGS[name]
        self.weights = random_weights(self.cfg, seed=len(name))
        rng = np.random.default_rng(17)
        self.tokens = {n: rng.integers(0, self.cfg["vocab"], size).tolist()
                       for n, size in (("a", 230), ("b", 97), ("c", 33), ("d", 1), ("e", 161))}
        self.expected = {n: metapel.forward(t, self.cfg, self.weights) for n, t in self.tokens.items()}

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
    # long decoding after a prompt: the window passes over decoded tokens
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


# ---- one mechanism at a time: the rest of the layer contributes nothing ----------------------------

def silence(w, *parts):
    for n in w:
        if any(p in n for p in parts):
            w[n] = np.zeros_like(w[n])
    return w


MECHANISMS = {
    "convolution and feed-forward": (config(72, 90, [mingru(16, 100)], taps=4), ("mix.o",)),
    "feed-forward": (config(72, 90, [mingru(16, 100)], taps=4), ("mix.o", "canon")),
    "convolution and recurrence": (config(72, 90, [mingru(56, 24)], taps=6), ("mlp.down",)),
    "recurrence": (config(72, 90, [mingru(56)], taps=2), ("canon",)),
    "attention": (config(96, 90, [latent(4, 16, 16, 16, 48, 13)], taps=2), ("canon",)),
    "attention without a rotated part's influence": (config(96, 90, [latent(4, 16, 16, 16, 48, 300, base=30.0)], taps=2), ("canon", "mix.uk")),
    "attention over everything before": (config(96, 90, [dict(e, mixer=dict(e["mixer"], mask=None)) for e in [latent(5, 32, 16, 32, 64, 0)]],
                                                taps=2), ("canon",)),
    "final norm and head": (config(72, 90, [mingru(16)], taps=2), ("mix.o",)),
}


@pytest.mark.parametrize("name", sorted(MECHANISMS))
def test_mechanism_alone(pkg, backend, dtype, name):
    cfg, silent = MECHANISMS[name]
    w = silence(random_weights(cfg, seed=3), *silent)
    t = np.random.default_rng(1).integers(0, cfg["vocab"], 150).tolist()
    exp = metapel.forward(t, cfg, w)
    f = Feeder(pkg, make_model(pkg, backend, cfg, w, dtype))
    assert worst_error(f.run("p", t, [150]), exp) < tol(dtype)
    assert worst_error(f.run("q", t, [30, 2, 9, 1]), exp) < tol(dtype)


def long_memory():
    """Update gates that open for token 2 and stay almost shut for the others; 900 tokens, the first of them 2."""
    width = 256
    cfg = config(width, 80, [mingru(96)], taps=1)
    w = silence(random_weights(cfg, seed=9), "canon")
    w["l0.norm1"] = np.ones_like(w["l0.norm1"])
    h = w["embed"][2].astype(np.float64)
    z = np.tile(20.0 * h / np.sqrt((h ** 2).mean()) / width, (96, 1))
    w["l0.mix.z"], w["l0.mix.z.b"] = (binding.round_to_bf16(x.astype(np.float32)) for x in (z, np.full(96, -10.0)))
    w["l0.mix.x"], w["l0.mix.o"] = binding.round_to_bf16(w["l0.mix.x"] * 2), binding.round_to_bf16(w["l0.mix.o"] * 3)
    return cfg, w, [2] + np.random.default_rng(2).integers(3, 80, 899).tolist()


def test_long_recurrence_keeps_its_state(pkg, backend, dtype):
    """The state that the first token leaves is still there after hundreds of tokens."""
    cfg, w, t = long_memory()
    exp = metapel.forward(t, cfg, w)
    other = metapel.forward([3] + t[1:], cfg, w)
    assert worst_error(other[-1:], exp[-1:]) > 0.2, "the first token still shows at the end"
    for sizes in ([900], [300, 1], [5, 70, 2]):
        f = Feeder(pkg, make_model(pkg, backend, cfg, w, dtype))
        assert worst_error(f.run("p", t, sizes), exp) < tol(dtype), sizes


# ---- windows: one score that stands out ---------------------------------------------------------------

def beacon_model(window, heads=2, dim=16, rank=32, vdim=16, width=128):
    """One attention layer without convolutions in which token 1, as a query, is drawn to token 2 as a key, so
    that the value of token 2 dominates wherever it is visible; the other tokens are noise to each other."""
    cfg = config(width, 64, [latent(heads, dim, 16, vdim, rank, window)], taps=2)
    rng = np.random.default_rng(8)
    w = silence(random_weights(cfg, seed=8, gain=0.3), "canon")
    w["l0.mix.dkv"] = w["l0.mix.dkv"] * 5  # the latents of other tokens point elsewhere
    hq, hk = (w["embed"][i].astype(np.float64) for i in (1, 2))
    hq, hk = hq / np.sqrt((hq ** 2).mean()), hk / np.sqrt((hk ** 2).mean())
    c = rng.standard_normal(rank)
    u = rng.standard_normal((heads, dim))
    w["l0.norm1"] = np.ones_like(w["l0.norm1"])
    w["l0.mix.dkv.norm"] = np.ones_like(w["l0.mix.dkv.norm"])
    dkv = w["l0.mix.dkv"].astype(np.float64)
    dkv[:rank] += 6.0 * np.outer(c, hk) / width
    uk = w["l0.mix.uk"].astype(np.float64) + u.reshape(-1, 1) * c[None] / rank
    q = w["l0.mix.q"].astype(np.float64).reshape(heads, dim + 16, width)
    q[:, :dim] += 5.0 * u[:, :, None] * hq / width
    w["l0.mix.dkv"], w["l0.mix.uk"] = (binding.round_to_bf16(x.astype(np.float32)) for x in (dkv, uk))
    w["l0.mix.q"] = binding.round_to_bf16(q.reshape(-1, width).astype(np.float32))
    w["l0.mix.uv"] = binding.round_to_bf16(w["l0.mix.uv"] * 8)
    w["l0.mix.o"] = binding.round_to_bf16(w["l0.mix.o"] * 4)
    return cfg, w


@pytest.mark.parametrize("window", [1, 2, 15, 16, 17, 33, 64, 65, 200])
def test_window_edges(pkg, backend, dtype, window):
    """The far key sits just inside or just outside the window, at and around page borders, early and late in
    the sequence, in a prompt, in a portion and in decoding."""
    cfg, w = beacon_model(window)
    rng = np.random.default_rng(3)
    f = Feeder(pkg, make_model(pkg, backend, cfg, w, dtype))
    runs = 0
    for start in (0, 1, 15, 16, 31, 47, 100):
        for dist in (window - 1, window):
            t = rng.integers(3, 64, start + dist + 9)
            t[start], t[start + dist] = 2, 1
            t = t.tolist()
            exp = metapel.forward(t, cfg, w)
            if dist > 0:  # the key shows exactly when it is inside
                blind = list(t)
                blind[start] = 3
                shift = worst_error(metapel.forward(blind, cfg, w)[start + dist:start + dist + 1], exp[start + dist:start + dist + 1])
                assert (shift > 0.15) == (dist < window), (start, dist, shift)
            q = start + dist
            for sizes in ([len(t)], [max(q, 1), 1], [max(q - 1, 1), 3], [max(q - 5, 1), 12]):
                runs += 1
                name = f"{start}-{dist}-{runs}"
                assert worst_error(f.run(name, t, sizes), exp) < tol(dtype), (start, dist, sizes)


def test_a_far_key_among_hundreds(pkg, backend, dtype):
    cfg, w = beacon_model(700, heads=9, rank=64)
    t = np.random.default_rng(4).integers(3, 64, 760)
    t[[20, 130]] = 2
    t[[400, 650, 712, 719, 720, 759]] = 1
    t = t.tolist()
    exp = metapel.forward(t, cfg, w)
    for sizes in ([760], [640, 1], [128]):
        f = Feeder(pkg, make_model(pkg, backend, cfg, w, dtype))
        assert worst_error(f.run("p", t, sizes), exp) < tol(dtype), sizes


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


# ---- the model inside the framework -----------------------------------------------------------------

def greedy(cfg, w, prompt, n):
    out = list(prompt)
    for _ in range(n):
        out.append(int(np.argmax(metapel.forward(out, cfg, w)[-1])))
    return out[len(prompt):]


def follows_greedily(cfg, w, prompt, out, margin):
    """Every token is the plain implementation's best one after the tokens before it, up to `margin` logits."""
    logits = metapel.forward(prompt + out, cfg, w)
    for i, tok in enumerate(out):
        row = logits[len(prompt) - 1 + i]
        if row[tok] < row.max() - margin:
            return False
    return True


def run_engine(pkg, model, prompts, n, blocks, **cfg):
    E = pkg.engine
    kw = dict(max_num_seqs=8, max_num_batched_tokens=64, request_timeout_secs=None)
    kw.update(cfg)
    eng = E.Engine(model, E.SchedulerConfig(**kw), blocks, 16, True)
    ids = [eng.submit(p, E.SamplingParams(temperature=0.0, max_tokens=n)) for p in prompts]
    tokens = {i: [] for i in ids}
    for _ in range(2000):
        if not eng.has_work():
            break
        eng.step()
        for ev in eng.take_events():
            if ev.kind == "token":
                tokens[ev.id].append(ev.token)
    assert not eng.has_work()
    return [tokens[i] for i in ids], eng


@pytest.mark.parametrize("name", ["odd", "tuned"])
def test_generation_through_the_engine(pkg, backend, name, dtype):
    """Chunked prompts, continuous batching, more requests than state slots: the tokens of plain greedy decoding."""
    c = Case.get(name)
    rng = np.random.default_rng(6)
    prompts = [rng.integers(0, c.cfg["vocab"], k).tolist() for k in (3, 40, 90, 17, 1, 64)]
    model = make_model(pkg, backend, c.cfg, c.weights, dtype, tokens=64, seqs=4)
    out, eng = run_engine(pkg, model, prompts, 20, 64)
    for p, o in zip(prompts, out):
        assert len(o) == 20
        if dtype == pkg.DType.F32:
            assert o == greedy(c.cfg, c.weights, p, 20)
        assert follows_greedily(c.cfg, c.weights, p, o, 1e-3 if dtype == pkg.DType.F32 else 0.25)
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

    c = Case.get("tuned")
    (tmp_path / "config.json").write_text(json.dumps(c.cfg))
    pkg.write_safetensors(str(tmp_path / "model.safetensors"), c.weights, pkg.DType.BF16)
    assert pkg.model_class(str(tmp_path)) is pkg.CudaLayeredModel
    r = TraceRunner.from_directory(str(tmp_path), pkg.DType.F32, 256)
    got = r.step([{"id": "x", "tokens": c.tokens["b"], "want": [3, 96, 50]}], ["x"])
    assert worst_error(got, c.expected["b"][[3, 96, 50]]) < 3e-5
    del c.weights["l1.mix.uv"], c.cache["tuned"]
    pkg.write_safetensors(str(tmp_path / "model.safetensors"), c.weights, pkg.DType.BF16)
    with pytest.raises(pkg.ModelError, match="missing tensor `l1.mix.uv`"):
        pkg.load_model(str(tmp_path), 8, 16, backend)


def test_batches_that_do_not_continue_the_state_are_refused(pkg, backend):
    c = Case.get("odd")
    m = make_model(pkg, backend, c.cfg, c.weights, pkg.DType.F32)
    B = lambda pos, slots, counts=None: pkg.ForwardBatch(
        [1] * len(pos), pos, list(range(1, 1 + len(slots))), counts or [len(pos)], [p + 1 for p in pos][-len(slots):],
        [[i] for i in range(len(slots))], state_slots=slots)
    m.forward(B([0, 1, 2], [3]))
    with pytest.raises(pkg.InternalError, match="state covers 3 tokens"):
        m.forward(B([4], [3]))
    with pytest.raises(pkg.InternalError, match="not consecutive"):
        m.forward(B([3, 5], [3]))
    with pytest.raises(pkg.InternalError, match="named twice"):
        m.forward(B([0, 0], [2, 2], [1, 1]))
    with pytest.raises(pkg.InternalError, match="out of range"):
        m.forward(B([0], [99]))
    with pytest.raises(pkg.InvalidRequest, match="state slot"):
        m.forward(pkg.ForwardBatch([1], [0], [1], [1], [1], [[0]]))
    m.forward(B([3], [3]))  # the refused batches changed nothing


def test_step_graph_replays_the_same_logits(pkg, backend):
    """A decode layout that stays is replayed as a graph; the replays run through the same state copies."""
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
    f.step([("x", [t[140]]), ("y", [t[107]])])  # a replay leaves the sequences where they were
    assert worst_error(f.all("x"), c.expected["a"][:141]) < TOL["BF16"]


def test_logits_of_chosen_rows_for_the_transformer(pkg, backend):
    """The row list is a property of the step, not of one design: the Llama layout honours it too."""
    from drivers import C1_META, c1_tensors

    meta = pkg.ModelMetadata(architecture="llama", name="c1", **C1_META)
    m = pkg.CudaTransformerModel.new(meta, c1_tensors(seed=5), 16, 16, backend, compute_dtype=pkg.DType.F32,
                                     max_batch_tokens=64, max_batch_sequences=2)
    toks = list(range(3, 33))
    b = pkg.ForwardBatch(toks, list(range(30)), [1], [30], [30], [[3, 9]], logit_rows=[29, 4, 11])
    got = m.forward(b).logits
    for row, k in zip(got, (30, 5, 12)):
        exp = m.forward(pkg.ForwardBatch(toks[:k], list(range(k)), [1], [k], [k], [[3, 9]])).logits[0]
        assert np.allclose(row, exp, atol=1e-5)
    assert m.num_state_slots() == 0
