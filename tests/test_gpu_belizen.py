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


