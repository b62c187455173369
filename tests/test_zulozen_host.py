"""Zulozen without a GPU: the configuration reader and the registry, the plain implementation's mechanisms against hand-made
values, and that the test weights would show a fault in each of them."""
import json

import numpy as np
import pytest

from metapel_models import worst_error
from oracle import zulozen
from zulozen_models import CONFIGS, ODD, attn, config, dense, moe, random_weights, tensor_shapes


def test_config_is_read_field_by_field(pkg):
    cfg = config(40, 70, [attn(6, 3, 10, 14, 21, dense(56), base=321.5, scale=0.31, rot_dims=4), attn(4, 4, 8, 8, None, moe(5, 2, 12, 30)),
                          attn(2, 1, 6, 4, 7), attn(2, 1, 6, 4, 7, moe(3, 1, 16))], eps=2e-4, mult=0.7)
    m = pkg.LayeredMetadata.from_config(json.loads(json.dumps(cfg)), "m")
    assert (m.architecture, m.hidden_size, m.vocab_size, m.norm_eps, m.num_layers) == ("Zulozen", 40, 70, 2e-4, 4)
    assert (m.block, m.untied_lm_head, m.residual_mult) == ("sandwich", True, 0.7)
    own = dict(qk_norm=True, sinks=True, head_gate=True)
    assert m.layers[0] == pkg.LayerSpec("attention", 56, heads=6, kv_heads=3, dim=10, value_dim=14, chunk=21, rope_dims=4, rope_base=321.5,
                                        scale=0.31, activation="relu2", ffn_bias=True, **own)
    assert m.layers[1] == pkg.LayerSpec("attention", 12, heads=4, kv_heads=4, dim=8, value_dim=8, rope_dims=4, rope_base=10000.0,
                                        scale=8 ** -0.5, experts=5, experts_per_token=2, shared_dim=30, **own)
    assert m.layers[2].ffn_dim == 0 and m.layers[3].shared_dim == 0
    assert m.cache_values_per_token() == 3 * 24 + 4 * 16 + 10 + 10


@pytest.mark.parametrize("spoil", [
    lambda c: c["layers"][0].update(type="unknown"), lambda c: c["layers"][0]["mlp"].update(kind="other"),
    lambda c: c["layers"][1]["mixer"].pop("kv_heads"), lambda c: c.pop("residual_mult"), lambda c: c["norm"].pop("eps"),
    lambda c: c["layers"][0].pop("mlp"), lambda c: c.update(layers=3), lambda c: c["layers"][1]["mlp"]["router"].pop("top"),
    lambda c: c.update(architecture="Other")])
def test_malformed_configs_are_refused(pkg, spoil):
    cfg = json.loads(json.dumps(ODD))
    spoil(cfg)
    with pytest.raises(pkg.ModelError):
        pkg.LayeredMetadata.from_config(cfg)


def test_registry_picks_the_class(pkg, tmp_path):
    (tmp_path / "config.json").write_text(json.dumps(ODD))
    assert pkg.model_class(str(tmp_path)) is pkg.CudaLayeredModel


# ---- the plain implementation ------------------------------------------------------------------------

def test_chunks_are_counted_from_the_start():
    m = zulozen.chunk_mask(7, 3)
    assert [list(np.flatnonzero(r)) for r in m] == [[0], [0, 1], [0, 1, 2], [3], [3, 4], [3, 4, 5], [6]]
    assert zulozen.chunk_mask(3, None).sum() == 6


def test_sink_takes_its_share_once():
    s = np.log(np.array([[3.0, 5.0, 100.0]]))
    p = zulozen.softmax_with_sink(s, np.array([[True, True, False]]), np.log(2.0))
    assert np.allclose(p, [[0.3, 0.5, 0.0]])


def test_scores_choose_and_weigh_without_normalisation():
    router = np.diag([1.0, 2.0, 3.0, -4.0])
    chosen, score = zulozen.route(np.array([[1.0, 1.0, 1.0, 1.0]]), router, 2)
    assert chosen.tolist() == [[2, 1]] and np.allclose(score, [[1 / (1 + np.exp(-3)), 1 / (1 + np.exp(-2))]])
    # equal scores: the lower index
    assert zulozen.route(np.ones((1, 3)), np.ones((4, 3)), 3)[0].tolist() == [[0, 1, 2]]


def test_the_score_multiplies_what_the_expert_reads():
    w = {"router": np.array([[0.0], [-9.0]]), "e0.gate": np.array([[2.0]]), "e0.up": np.array([[1.0]]), "e0.down": np.array([[1.0]]),
         "e1.gate": np.array([[7.0]]), "e1.up": np.array([[7.0]]), "e1.down": np.array([[7.0]])}
    out = zulozen.mixture(np.array([[3.0]]), w, {"router": {"experts": 2, "top": 1}, "expert": {"ff": 1}, "shared": None})
    h = 0.5 * 3.0
    assert np.allclose(out, 2 * h / (1 + np.exp(-2 * h)) * h)


def test_dense_feed_forward_by_hand():
    w = {"up": np.array([[1.0], [-1.0]]), "up.b": np.array([0.5, 1.0]), "down": np.array([[2.0, 10.0]]), "down.b": np.array([-3.0])}
    assert zulozen.dense_relu2(np.array([[2.0]]), w).tolist() == [[2 * 2.5 ** 2 - 3.0]]


def test_norm_spans_all_heads():
    """Scaling one head's queries changes what the others come out as."""
    cfg = config(32, 20, [attn(2, 2, 8, 8, 9)])
    w = random_weights(cfg, seed=1)
    t = list(range(9))
    exp = zulozen.forward(t, cfg, w)
    w["l0.mix.q"] = w["l0.mix.q"].copy()
    w["l0.mix.q"][:8] *= 8
    assert worst_error(zulozen.forward(t, cfg, w), exp) > 0.02


# ---- faults that the test weights have to show --------------------------------------------------------

def _no_gate(x):
    return np.ones_like(x) if x.ndim == 2 and x.shape[1] < 25 else 1.0 / (1.0 + np.exp(-x))


def _scored_output(h, w, mlp):
    chosen, score = zulozen.route(h, w["router"], mlp["router"]["top"])
    out = zulozen.expert(h, w, "shared") if mlp.get("shared") else np.zeros_like(h)
    for t in range(len(h)):
        for e, s in zip(chosen[t], score[t]):
            out[t] += s * zulozen.expert(h[t:t + 1], w, f"e{e}")[0]
    return out


def _renormalised(h, router, top, real=zulozen.route):
    chosen, score = real(h, router, top)
    return chosen, score / score.sum(axis=1, keepdims=True)


def _halves(x, positions, base, dims):
    """Dimension i rotated with dimension i + dims / 2."""
    order = np.concatenate([np.arange(dims).reshape(2, -1).T.ravel(), np.arange(dims, x.shape[-1])])
    out = np.empty_like(x)
    out[..., order] = ROTATE(x[..., order], positions, base, dims)
    return out


ROTATE = zulozen.rotate_interleaved
FAULTS = {
    "sink left out": ("softmax_with_sink", lambda s, m, sink, real=zulozen.softmax_with_sink: real(s, m, -np.inf)),
    "sink counted twice": ("softmax_with_sink", lambda s, m, sink, real=zulozen.softmax_with_sink: real(s, m, sink + np.log(2.0))),
    "chunk one token larger": ("chunk_mask", lambda T, size, real=zulozen.chunk_mask: real(T, size and size + 1)),
    "window instead of chunk": ("chunk_mask", lambda T, size: np.tril(np.ones((T, T), bool)) & (
        np.arange(T)[:, None] - np.arange(T)[None, :] < (size or T))),
    "halves rotated together": ("rotate_interleaved", _halves),
    "score on the output": ("mixture", _scored_output),
    "scores renormalised": ("route", _renormalised),
    "one expert fewer": ("route", lambda h, r, top, real=zulozen.route: tuple(x[:, :max(top - 1, 1)] for x in real(h, r, top))),
    "relu not squared": ("dense_relu2", lambda h, w: np.maximum(h @ w["up"].T + w["up.b"], 0.0) @ w["down"].T + w["down.b"]),
    "bias left out": ("dense_relu2", lambda h, w: np.maximum(h @ w["up"].T + w["up.b"], 0.0) ** 2 @ w["down"].T),
    "gate left out": ("sigmoid", _no_gate),
}


@pytest.mark.parametrize("fault", sorted(FAULTS))
def test_weights_show_faults(monkeypatch, fault):
    cfg, name = CONFIGS["tuned"], FAULTS[fault][0]
    w = random_weights(cfg, seed=5)
    t = np.random.default_rng(3).integers(0, cfg["vocab"], 110).tolist()
    exp = zulozen.forward(t, cfg, w)
    monkeypatch.setattr(zulozen, name, FAULTS[fault][1])
    assert worst_error(zulozen.forward(t, cfg, w), exp) > 0.06


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_routers_of_the_test_weights_are_decisive(monkeypatch, name):
    """Rounding does not change an expert, and the experts do change from token to token."""
    cfg = CONFIGS[name]
    w = random_weights(cfg, seed=len(name))
    gaps, used = [], set()

    def watched(h, router, top, real=zulozen.route):
        z = np.sort(h @ router.T, axis=1)
        if top < len(router):
            gaps.append((z[:, -top] - z[:, -top - 1]).min())
        chosen, score = real(h, router, top)
        used.update(chosen.ravel().tolist())
        return chosen, score

    monkeypatch.setattr(zulozen, "route", watched)
    zulozen.forward(np.random.default_rng(17).integers(0, cfg["vocab"], 230).tolist(), cfg, w)
    assert min(gaps) > 0.1 and len(used) >= 5


def test_every_tensor_has_a_shape_the_reader_expects(pkg):
    """The tests' list of tensors covers each layer's kind once."""
    names = set(tensor_shapes(CONFIGS["odd"]))
    assert {"l0.mlp.up.b", "l1.mlp.router", "l1.mlp.e4.gate", "l1.mlp.shared.down", "l3.mlp.e2.down", "head"} <= names
    assert "l2.norm2" not in names and "l3.mlp.shared.gate" not in names
