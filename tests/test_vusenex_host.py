"""Vusenex without a GPU: the configuration reader and the registry, the plain implementation's mechanisms against hand-made
values, and that the test weights would show a fault in each of them."""
import json

import numpy as np
import pytest

from metapel_models import worst_error
from oracle import vusenex
from vusenex_models import CONFIGS, ODD, attn, config, gaps, latent, moe, random_weights, tensor_shapes


def read(pkg, cfg, name="m"):
    return pkg.LayeredMetadata.from_config(json.loads(json.dumps(cfg)), name, tensor_shapes(cfg))


def test_config_is_read_field_by_field(pkg):
    cfg = config(40, 70, [attn(6, 3, 10, moe(8, 4, 3, 5, 12, 30), temp=(0.25, 17), scale=0.31), latent(3, 10, 12, 9, moe(5, 0, 0, 3, 14), scale=0.4),
                          attn(2, 1, 6, None, temp=None)], eps=2e-4, pairs=(77, 5, 3), positions=123)
    m = read(pkg, cfg)
    assert (m.architecture, m.hidden_size, m.vocab_size, m.norm_eps, m.num_layers) == ("Vusenex", 40, 70, 2e-4, 3)
    assert (m.block, m.untied_lm_head, m.scalar_norms, m.max_positions, m.residual_mult) == ("gated_postnorm", True, True, 123, 1.0)
    assert m.bigram == pkg.Bigram(77, 5, 3)
    own = dict(qk_norm=True, qkv_bias=True, sinks="zero", keys_as_values=True, distance_bias=True)
    mix = dict(router="softmax_renorm", expert_form="gelu")
    assert m.layers[0] == pkg.LayerSpec("attention", 12, heads=6, kv_heads=3, dim=10, value_dim=10, scale=0.31, experts=8, experts_per_token=5,
                                        shared_dim=30, router_groups=4, router_keep=3, q_temp=pkg.QueryTemperature(0.25, 17.0), **own, **mix)
    assert m.layers[1] == pkg.LayerSpec("latent_attention", 14, heads=3, dim=10, value_dim=12, kv_rank=9, scale=0.4, ungated=True, experts=5,
                                        experts_per_token=3, **mix)
    assert m.layers[2].q_temp is None and m.layers[2].ffn_dim == 0
    assert m.cache_values_per_token() == 30 + 9 + 6


@pytest.mark.parametrize("spoil", [
    lambda c: c["layers"][0].update(type="unknown"), lambda c: c["layers"][0]["mlp"].update(kind="dense"), lambda c: c["layers"][0]["mixer"].pop("kv_rank"),
    lambda c: c["layers"][1]["mixer"].pop("kv_heads"), lambda c: c.pop("max_positions"), lambda c: c["norm"].pop("eps"), lambda c: c.pop("embedding"),
    lambda c: c["embedding"]["bigram"].pop("mul_prev"), lambda c: c["layers"][0].pop("mlp"), lambda c: c.update(layers=3),
    lambda c: c["layers"][1]["mlp"]["router"].pop("top"), lambda c: c["layers"][1]["mlp"]["expert"].pop("ff"), lambda c: c["layers"][1]["mixer"].update(vdim=11),
    lambda c: c["layers"][1]["mixer"]["q_temp"].pop("every"), lambda c: c["layers"][1]["mlp"]["router"]["groups"].pop("keep"),
    lambda c: c.update(architecture="Other")])
def test_malformed_configs_are_refused(pkg, spoil):
    cfg = json.loads(json.dumps(ODD))
    spoil(cfg)
    with pytest.raises(pkg.ModelError):
        pkg.LayeredMetadata.from_config(cfg, "m", tensor_shapes(ODD))


def test_single_numbers_keep_their_rank_in_a_checkpoint(pkg, tmp_path):
    (tmp_path / "config.json").write_text(json.dumps(ODD))
    assert pkg.model_class(str(tmp_path)) is pkg.CudaLayeredModel
    w = random_weights(ODD)
    pkg.write_safetensors(str(tmp_path / "m.safetensors"), w, pkg.DType.BF16)
    back = pkg.read_safetensors(str(tmp_path / "m.safetensors"))
    assert back["l0.norm1"][1] == () and back["l0.rg1.b"][1] == (50,)
    assert pkg.LayeredMetadata.load(str(tmp_path)).layers[1].heads == 3


# ---- the plain implementation ------------------------------------------------------------------------

def test_rows_of_pairs_by_hand():
    assert vusenex.bigram_rows([4, 2, 2], {"buckets": 10, "mul_prev": 3, "mul_cur": 7}) == [10, (12 + 14) % 10, (6 + 14) % 10]


def test_query_factor_by_hand():
    f = vusenex.query_factor(7, {"coef": 0.5, "every": 3})
    assert np.allclose(f, 1 + 0.5 * np.log([1, 1, 2, 2, 2, 3, 3]))
    assert vusenex.query_factor(3, None).tolist() == [1.0, 1.0, 1.0]


def test_distance_bias_by_hand():
    b = vusenex.distance_bias(3, 2.0, 4.0)
    assert np.allclose(b[2], [2 * np.log(9.0), 2 * np.log(5.0), 0.0])


def test_softmax_plus_one_by_hand():
    p = vusenex.softmax_plus_one(np.log(np.array([[1.0, 9.0], [2.0, 3.0]])), vusenex.causal(2))
    assert np.allclose(p, [[0.5, 0.0], [2 / 6, 3 / 6]])
    assert np.allclose(vusenex.softmax_plus_one(np.array([[-2000.0]]), np.ones((1, 1), bool)), 0.0)


def test_gelu_by_hand():
    assert np.allclose(vusenex.gelu(np.array([0.0, 1.0, -2.0])), [0.0, 0.8413447460685429, -2 * 0.02275013194817921])


def test_choice_among_the_best_groups():
    """Expert 1 has the third largest score but stands in a group whose best is only third."""
    z = np.log(np.array([[1.0, 7.0, 2.0, 9.0, 8.0, 3.0]]))
    chosen, weight = vusenex.route(np.ones((1, 1)), z.T, {"top": 3, "groups": {"count": 3, "keep": 2}})
    assert chosen.tolist() == [[3, 4, 5]] and np.allclose(weight, [[0.45, 0.4, 0.15]])
    chosen, _ = vusenex.route(np.ones((1, 1)), z.T, {"top": 3})
    assert chosen.tolist() == [[3, 4, 1]]


def test_values_are_the_keys_before_their_norm():
    """One head, one key: its weight is e^s / (1 + e^s), its value the projection with its bias."""
    h = np.array([[1.0, 0.0]])
    w = {"q": np.eye(2), "k": 2 * np.eye(2), "q.b": np.zeros(2), "k.b": np.array([0.0, 2.0]), "q.norm": np.ones(2), "k.norm": np.array([3.0, 0.0]),
         "r1": np.ones(1), "r2": np.ones(1), "o": np.eye(2)}
    out = vusenex.attention(h, w, {"heads": 1, "kv_heads": 1, "dim": 2, "scale": 0.5}, 0.0)
    s = 0.5 * np.sqrt(2.0) * 3.0
    assert np.allclose(out, np.exp(s) / (1 + np.exp(s)) * np.array([[2.0, 2.0]]))


# ---- faults that the test weights have to show --------------------------------------------------------

ATTEND, MASKED, PLUS_ONE, BIAS, FACTOR, ROUTE, GATED, ROWS = (vusenex.attention, vusenex.softmax_masked, vusenex.softmax_plus_one, vusenex.distance_bias,
                                                             vusenex.query_factor, vusenex.route, vusenex.gated, vusenex.bigram_rows)


def _normed_values(h, w, m, eps):
    """The values taken after the norm of the keys."""
    k = h @ w["k"].T + w["k.b"]
    s = 1.0 / np.sqrt((k * k).mean(axis=1, keepdims=True) + eps) * w["k.norm"]
    T, H, G, D = len(h), m["heads"], m["kv_heads"], m["dim"]
    q = (vusenex.rms_norm(h @ w["q"].T + w["q.b"], w["q.norm"], eps).reshape(T, H, D) * FACTOR(T, m.get("q_temp"))[:, None, None])
    k = (k * s).reshape(T, G, D)
    out = np.empty((T, H, D))
    for a in range(H):
        b = a // (H // G)
        out[:, a] = PLUS_ONE(q[:, a] @ k[:, b].T * m["scale"] - BIAS(T, w["r1"][a], w["r2"][a]), vusenex.causal(T)) @ k[:, b]
    return out.reshape(T, H * D) @ w["o"].T


def _norm_per_head(x, w, eps, real=vusenex.rms_norm):
    """Attention's norms over heads of 48 or 64 instead of all of them at once."""
    if np.ndim(w) != 1 or w.size not in (704, 288):
        return real(x, w, eps)
    d = 64 if w.size == 704 else 48
    return real(x.reshape(len(x), -1, d), w.reshape(-1, d), eps).reshape(len(x), -1)


def _latent_as_it_is(x, w, eps, real=vusenex.rms_norm):
    """No norm where the gains are those of a latent (of 64 or 96 values; gains of keys are larger on average)."""
    return x * w if np.ndim(w) == 1 and w.size in (64, 96) and w.mean() < 1.3 else real(x, w, eps)


def _without(*names):
    def fn(h, w, m, eps):
        return ATTEND(h, {**w, **{n: 0 * w[n] for n in names}}, m, eps)
    return fn


def _group_sum(s, g):
    if not g:
        return np.ones(s.shape, bool)
    best = s.reshape(len(s), g["count"], -1).sum(axis=-1)
    kept = np.zeros(best.shape, bool)
    np.put_along_axis(kept, np.argsort(-best, axis=-1, kind="stable")[:, :g["keep"]], True, axis=-1)
    return np.repeat(kept, s.shape[1] // g["count"], axis=1)


def _strided_groups(s, g, real=vusenex.eligible):
    if not g:
        return np.ones(s.shape, bool)
    order = np.arange(s.shape[1]).reshape(-1, g["count"]).T.ravel()  # experts e, e + count, ... form a group
    out = np.empty(s.shape, bool)
    out[:, order] = real(s[:, order], g)
    return out


FAULTS = {
    "values after the norm": ("attention", _normed_values),
    "no bias of the keys": ("attention", _without("k.b")),
    "no bias of the queries": ("attention", _without("q.b")),
    "norms per head": ("rms_norm", _norm_per_head),
    "sink left out": ("softmax_plus_one", MASKED),
    "sink with the score one": ("softmax_plus_one", lambda s, m: PLUS_ONE(s - 1.0, m)),
    "no distance term": ("distance_bias", lambda T, r1, r2: 0.0 * BIAS(T, r1, r2)),
    "distance one too large": ("distance_bias", lambda T, r1, r2: r1 * np.log(1 + r2 * (np.maximum(np.arange(T)[:, None] - np.arange(T), 0) + 1.0))),
    "distance term linear": ("distance_bias", lambda T, r1, r2: r1 * r2 * np.maximum(np.arange(T)[:, None] - np.arange(T), 0)),
    "query factor left out": ("query_factor", lambda T, temp: np.ones(T)),
    "query factor one position late": ("query_factor", lambda T, temp: np.concatenate([[1.0], FACTOR(T, temp)[:-1]]), "odd"),
    "heads of a group interleaved": ("attention", lambda h, w, m, eps: ATTEND(h, {**w, "k": np.roll(w["k"], m["dim"], axis=0)}, m, eps)),
    "norm of the latent left out": ("rms_norm", _latent_as_it_is),
    "pairs the other way round": ("bigram_rows", lambda t, b: ROWS(t, {**b, "mul_prev": b["mul_cur"], "mul_cur": b["mul_prev"]})),
    "first token with a predecessor 0": ("bigram_rows", lambda t, b: [t[0] * b["mul_cur"] % b["buckets"]] + ROWS(t, b)[1:]),
    "predecessor lost at a portion": ("bigram_rows", lambda t, b: [b["buckets"] if i % 64 == 0 else r for i, r in enumerate(ROWS(t, b))]),
    "positions from one": ("embedding", lambda t, c, w, d, real=vusenex.embedding: real(t, c, {**w, "pos": w["pos"][1:]}, d)),
    "no positions": ("embedding", lambda t, c, w, d, real=vusenex.embedding: real(t, c, {**w, "pos": 0 * w["pos"]}, d)),
    "gates left out": ("gated", lambda y, h, m, b: y),
    "gates without bias": ("gated", lambda y, h, m, b: GATED(y, h, m, 0 * b)),
    "weights not renormalised": ("route", lambda h, m, r: (ROUTE(h, m, r)[0], ROUTE(h, m, r)[1] * 0.8)),
    "groups ignored": ("eligible", lambda s, g: np.ones(s.shape, bool)),
    "groups by the sum of their scores": ("eligible", _group_sum, "broad"),
    "groups of every n-th expert": ("eligible", _strided_groups),
    "silu for gelu": ("gelu", lambda x: x / (1 + np.exp(-x))),
    "shared expert left out": ("mixture", lambda h, w, mlp, real=vusenex.mixture: real(h, w, {**mlp, "shared": None})),
}


@pytest.mark.parametrize("fault", sorted(FAULTS))
def test_weights_show_faults(monkeypatch, fault):
    name, fn, which = (FAULTS[fault] + ("tuned",))[:3]
    cfg = CONFIGS[which]
    w = random_weights(cfg, seed=5)
    t = np.random.default_rng(3).integers(0, cfg["vocab"], 130).tolist()
    exp = vusenex.forward(t, cfg, w)
    monkeypatch.setattr(vusenex, name, fn)
    assert worst_error(vusenex.forward(t, cfg, w), exp) > 0.04


def test_weights_show_a_gate_after_the_norm(monkeypatch):
    cfg = CONFIGS["tuned"]
    w = random_weights(cfg, seed=5)
    t = np.random.default_rng(3).integers(0, cfg["vocab"], 130).tolist()
    exp = vusenex.forward(t, cfg, w)

    def layer(x, i, config, weights):
        spec, eps = config["layers"][i], config["norm"]["eps"]
        lw = vusenex._sub(weights, f"l{i}.", x.dtype)
        mixer = {"attention": vusenex.attention, "latent_attention": vusenex.latent_attention}[spec["type"]]
        x = x + GATED(vusenex.rms_norm(mixer(x, vusenex._sub(lw, "mix.", x.dtype), spec["mixer"], eps), lw["norm1"], eps), x, lw["rg1"], lw["rg1.b"])
        if spec["mlp"] is not None:
            x = x + GATED(vusenex.rms_norm(vusenex.mixture(x, vusenex._sub(lw, "mlp.", x.dtype), spec["mlp"]), lw["norm2"], eps), x, lw["rg2"], lw["rg2.b"])
        return x

    monkeypatch.setattr(vusenex, "layer", layer)
    assert worst_error(vusenex.forward(t, cfg, w), exp) > 0.04


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_routers_of_the_test_weights_are_decisive(monkeypatch, name):
    """Rounding does not change an expert or a group, the experts do change from token to token, and the groups change the choice."""
    cfg = CONFIGS[name]
    w = random_weights(cfg, seed=len(name))
    seen, used, turned = [], set(), []

    def watched(h, matrix, router, real=vusenex.route):
        chosen, weight = real(h, matrix, router)
        z = h @ matrix.T
        seen.extend(gaps(row, router) for row in z)
        if router["groups"] and router["groups"]["keep"] < router["groups"]["count"]:
            free = np.argsort(-z, axis=1, kind="stable")[:, :router["top"]]
            turned.append((np.sort(free, axis=1) != np.sort(chosen, axis=1)).any(axis=1).mean())
        used.update((len(matrix), int(e)) for e in chosen.ravel())
        return chosen, weight

    monkeypatch.setattr(vusenex, "route", watched)
    vusenex.forward(np.random.default_rng(17).integers(0, cfg["vocab"], 230).tolist(), cfg, w)
    assert min(seen) > 0.1 and len(used) >= 5
    assert name == "wide" or max(turned) > 0.05


def test_every_tensor_has_a_shape_the_reader_expects(pkg):
    """The tests' list of tensors covers each layer's kind once."""
    names = set(tensor_shapes(CONFIGS["odd"]))
    assert {"bigram", "pos", "head", "l0.mix.uk", "l0.mlp.shared.down", "l1.mix.r2", "l1.mix.k.b", "l1.mlp.e4.up", "l0.rg2.b", "l3.norm2"} <= names
    assert not names & {"l2.norm2", "l2.rg2", "l1.mlp.e5.up", "l1.mlp.shared.up", "l1.mix.v", "l0.mix.g", "l0.mlp.e0.gate"}
