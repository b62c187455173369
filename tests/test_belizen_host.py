"""Belizen without a GPU: the configuration reader and the registry, the plain implementation's mechanisms against hand-made
values, and that the test weights would show a fault in each of them."""
import json

import numpy as np
import pytest

from belizen_models import CONFIGS, ODD, attn, config, dense, gla, moe, random_weights, tensor_shapes, yarn
from metapel_models import worst_error
from oracle import belizen


def read(pkg, cfg, name="m"):
    return pkg.LayeredMetadata.from_config(json.loads(json.dumps(cfg)), name, tensor_shapes(cfg))


def test_config_is_read_field_by_field(pkg):
    cfg = config(40, 70, [attn(6, 3, 10, 14, 21, 6, dense(56), base=321.5, scale=0.31, rot_dims=4, yarn=yarn(3.0, 77, 9.0, 2.0), cap=4.5),
                          gla(3, 10, 12, 5.0, 9, moe(5, 2, 3, 12, 0.8, 30, 1.2)), attn(2, 1, 6, 4, None, 0, moe(3, 0, 1, 16, 2.0)), gla(2, 4, 6, 1.0, 2)],
                 eps=2e-4, mult=0.7, scale=3.5, loop=(1, 4, 3), cap=12.0)
    m = read(pkg, cfg)
    assert (m.architecture, m.hidden_size, m.vocab_size, m.norm_eps, m.num_layers) == ("Belizen", 40, 70, 2e-4, 4)
    assert (m.block, m.untied_lm_head, m.residual_mult, m.embed_scale, m.logit_softcap) == ("prenorm", False, 0.7, 3.5, 12.0)
    assert m.loop == pkg.Loop(1, 4, 3)
    own = dict(qk_norm="per_head", rope_halves=True, qkv_bias=True, value_gate=True)
    assert m.layers[0] == pkg.LayerSpec("attention", 56, heads=6, kv_heads=3, dim=10, value_dim=14, window=21, keep_first=6, rope_dims=4,
                                        rope_base=321.5, scale=0.31, softcap=4.5, yarn=pkg.Yarn(3.0, 77.0, 9.0, 2.0), activation="geglu_tanh", **own)
    assert m.layers[1] == pkg.LayerSpec("gla", 12, heads=3, dim=10, value_dim=12, decay_tau=5.0, decay_rank=9, experts=5, experts_per_token=3,
                                        router="softmax", router_identity=2, expert_form="clamped", expert_limit=0.8, shared_dim=30, shared_limit=1.2)
    assert m.layers[2].window == 0 and m.layers[2].shared_dim == 0 and m.layers[3].ffn_dim == 0
    assert [s.mixer for s in m.layer_runs()] == ["attention"] + ["gla", "attention", "gla"] * 3
    assert m.cache_values_per_token() == 3 * 24 + 3 * 10
    assert read(pkg, CONFIGS["broad"]).loop is None


@pytest.mark.parametrize("spoil", [
    lambda c: c["layers"][0].update(type="unknown"), lambda c: c["layers"][0]["mlp"].update(kind="other"), lambda c: c["layers"][0]["mixer"].pop("tau"),
    lambda c: c["layers"][1]["mixer"].pop("kv_heads"), lambda c: c.pop("residual_mult"), lambda c: c["norm"].pop("eps"), lambda c: c.pop("embedding"),
    lambda c: c["layers"][0].pop("mlp"), lambda c: c.update(layers=3), lambda c: c["layers"][1]["mlp"]["router"].pop("top"),
    lambda c: c["layers"][1]["mlp"]["expert"].pop("limit"), lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].pop("factor"),
    lambda c: c["loop"].update(stop=9), lambda c: c["loop"].update(times=0), lambda c: c.update(architecture="Other")])
def test_malformed_configs_are_refused(pkg, spoil):
    cfg = json.loads(json.dumps(ODD))
    spoil(cfg)
    with pytest.raises(pkg.ModelError):
        pkg.LayeredMetadata.from_config(cfg, "m", tensor_shapes(ODD))


def test_the_rank_of_the_decays_comes_from_the_checkpoint(pkg, tmp_path):
    (tmp_path / "config.json").write_text(json.dumps(ODD))
    assert pkg.model_class(str(tmp_path)) is pkg.CudaLayeredModel
    with pytest.raises(pkg.ModelError, match="missing tensor `l0.mix.a1`"):
        pkg.LayeredMetadata.load(str(tmp_path))
    w = random_weights(ODD)
    half = {n: x for n, x in w.items() if n < "l1"}
    pkg.write_safetensors(str(tmp_path / "a.safetensors"), half, pkg.DType.BF16)
    pkg.write_safetensors(str(tmp_path / "b.safetensors"), {n: x for n, x in w.items() if n not in half}, pkg.DType.BF16)
    assert [s.decay_rank for s in pkg.LayeredMetadata.load(str(tmp_path)).layers] == [3, 0, 5, 0]
    (tmp_path / "b.safetensors").write_bytes(b"short")
    with pytest.raises(pkg.ModelError, match="malformed"):
        pkg.LayeredMetadata.load(str(tmp_path))


# ---- the plain implementation ------------------------------------------------------------------------

def test_window_and_kept_tokens_by_hand():
    m = belizen.kept_window_mask(7, 2, 2)
    assert [list(np.flatnonzero(r)) for r in m] == [[0], [0, 1], [0, 1, 2], [0, 1, 2, 3], [0, 1, 3, 4], [0, 1, 4, 5], [0, 1, 5, 6]]
    assert belizen.kept_window_mask(3, None, 0).sum() == 6


def test_yarn_by_hand():
    f, mult = belizen.yarn_frequencies({"dims": 8, "base": 100.0, "scaling": yarn(4.0, 200.0, 10.0, 1.0)})
    # dimension by turns: 8 ln(200 / (2 pi t)) / (2 ln 100) = 1.005 for ten turns, 3.006 for one: pairs 0 and 1 stay, 2 and 3 are blended
    plain = 100.0 ** (-np.arange(4) / 4.0)
    ramp = np.array([0.0, 0.0, 1.0 / 3.0, 2.0 / 3.0])
    assert np.allclose(f, plain / 4 * ramp + plain * (1 - ramp)) and np.isclose(mult, 0.1 * np.log(4.0) + 1.0)
    assert np.allclose(belizen.yarn_frequencies({"dims": 8, "base": 100.0})[0], plain)


def test_halves_turn_together():
    x = np.zeros((2, 1, 6))
    x[1, 0] = [1.0, 0.0, 0.0, 2.0, 5.0, 6.0]
    out = belizen.rotate_halves(x, np.arange(2), np.array([np.pi / 2, 0.0]), 2.0)
    assert np.allclose(out[1, 0], [0.0, 0.0, 2.0, 4.0, 5.0, 6.0])


def test_linear_attention_by_hand():
    """One channel: the state halves, gains k v, and is read by q."""
    o = belizen.gla_scan(np.array([[1.0], [2.0], [1.0]]), np.array([[1.0], [1.0], [0.0]]), np.array([[4.0], [6.0], [9.0]]), np.full((3, 1), 0.5))
    assert o.ravel().tolist() == [4.0, 2.0 * (2.0 + 6.0), 4.0]
    w = {"a1": np.array([[2.0]]), "a2": np.array([[0.5]]), "a2.b": np.array([-1.0])}
    assert np.allclose(belizen.decays(np.array([[1.0]]), w, 4.0), 0.5 ** 0.25)


def test_choice_by_corrected_scores_weights_by_plain_ones():
    h, w = np.ones((1, 1)), {"router": np.log(np.array([[4.0], [3.0], [2.0], [1.0]])), "correction": np.array([-0.3, 0.0, 0.0, 0.25])}
    chosen, weight = belizen.route(h, w, 2)
    assert chosen.tolist() == [[3, 1]] and np.allclose(weight, [[0.1, 0.3]])


def test_identity_and_clamped_experts_by_hand():
    w = {"router": np.array([[0.0], [np.log(3.0)]]), "correction": np.zeros(2), "e0.gate": np.array([[5.0]]), "e0.up": np.array([[-7.0]]), "e0.down": np.array([[1.0]])}
    out = belizen.mixture(np.array([[1.0]]), w, {"router": {"experts": 1, "identity": 1, "top": 2}, "expert": {"limit": 2.0}, "shared": None})
    assert np.allclose(out, 0.75 * 1.0 + 0.25 * (2.0 / (1 + np.exp(-3.404))) * (-2.0 + 1.0))


def test_order_of_layer_runs():
    assert belizen.layer_runs({"layers": [0] * 4, "loop": {"start": 1, "stop": 3, "times": 2}}) == [(0, None), (1, 0), (2, 0), (1, 1), (2, 1), (3, None)]


# ---- faults that the test weights have to show --------------------------------------------------------

def _renormalised(h, w, top, real=belizen.route):
    chosen, weight = real(h, w, top)
    return chosen, weight / weight.sum(axis=1, keepdims=True)


def _corrected_weights(h, w, top, real=belizen.route):
    chosen, weight = real(h, w, top)
    return chosen, weight + w["correction"][chosen]


def _neighbours(x, positions, freq, mult):
    n = len(freq)
    order = np.concatenate([np.arange(2 * n).reshape(-1, 2).T.ravel(), np.arange(2 * n, x.shape[-1])])
    out = np.empty_like(x)
    out[..., order] = ROTATE(x[..., order], positions, freq, mult)
    return out


def _without_identity(h, w, mlp, real=belizen.mixture):
    n = mlp["router"]["experts"]
    w = dict(w)
    for e in range(n, n + mlp["router"]["identity"]):  # experts that return nothing
        w.update({f"e{e}.{part}": 0 * w[f"e0.{part}"] for part in ("gate", "up", "down")})
    return real(h, w, {**mlp, "router": {**mlp["router"], "experts": n + mlp["router"]["identity"]}})


def _plain_swiglu(h, w, name, limit):
    g, u = np.minimum(h @ w[name + ".gate"].T, limit), np.clip(h @ w[name + ".up"].T, -limit, limit)
    return (g / (1 + np.exp(-1.702 * g)) * u) @ w[name + ".down"].T


ROTATE, SCAN, MASK, YARN, EXPERT = belizen.rotate_halves, belizen.gla_scan, belizen.kept_window_mask, belizen.yarn_frequencies, belizen.clamped_expert
FAULTS = {
    "window one token larger": ("kept_window_mask", lambda T, size, keep: MASK(T, size and size + 1, keep), "odd"),
    "one kept token fewer": ("kept_window_mask", lambda T, size, keep: MASK(T, size, max(keep - 1, 0)), "odd"),
    "one kept token more": ("kept_window_mask", lambda T, size, keep: MASK(T, size, keep + 1 if keep else 0), "odd"),
    "neighbours rotated together": ("rotate_halves", _neighbours),
    "frequencies not stretched": ("yarn_frequencies", lambda rot: (YARN({**rot, "scaling": None})[0], YARN(rot)[1])),
    "rotation not scaled": ("yarn_frequencies", lambda rot: (YARN(rot)[0], 1.0)),
    "no soft cap": ("softcap", lambda x, cap: x),
    "state lost at a chunk": ("gla_scan", lambda q, k, v, a: np.concatenate([SCAN(*(x[i:i + 64] for x in (q, k, v, a))) for i in range(0, len(q), 64)])),
    "decay of the row before": ("gla_scan", lambda q, k, v, a: SCAN(q, k, v, np.concatenate([a[:1], a[:-1]]))),
    "state read before the row": ("gla_scan", lambda q, k, v, a: SCAN(q, k, v, a) - (q * k).sum(1, keepdims=True) * v),
    "one decay for all channels": ("gla_scan", lambda q, k, v, a: SCAN(q, k, v, np.repeat(a.mean(1, keepdims=True), a.shape[1], 1))),
    "weights renormalised": ("route", _renormalised),
    "correction in the weights": ("route", _corrected_weights),
    "correction left out": ("route", lambda h, w, top, real=belizen.route: real(h, {**w, "correction": 0 * w["correction"]}, top)),
    "identity experts return nothing": ("mixture", _without_identity),
    "no limits": ("clamped_expert", lambda h, w, name, limit: EXPERT(h, w, name, 1e9)),
    "up without its one": ("clamped_expert", _plain_swiglu),
    "silu for gelu": ("gelu_tanh", lambda x: x / (1 + np.exp(-x))),
    "start not added again": ("before_pass", lambda x, start, t, step: x + step[t]),
    "vector of the first pass": ("before_pass", lambda x, start, t, step: x + (start if t else 0.0) + step[0]),
}


@pytest.mark.parametrize("fault", sorted(FAULTS))
def test_weights_show_faults(monkeypatch, fault):
    name, fn, which = (FAULTS[fault] + ("tuned",))[:3]
    cfg = CONFIGS[which]
    w = random_weights(cfg, seed=5)
    t = np.random.default_rng(3).integers(0, cfg["vocab"], 130).tolist()
    exp = belizen.forward(t, cfg, w)
    monkeypatch.setattr(belizen, name, fn)
    assert worst_error(belizen.forward(t, cfg, w), exp) > 0.04


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_routers_of_the_test_weights_are_decisive(monkeypatch, name):
    """Rounding does not change an expert, the experts do change from token to token, and the correction changes the choice."""
    cfg = CONFIGS[name]
    w = random_weights(cfg, seed=len(name))
    gaps, used, turned = [], set(), []

    def watched(h, wl, top, real=belizen.route):
        chosen, weight = real(h, wl, top)
        if top < len(wl["router"]):
            z = h @ wl["router"].T
            s = np.exp(z - z.max(axis=1, keepdims=True))
            s = np.sort(s / s.sum(axis=1, keepdims=True) + wl["correction"], axis=1)
            gaps.append((s[:, -top] - s[:, -top - 1]).min())
            plain = np.argsort(-z, axis=1, kind="stable")[:, :top]
            turned.append((np.sort(plain, axis=1) != np.sort(chosen, axis=1)).any(axis=1).mean())
        used.update((len(wl["router"]), int(e)) for e in chosen.ravel())
        return chosen, weight

    monkeypatch.setattr(belizen, "route", watched)
    belizen.forward(np.random.default_rng(17).integers(0, cfg["vocab"], 230).tolist(), cfg, w)
    assert min(gaps) > 0.02 and len(used) >= 5
    assert max(turned) > 0.02


def test_every_tensor_has_a_shape_the_reader_expects(pkg):
    """The tests' list of tensors covers each layer's kind once."""
    names = set(tensor_shapes(CONFIGS["odd"]))
    assert {"loop.step", "l0.mlp.gate", "l0.mix.a2.b", "l1.mlp.router", "l1.mlp.correction", "l1.mlp.e4.gate", "l1.mlp.shared.down", "l1.mix.q.b"} <= names
    assert "l2.norm2" not in names and "l1.mlp.e5.up" not in names and "head" not in names
