"""Metapel without a GPU: the configuration reader and the registry, the plain implementation's mechanisms against
hand-made values, state slots in the cache manager, recomputation after preemption in the scheduler, and the trace
replay around a model that keeps its state on the host."""
import json

import numpy as np
import pytest

from metapel_models import CONFIGS, ODD, TUNED, config, latent, mingru, random_weights, tensor_shapes, worst_error
from oracle import metapel


# ---- configuration -----------------------------------------------------------------------------------

def test_config_is_read_field_by_field(pkg):
    cfg = config(40, 70, [mingru(24, 56), latent(3, 10, 6, 7, 18, 5, base=321.5, scale=0.31, rot_dims=4), mingru(8)], taps=3, eps=2e-4)
    m = pkg.LayeredMetadata.from_config(json.loads(json.dumps(cfg)), "m")
    assert (m.architecture, m.hidden_size, m.vocab_size, m.norm_eps, m.conv_taps, m.num_layers) == ("Metapel", 40, 70, 2e-4, 3, 3)
    assert m.layers[0] == pkg.LayerSpec("mingru", 56, width=24)
    assert m.layers[1] == pkg.LayerSpec("latent_attention", 0, heads=3, dim=10, rot_dim=6, value_dim=7, kv_rank=18, window=5,
                                        rope_dims=4, rope_base=321.5, scale=0.31)
    assert m.layers[2] == pkg.LayerSpec("mingru", 0, width=8)
    assert m.cache_values_per_token() == 24


@pytest.mark.parametrize("spoil", [
    lambda c: c["layers"][0].update(type="unknown"), lambda c: c["layers"][0]["mlp"].update(kind="other"),
    lambda c: c["layers"][1]["mixer"].pop("kv_rank"), lambda c: c.pop("canon"), lambda c: c["norm"].pop("eps"),
    lambda c: c["layers"][0].pop("mlp"), lambda c: c.update(layers=3)])
def test_malformed_configs_are_refused(pkg, spoil):
    cfg = json.loads(json.dumps(ODD))
    spoil(cfg)
    with pytest.raises(pkg.ModelError):
        pkg.LayeredMetadata.from_config(cfg)


def test_registry_picks_the_class(pkg, tmp_path):
    path = tmp_path / "config.json"
    path.write_text(json.dumps(TUNED))
    assert pkg.model_class(str(tmp_path)) is pkg.CudaLayeredModel
    path.write_text(json.dumps({"architectures": ["LlamaForCausalLM"], "hidden_size": 8}))
    assert pkg.model_class(str(tmp_path)) is pkg.CudaTransformerModel
    path.write_text(json.dumps({"architecture": "Other"}))
    with pytest.raises(pkg.ModelError, match="unsupported architecture Other"):
        pkg.model_class(str(tmp_path))
    path.write_text("{")
    with pytest.raises(pkg.ModelError, match="malformed"):
        pkg.model_class(str(tmp_path))
    with pytest.raises(pkg.ModelError):
        pkg.model_class(str(tmp_path / "missing"))


# ---- the plain implementation ------------------------------------------------------------------------

def test_convolution_by_hand():
    h = np.array([[1.0], [2.0], [4.0]])
    w = np.array([[10.0, 100.0, 1000.0]])  # two back, one back, current
    assert metapel.causal_conv(h, w).ravel().tolist() == [1000.0, 2100.0, 4210.0]
    assert metapel.causal_conv(h[:1], w).ravel().tolist() == [1000.0]


def test_recurrence_by_hand():
    z = np.array([[1.0], [0.5], [0.25]])
    c = np.array([[8.0], [2.0], [4.0]])
    assert metapel.min_gru_scan(z, c).ravel().tolist() == [8.0, 5.0, 4.75]
    w = {"z": np.zeros((2, 1)), "z.b": np.array([0.0, 2.0]), "x": np.array([[1.0], [-1.0]]), "x.b": np.zeros(2)}
    z, c = metapel.min_gru_gates(np.array([[3.0]]), w)
    assert np.allclose(z, [[0.5, 1 / (1 + np.exp(-2.0))]]) and np.allclose(c, [[3.5, 1 / (1 + np.exp(3.0))]])


def test_rotation_pairs_neighbours_and_leaves_the_rest():
    x = np.array([[1.0, 0.0, 0.0, 1.0, 5.0, 6.0]])
    y = metapel.rotate_interleaved(x, np.array([3]), 100.0, 4)
    a, b = 3.0, 3.0 * 100.0 ** -0.5
    assert np.allclose(y, [[np.cos(a), np.sin(a), -np.sin(b), np.cos(b), 5.0, 6.0]])
    # scores of rotated vectors depend on the distance only
    q, k = np.random.default_rng(0).standard_normal((2, 1, 8))
    s = [float((metapel.rotate_interleaved(q, np.array([p + 5]), 50.0, 8) * metapel.rotate_interleaved(k, np.array([p]), 50.0, 8)).sum())
         for p in (0, 7, 90)]
    assert np.allclose(s, s[0])


def test_window_counts_the_token_itself():
    m = metapel.window_mask(5, 2)
    assert m.tolist() == [[j in (i, i - 1) for j in range(5)] for i in range(5)]
    assert metapel.window_mask(4, 1).tolist() == np.eye(4, dtype=bool).tolist()
    assert metapel.window_mask(3, None).sum() == 6


def test_activations():
    x = np.array([-50.0, -1.0, 0.0, 2.0, 900.0])
    assert np.allclose(metapel.sigmoid(x)[1:4], 1 / (1 + np.exp(-x[1:4]))) and np.isfinite(metapel.sigmoid(-x)).all()
    assert np.allclose(metapel.gelu_tanh(np.array([1.0])), 0.841192, atol=1e-5)


def test_one_token_attends_to_itself():
    """With one visible key the weights are one: the layer is the value path whatever the queries are."""
    cfg = config(24, 30, [latent(2, 4, 2, 6, 8, 1)], taps=2)
    w = random_weights(cfg, 4)
    t = [3, 9, 9, 1]
    a = metapel.forward(t, cfg, w)
    w["l0.mix.q"] = -3 * w["l0.mix.q"]
    assert np.allclose(a, metapel.forward(t, cfg, w))


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_prefixes_are_causal(name):
    cfg = CONFIGS[name]
    w = random_weights(cfg, 2)
    assert set(w) == set(tensor_shapes(cfg))
    t = np.random.default_rng(3).integers(0, cfg["vocab"], 30).tolist()
    whole = metapel.forward(t, cfg, w)
    assert np.allclose(metapel.forward(t[:17], cfg, w), whole[:17])
    assert worst_error(metapel.forward([(t[0] + 1) % cfg["vocab"]] + t[1:], cfg, w)[1:], whole[1:]) > 1e-3


# ---- state slots and recomputation in the driver --------------------------------------------------------

def test_state_slots_come_and_go_with_the_block_table(pkg):
    m = pkg.KvCacheManager(8, 4, False, num_state_slots=2)
    m.allocate(1, [1] * 5)
    m.allocate(2, [1] * 3)
    assert (m.state_slot(1), m.state_slot(2), m.state_slot(3)) == (0, 1, None)
    free = m.free_blocks()
    with pytest.raises(pkg.CacheExhausted, match="state slots"):
        m.allocate(3, [1])
    assert m.free_blocks() == free, "a refused allocation takes nothing"
    m.free(1)
    assert m.state_slot(1) is None
    m.allocate(3, [1])
    assert m.state_slot(3) == 0
    m.free(2)
    m.free(2)
    m.allocate(4, [1])
    assert m.state_slot(4) == 1
    assert pkg.KvCacheManager(8, 4, False).state_slot(1) is None


def test_extend_is_all_or_nothing(pkg):
    m = pkg.KvCacheManager(4, 4, False, num_state_slots=1)
    m.allocate(1, [1] * 3)
    m.extend(1, 1)
    assert m.block_table(1) == ([0], 4)
    m.extend(1, 6)
    assert m.block_table(1) == ([0, 1, 2], 10)
    with pytest.raises(pkg.CacheExhausted):
        m.extend(1, 7)
    assert m.block_table(1) == ([0, 1, 2], 10)
    m.extend(1, 6)
    assert m.free_blocks() == 0
    with pytest.raises(pkg.InternalError):
        m.extend(9, 1)


class Stateful:
    """Stands in for a model with state: per sequence it keeps the tokens it was fed, insists that every portion
    continues them (or starts over at position 0), and answers with a function of all of them."""

    def __init__(self, fail_steps=()):
        self.history, self.calls, self.fail_steps = {}, 0, set(fail_steps)

    @staticmethod
    def next_token(tokens):
        h = 17
        for t in tokens:
            h = (h * 31 + t + 1) % 1000003
        return h % 97

    def __call__(self, batch):
        import orionserve_rs_b200 as pkg

        self.calls += 1
        if self.calls in self.fail_steps:
            raise pkg.BackendError("injected")
        assert len(set(batch.sequence_ids)) == len(batch.sequence_ids)
        out, at = [], 0
        for s, n in zip(batch.sequence_ids, batch.slot_token_counts):
            pos, tok = batch.positions[at:at + n], batch.tokens[at:at + n]
            have = [] if pos[0] == 0 else self.history[s]
            assert pos == list(range(len(have), len(have) + n)), (s, pos, len(have))
            self.history[s] = have + tok
            out.append(self.next_token(self.history[s]))
            at += n
        return out


def run_stateful(pkg, blocks, fail_steps=(), **cfg):
    E = pkg.engine
    kw = dict(max_num_seqs=6, max_num_batched_tokens=24, request_timeout_secs=None, logical_decode_positions=True,
              recompute_on_preempt=True)
    kw.update(cfg)
    model = Stateful(fail_steps)
    eng = E.Engine(model, E.SchedulerConfig(**kw), blocks, 4, True)
    rng = np.random.default_rng(1)
    prompts = [rng.integers(0, 97, int(n)).tolist() for n in (5, 13, 30, 2, 9, 17, 21)]
    ids = [eng.submit(p, E.SamplingParams(temperature=0.0, max_tokens=18)) for p in prompts]
    tokens = {i: [] for i in ids}
    for _ in range(3000):
        if not eng.has_work():
            break
        try:
            eng.step()
        except pkg.BackendError:
            pass
        for ev in eng.take_events():
            if ev.kind == "token":
                tokens[ev.id].append(ev.token)
    assert not eng.has_work()
    for p, i in zip(prompts, ids):
        exp = list(p)
        for _ in range(18):
            exp.append(Stateful.next_token(exp))
        assert tokens[i] == exp[len(p):]
    return eng


def test_preempted_sequences_prefill_their_output_again(pkg):
    assert run_stateful(pkg, 200).scheduler().stats()["total_preempted"] == 0
    assert run_stateful(pkg, 22).scheduler().stats()["total_preempted"] > 0
    assert run_stateful(pkg, 18, prioritize_decode=False).scheduler().stats()["total_preempted"] > 0
    assert run_stateful(pkg, 22, max_num_batched_tokens=7).scheduler().stats()["total_preempted"] > 0


def test_a_failed_step_is_prefilled_again(pkg):
    run_stateful(pkg, 200, fail_steps=(1, 3, 4, 9, 20))
    run_stateful(pkg, 22, fail_steps=(2, 6, 11, 30))


# ---- trace replay ------------------------------------------------------------------------------------

class SlotModel:
    """A model on the host that keeps what each state slot has been fed and evaluates the plain implementation."""

    def __init__(self, cfg, weights, blocks, slots):
        self.cfg, self.weights, self.num_blocks, self.block_size, self.slots = cfg, weights, blocks, 16, slots
        self.fed, self.batches = {}, []

    def num_state_slots(self):
        return self.slots

    def forward(self, b):
        b.validate()
        self.batches.append(b)
        rows, at = [], 0
        for slot, n, table, ctx in zip(b.state_slots, b.slot_token_counts, b.block_tables, b.context_lens):
            start = b.positions[at]
            seq = (self.fed[slot] if start else []) + list(b.tokens[at:at + n])
            assert len(seq) == start + n == ctx and len(table) == -(-ctx // 16)
            self.fed[slot] = seq
            rows.append(metapel.forward(seq, self.cfg, self.weights)[start:])
            at += n
        flat = [t for i, t in enumerate(b.block_tables)]
        assert len({x for t in flat for x in t}) == sum(map(len, flat)), "no page belongs to two requests"
        return type("Out", (), {"logits": np.concatenate(rows)[list(b.logit_rows)].astype(np.float32)})


def test_trace_replay_keeps_requests_apart(pkg):
    from orionserve_rs_b200.trace import TraceRunner

    cfg = config(16, 40, [mingru(8, 12), latent(2, 4, 2, 4, 6, 5)], taps=3)
    w = random_weights(cfg, 1)
    rng = np.random.default_rng(2)
    t = {n: rng.integers(0, 40, k).tolist() for n, k in (("a", 40), ("b", 21), ("c", 33))}
    r = TraceRunner(SlotModel(cfg, w, 6, 2))
    steps = [([("a", 0, 18, [17, 0])], []), ([("a", 18, 19, []), ("b", 0, 20, [5])], []), ([("b", 20, 21, [0])], ["b"]),
             ([("c", 0, 2, [1]), ("a", 19, 40, [20, 3])], ["a"]), ([("c", 2, 33, [30])], ["c"])]
    exp = {n: metapel.forward(x, cfg, w) for n, x in t.items()}
    for entries, end in steps:
        out = r.step([{"id": n, "tokens": t[n][lo:hi], "want": want} for n, lo, hi, want in entries], end)
        want = [exp[n][lo + k] for n, lo, _, ks in entries for k in ks]
        assert (out is None) == (not want)
        if want:
            assert np.allclose(out, want, atol=1e-4)
    assert not r.live and r.cache.free_blocks() == 6
    assert {s for b in r.model.batches for s in b.state_slots} == {0, 1}


def test_trace_runner_prints_and_writes(pkg, tmp_path, monkeypatch, capsys):
    import io
    import sys

    from orionserve_rs_b200 import trace

    cfg = config(16, 40, [mingru(8)], taps=2)
    w = random_weights(cfg, 1)
    monkeypatch.setattr(trace, "load_model", lambda d, blocks, block, backend, **kw: SlotModel(cfg, w, blocks, kw["num_state_slots"]))
    monkeypatch.setattr(trace, "CudaBackend", lambda i: None)
    lines = [{"step": 0, "entries": [{"id": "a", "tokens": [1, 2, 3], "want": []}], "end": []},
             {"step": 7, "entries": [{"id": "a", "tokens": [4], "want": [0]}], "end": ["a"]}, {"step": 8, "entries": [], "end": []}]
    monkeypatch.setattr(sys, "stdin", io.StringIO("".join(json.dumps(x) + "\n" for x in lines)))
    assert trace.main(["--model", "m", "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "100"]) == 0
    assert capsys.readouterr().out.split("\n")[:3] == ["done 0", "done 7", "done 8"]
    assert [p.name for p in tmp_path.iterdir()] == ["7.f32"]
    got = np.fromfile(tmp_path / "7.f32", "<f4")
    assert np.allclose(got, metapel.forward([1, 2, 3, 4], cfg, w)[-1], atol=1e-4)
