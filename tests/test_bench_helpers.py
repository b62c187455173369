"""Host-side arithmetic of the benchmark: algorithmic byte counts and the synthetic decode batch."""
import numpy as np

import bench


def test_algorithmic_bytes_of_the_headline_step():
    m = bench.LLAMA3_8B
    # 218.1 M parameters per layer x 32 + 525.3 M of LM head, bf16: 15.0 GB of weights per step
    assert bench.layer_param_count(m) == 218_103_808
    assert bench.weight_bytes_per_step(m) == 2 * (32 * 218_103_808 + 128256 * 4096)
    # 4096 B per context token per sequence per layer + q/out + table entries
    kv = bench.kv_bytes_per_step(m, [bench.CONTEXT] * bench.BATCH)
    per_layer = 64 * (1024 * 4096 + 32 * 128 * 2 * 2 + 64 * 4)
    assert kv == 32 * per_layer
    assert abs(kv / 1e9 - 8.62) < 0.01


def test_tensor_parallel_ranks_share_the_layers_and_the_head():
    for m in (bench.LLAMA3_8B, bench.LLAMA3_70B):
        whole = bench.weight_bytes_per_step(m)
        head = 2 * m["vocab_size"] * m["hidden_size"]
        for world in (2, 4, 8):
            # the head is split by vocabulary in multiples of 128 rows; the busiest rank holds the rounded-up share
            rows = -(-(-(-m["vocab_size"] // world)) // 128) * 128
            assert bench.head_rows_per_rank(m, world) == rows and rows * world >= m["vocab_size"] > rows * (world - 1)
            assert bench.weight_bytes_per_step(m, world) == (whole - head) // world + 2 * rows * m["hidden_size"]
            ctx = [1024, 4096, 2000]
            tables = m["num_layers"] * sum((c + 15) // 16 for c in ctx) * 4  # every rank reads the whole table
            assert bench.kv_bytes_per_step(m, ctx, world) * world - bench.kv_bytes_per_step(m, ctx) == tables * (world - 1)


def test_decode_batches_are_valid_and_their_tables_disjoint(pkg):
    rng = np.random.default_rng(0)
    for contexts in ([1024] * 8, [1024, 4096, 1500, 16, 17, 1]):
        num_blocks = sum(c // 16 + 1 for c in contexts) + 4
        b = bench.make_decode_batch(pkg, rng, num_blocks, contexts, 1000)
        b.validate()
        tokens, positions, counts, ctx, flat, offsets = b.flatten()
        assert positions.tolist() == [c - 1 for c in contexts] and ctx.tolist() == contexts
        assert counts.tolist() == [1] * len(contexts) and int(tokens.max()) < 1000
        lens = np.diff(offsets).tolist()
        assert lens == [(c + 15) // 16 for c in contexts]
        used = flat[:int(offsets[-1])]
        assert len(set(used.tolist())) == len(used) and int(used.max()) < num_blocks


def test_algorithmic_work_of_a_metapel_step(pkg):
    z = dict(heads=4, dim=32, rot_dim=16, value_dim=24, kv_rank=64, window=10)
    meta = pkg.LayeredMetadata("Metapel", "m", 48, 100, [pkg.LayerSpec("mingru", 20, width=30),
                               pkg.LayerSpec("latent_attention", 0, **z)], 1e-5, 4)
    gru = 48 * 3 * 30 + 30 * 48 + 2 * 48 * 20
    att = 48 * (4 * 48 + 80 + 4 * 24) + 4 * 24 * 48
    head = bench.LAYERED_VOCAB * 48
    w, fl, cache, attn = bench.metapel_work(meta, 2, [7, 300], [])
    assert w == 2 * (gru + att + head) and fl == 2 * 2 * (gru + att + head)
    assert cache == (7 + 10) * 80 * 2 and attn == (7 + 10) * 4 * 2 * (2 * 64 + 16)
    w, fl, cache, attn = bench.metapel_work(meta, 12, [], [12])
    att += 4 * (32 + 24) * 64
    assert w == 2 * (gru + att + head) and fl == 2 * (12 * (gru + att) + head)
    assert cache == 0 and attn == (55 + 2 * 10) * 4 * 2 * (32 + 16 + 24)


def test_algorithmic_work_of_a_zulozen_step(pkg):
    att = dict(heads=4, kv_heads=2, dim=32, value_dim=24, chunk=10)
    meta = pkg.LayeredMetadata("Zulozen", "m", 48, 100, [pkg.LayerSpec("attention", 20, **att),
                               pkg.LayerSpec("attention", 12, experts=4, experts_per_token=1, shared_dim=8, **att)], 1e-5, block="sandwich")
    mix = 48 * (4 * 32 + 2 * 56 + 4) + 4 * 24 * 48
    dense, fixed, expert = 2 * 48 * 20, 4 * 48 + 3 * 48 * 8, 3 * 48 * 12
    head = bench.LAYERED_VOCAB * 48
    w, fl, cache, attn = bench.zulozen_work(meta, 1, [27], [])  # one row reaches one expert; 7 keys of its chunk
    assert w == 2 * (2 * mix + dense + fixed + expert + head) == fl
    assert cache == 2 * 7 * 2 * 56 * 2 and attn == 2 * 7 * 4 * 2 * 56
    w, fl, cache, attn = bench.zulozen_work(meta, 12, [], [12])
    assert w == 2 * (2 * mix + dense + fixed + head) + 2 * int(4 * (1 - 0.75 ** 12) * expert)
    assert fl == 2 * (12 * (2 * mix + dense + fixed + expert) + head)
    assert cache == 0 and attn == 2 * (55 + 3) * 4 * 2 * 56


def test_algorithmic_work_of_a_belizen_step(pkg):
    layers = [pkg.LayerSpec("gla", 20, heads=4, dim=8, value_dim=12, decay_rank=3, decay_tau=4.0, activation="geglu_tanh"),
              pkg.LayerSpec("attention", 12, heads=4, kv_heads=2, dim=32, value_dim=24, window=10, keep_first=2, qk_norm="per_head", experts=3,
                            router="softmax", router_identity=1, experts_per_token=1, shared_dim=8)]
    meta = pkg.LayeredMetadata("Belizen", "m", 48, 100, layers, 1e-5, block="prenorm", loop=pkg.Loop(0, 1, 2))
    lin = 48 * (2 * 32 + 2 * 48 + 3) + 32 * 3 + 48 * 48 + 3 * 48 * 20
    att = 48 * (4 * 32 + 2 * 56 + 4 * 24) + 4 * 24 * 48 + 4 * 48 + 3 * 48 * 8
    expert, head = 3 * 48 * 12, bench.LAYERED_VOCAB * 48
    w, fl, cache, attn = bench.belizen_work(meta, 1, [27], [])  # one row reaches an expert three times out of four
    assert w == 2 * (2 * lin + att + int(0.75 * expert) + head) and fl == 2 * (2 * lin + att + head) + int(2 * 0.75 * expert)
    assert cache == 2 * 2 * 32 * 12 * 4 + 12 * 2 * 56 * 2 and attn == 2 * 4 * 32 * 12 + 12 * 4 * 2 * 56
    w, fl, cache, attn = bench.belizen_work(meta, 14, [], [14])
    assert w == 2 * (2 * lin + att + head) + 2 * int(3 * (1 - 0.75 ** 14) * expert)
    assert cache == 0 and attn == 14 * 2 * 4 * 32 * 12 + (78 + 2 * 12) * 4 * 2 * 56


def test_algorithmic_work_of_a_vusenex_step(pkg):
    moe = dict(ffn_dim=12, experts=4, experts_per_token=1, shared_dim=8, router="softmax_renorm", expert_form="gelu")
    layers = [pkg.LayerSpec("latent_attention", heads=4, dim=32, value_dim=24, kv_rank=64, ungated=True, **moe),
              pkg.LayerSpec("attention", heads=4, kv_heads=2, dim=32, value_dim=32, qk_norm=True, keys_as_values=True, **moe)]
    meta = pkg.LayeredMetadata("Vusenex", "m", 48, 100, layers, 1e-5, block="gated_postnorm")
    lat, att = 48 * (128 + 64) + 96 * 48, 48 * (128 + 64) + 128 * 48
    rest, expert, head = 2 * 48 * 48 + 4 * 48 + 2 * 48 * 8, 2 * 48 * 12, bench.LAYERED_VOCAB * 48
    w, fl, cache, attn = bench.vusenex_work(meta, 1, [27], [])  # one row reaches one expert
    assert w == 2 * (lat + att + 2 * rest + 2 * expert + head) == fl
    assert cache == 27 * (64 * 2 + 2 * (32 * 2 + 4)) and attn == 27 * (4 * 4 * 64 + 2 * 2 * 128)
    w, fl, cache, attn = bench.vusenex_work(meta, 12, [], [12])
    lat += (128 + 96) * 64
    assert w == 2 * (lat + att + 2 * rest + head) + 2 * 2 * int(4 * (1 - 0.75 ** 12) * expert)
    assert fl == 2 * (12 * (lat + att + 2 * rest + 2 * expert) + head)
    assert cache == 0 and attn == 78 * (2 * (128 + 96) + 2 * 256)
