"""Varolorn without a GPU: the configuration and its errors, tensor names and shapes (one of them known to the file only), the
cache and state each layer asks for, pages of earlier stretches given back, distance buckets and the cuts of a stretch, random
model folders, and the plain implementation's mechanisms against closed forms."""
import copy
import dataclasses
import math

import numpy as np
import pytest
import torch

import plain_varolorn as P
import varolorn_helpers as H


def test_configuration_reads_every_key_and_round_trips():
    import zinfer_b200 as z
    for name, d in H.CONFIGS.items():
        c = z.config_from_dict(d)
        assert c.architecture == "Varolorn" and c.vocab_size == d["vocab"] and c.hidden_size == d["width"], name
        assert c.norm_eps == d["norm"]["eps"] and c.streams == d.get("streams", 0) and len(c.layers) == len(d["layers"])
        assert c.embedding_scale == d.get("embedding", {}).get("scale", 1.0)
        again = c.to_json_dict()
        assert dataclasses.replace(z.config_from_dict(again), raw={}) == dataclasses.replace(c, raw={})
        assert again["layers"] == d["layers"] and again.get("streams") == d.get("streams")
        assert again["embedding"].get("bigram") == d.get("embedding", {}).get("bigram")
    c = z.config_from_dict(H.CONFIGS["va"])
    m = c.layers[0].mixer
    assert (m.heads, m.kv_heads, m.dim, m.vdim, m.scale, m.bias_max, m.chunk, m.v_mix) == (4, 2, 16, 12, 0.3, 9.5, 7, True)
    s = c.layers[1].mixer
    assert (s.heads, s.vdim, s.state, s.groups, s.conv, s.norm_groups) == (3, 10, 8, 1, 3, 2)
    assert c.layers[2].ff is None and c.layers[4].ff == 16 and c.bigram.mul_cur == 11 and c.first_value_layer() == 0
    assert z.config_from_dict(H.CONFIGS["vb"]).first_value_layer() is None


@pytest.mark.parametrize("change,message", [
    (lambda d: d["layers"][0].update(type="hgrn2"), "known types"),
    (lambda d: d["layers"][0]["mixer"].update(kv_heads=3), "not a multiple"),
    (lambda d: d["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda d: d["layers"][0]["mixer"].pop("bias_max"), "bias_max"),
    (lambda d: d["layers"][0]["mixer"].update(bias_max=1), "bias_max"),
    (lambda d: d["layers"][0]["mixer"].update(mask={"size": 0}), "mask.size"),
    (lambda d: d["layers"][0]["mixer"].update(v_mix=1), "v_mix"),
    (lambda d: d["layers"][2]["mixer"].update(vdim=13), "mix values"),
    (lambda d: d["layers"][1]["mixer"].pop("state"), "state"),
    (lambda d: d["layers"][1]["mixer"].update(groups=2), "groups"),
    (lambda d: d["layers"][1]["mixer"].update(norm_groups=4), "equal parts"),
    (lambda d: d["layers"][1]["mixer"].update(conv=0), "conv"),
    (lambda d: d["layers"][1]["mlp"].update(kind="moe"), "dense"),
    (lambda d: d["embedding"]["bigram"].pop("mul_prev"), "mul_prev"),
    (lambda d: d["embedding"]["bigram"].update(buckets=0), "buckets"),
    (lambda d: d.update(streams=0), "streams"),
    (lambda d: d.pop("vocab"), "vocab"),
])
def test_configuration_errors_name_the_key(change, message):
    import zinfer_b200 as z
    d = copy.deepcopy(H.CONFIGS["va"])
    change(d)
    with pytest.raises(z.ConfigError, match=message):
        z.config_from_dict(d)


def test_model_asks_for_the_tensors_of_the_design():
    import zinfer_b200 as z
    from zinfer_b200.config.registry import build_model
    from zinfer_b200.parts.base import ANY_SIZE
    specs = build_model(z.config_from_dict(H.CONFIGS["va"])).weight_specs()
    want = {"embed": (101, 48), "bigram": (38, 48), "final.norm": (48,), "l0.norm1": (48,), "l0.norm2": (48,), "l0.mix.q": (64, 48),
            "l0.mix.q.b": (64,), "l0.mix.k": (32, 48), "l0.mix.k.b": (32,), "l0.mix.v": (24, 48), "l0.mix.v.b": (24,),
            "l0.mix.q.norm": (16,), "l0.mix.k.norm": (16,), "l0.mix.rel": (ANY_SIZE, 4), "l0.mix.vmix": (), "l0.mix.g": (4, 48),
            "l0.mix.o": (48, 48), "l0.mix.o.b": (48,), "l0.mlp.gate": (40, 48), "l0.mlp.up": (40, 48), "l0.mlp.down": (48, 40),
            "l0.hc1.in": (3,), "l0.hc1.out": (3,), "l0.hc1.mix": (3, 3), "l0.hc2.in": (3,), "l0.hc2.out": (3,), "l0.hc2.mix": (3, 3),
            "l1.mix.in": (30 + 30 + 16 + 3, 48), "l1.mix.conv": (46, 3), "l1.mix.conv.b": (46,), "l1.mix.dt_bias": (3,),
            "l1.mix.A_log": (3,), "l1.mix.D": (3,), "l1.mix.norm": (30,), "l1.mix.o": (48, 30)}
    for name, shape in want.items():
        assert specs[name].shape == shape, name
    assert not any(n in specs for n in ("l2.norm2", "l2.hc2.in", "l2.mlp.gate", "l3.mix.vmix", "head"))
    assert len(specs) == 3 + (13 + 5 + 6) + (8 + 5 + 6) + (13 + 1 + 3) + (12 + 1 + 3) + (13 + 5 + 6)
    plain = build_model(z.config_from_dict(H.CONFIGS["vd"])).weight_specs()
    assert sorted(plain) == sorted(["embed", "bigram", "final.norm", "l0.norm1"] + [f"l0.mix.{n}" for n in
                                   ("in", "conv", "conv.b", "dt_bias", "A_log", "D", "norm", "o")])


def test_storage_each_layer_asks_for():
    import zinfer_b200 as z
    from zinfer_b200.config.registry import build_model
    cs = build_model(z.config_from_dict(H.CONFIGS["va"])).cache_specs()
    assert len(cs) == 6                                       # five layers and, behind them, the embedding's last token
    assert (cs[0].kv.n_kv_heads, cs[0].kv.head_dim, cs[0].kv.v_dim, cs[0].kv.window, cs[0].kv.chunk) == (2, 16, 12, 0, 7)
    assert cs[1].kv is None and cs[1].state.shape == (-(-(2 * 46 + 3 * 8 * 10) // 4) * 4,) and cs[1].state.dtype == torch.float32
    assert cs[5].kv is None and cs[5].state.shape == (1,) and cs[5].state.dtype == torch.int32
    assert len(build_model(z.config_from_dict(H.CONFIGS["vb"])).cache_specs()) == 3      # no pair rows: no state


def test_pages_of_earlier_stretches_come_back():
    """Stretches of 40 positions on pages of 16: a page goes back when no position of it lies in the next token's stretch."""
    from zinfer_b200.cache import CacheManager, CallCacheSpec
    from zinfer_b200.parts.base import KVRequest
    cache = CacheManager([CallCacheSpec(kv=KVRequest(1, 8, chunk=40)), CallCacheSpec(kv=KVRequest(1, 8))], 2, 256, 128, 16, torch.float32, "cpu")
    assert len(cache.groups) == 2
    slot, = cache.alloc_slots(1)
    for n in range(1, 128):
        cache.reserve([slot], [1])
        cache.advance([slot], [1])
        first = n // 40 * 40                                  # the next token stands at position n
        held = [i for i in range(-(-n // 16)) if cache.groups[0].table_host[slot, i] >= 0]
        assert held == [i for i in range(-(-n // 16)) if i >= first // 16], n
        assert all(cache.groups[1].table_host[slot, i] >= 0 for i in range(-(-n // 16)))
        cache.check_consistency()
    cache.free_slots([slot])
    cache.check_consistency()
    assert cache.free_page_count() == [16, 16]


def test_readers_of_a_cache_in_stretches():
    from zinfer_b200.cache import CacheManager, CallCacheSpec
    from zinfer_b200.parts.base import KVRequest
    def group(a, b):
        c = CacheManager([CallCacheSpec(kv=a), CallCacheSpec(kv=b, kv_owner=0)], 1, 64, 64, 16, torch.float32, "cpu")
        return c.groups[0].request
    assert group(KVRequest(1, 8, chunk=20), KVRequest(1, 8, chunk=20)).chunk == 20
    assert group(KVRequest(1, 8, chunk=20), KVRequest(1, 8, chunk=30)).chunk == 0       # not the same: everything stays
    assert group(KVRequest(1, 8, chunk=20), KVRequest(1, 8)).chunk == 0


@pytest.mark.parametrize("rows,most", [(16, 100), (32, 128), (7, 20), (2, 3), (3, 1.5), (8, 16), (6, 27), (64, 1000.5), (24, 12.5)])
def test_distance_buckets(rows, most):
    """Against the logarithm where no edge is near, and at the edges that are whole numbers."""
    from zinfer_b200.parts.attention import distance_buckets
    half = rows // 2
    got = distance_buckets(rows, most, 1200)
    assert got == [P.distance_bucket(n, rows, most) for n in range(1200)]
    assert got[:half] == list(range(half)) and all(b - a in (0, 1) or a < b for a, b in zip(got, got[1:]))
    assert got[math.ceil(most):] == [rows - 1] * (1200 - math.ceil(most)) and max(got) == rows - 1
    for n in range(max(half, 1), 1200):
        x = math.log(n / half) / math.log(most / half) * (rows - half)
        if abs(x - round(x)) > 1e-9:
            assert got[n] == min(rows - 1, half + math.floor(x)), n
        else:
            assert got[n] == min(rows - 1, half + round(x)), n


def test_distance_buckets_refuse_what_has_no_geometric_part():
    from zinfer_b200.parts.attention import distance_buckets
    for rows, most in ((16, 8), (1, 10), (40, 20)):
        with pytest.raises(ValueError):
            distance_buckets(rows, most, 5)


def test_key_cuts_of_a_stretch():
    from zinfer_b200.parts.attention import key_chunks
    assert key_chunks(8, 8, 5000, 148, most=90) == (1, 0)                       # one block walks a short stretch
    n, keys = key_chunks(1, 1, 5000, 148, most=1000)
    assert keys % 64 == 0 and n == -(-1000 // keys) > 1
    assert key_chunks(1, 1, 300, 148, most=100000) == key_chunks(1, 1, 300, 148)


def test_random_model_folders_load_back(tmp_path):
    import zinfer_b200 as z
    from zinfer_b200.config.registry import build_model
    from zinfer_b200.weights.loader import WeightError, check_tensors
    from zinfer_b200.weights.safetensors_io import SafetensorsFile
    cfg = z.config_from_dict(H.CONFIGS["ve"])
    folder = z.write_random_model(tmp_path / "m", cfg, seed=3)
    assert dataclasses.replace(z.config_from_folder(folder), raw={}) == dataclasses.replace(cfg, raw={})
    specs = build_model(cfg).weight_specs()
    with SafetensorsFile(folder / "model.safetensors") as f:
        assert sorted(f.names()) == sorted(specs)
        found = {n: (f.infos[n].dtype, f.infos[n].shape) for n in f.names()}
    assert found["l0.mix.rel"][1][1] == 5 and found["l0.mix.vmix"][1] == ()
    check_tensors("here", specs, found)
    check_tensors("here", specs, {**found, "l0.mix.rel": (torch.bfloat16, (9, 5))})         # the file says how many buckets
    with pytest.raises(WeightError, match="'any', 5"):
        check_tensors("here", specs, {**found, "l0.mix.rel": (torch.bfloat16, (9, 6))})
    with pytest.raises(WeightError, match="rel"):
        check_tensors("here", specs, {**found, "l0.mix.rel": (torch.bfloat16, (0, 5))})


# ------------------------------------------------------------------------------- the plain implementation's own mechanisms

def test_plain_scan_is_its_closed_form():
    """y_t = sum_{j <= t} exp(-exp(a) sum_{j < i <= t} dt_i) dt_j (C_t . B_j) x_j + D x_t."""
    rng = np.random.default_rng(0)
    n, H, e, G, N = 9, 4, 3, 2, 5
    x, B, C = rng.normal(size=(n, H, e)), rng.normal(size=(n, G, N)), rng.normal(size=(n, G, N))
    dt, a, D = rng.uniform(0.1, 2.0, (n, H)), rng.normal(size=H), rng.normal(size=H)
    got = P.ssd_scan(x, B, C, dt, a, D)
    for h in range(H):
        g = h // 2
        for t in range(n):
            want = D[h] * x[t, h]
            for j in range(t + 1):
                want = want + math.exp(-math.exp(a[h]) * dt[j + 1:t + 1, h].sum()) * dt[j, h] * (C[t, g] @ B[j, g]) * x[j, h]
            assert np.allclose(got[t, h], want)


def test_plain_convolution_and_group_norm():
    x = np.arange(12.0).reshape(6, 2)
    y = P.short_conv(x, np.array([[1.0, 10.0, 100.0], [0.0, 0.0, 1.0]]), np.array([0.5, 0.0]))
    assert np.allclose(y[0], [0.5, 1.0]) and np.allclose(y[3], [0.5 + 100 * 6 + 10 * 4 + 2, 7.0])
    u = P.gated_group_norm(np.array([[1.0, 2.0, 30.0, 40.0]]), np.full((1, 4), 50.0), np.ones(4), 2, 0.0)
    r = math.sqrt(2.5), math.sqrt(1250.0)
    assert np.allclose(u, [[1 / r[0], 2 / r[0], 30 / r[1], 40 / r[1]]])


def test_plain_streams_read_from_and_write_to():
    X = np.arange(12.0).reshape(2, 3, 2)
    assert np.allclose(P.stream_read(X, np.array([1.0, -2.0])), X[0] - 2 * X[1])
    Y = P.stream_write(X, np.array([[0.0, 1.0], [5.0, 0.0]]), np.array([1.0, 0.0]), np.ones((3, 2)))
    assert np.allclose(Y[0], 5 * X[1] + 1) and np.allclose(Y[1], X[0])          # mix is [from, to]


def test_plain_pair_rows_and_stretches():
    table, rows = np.zeros((10, 4)), np.arange(6.0)[:, None] * np.ones((1, 4))
    x = P.embed_rows([3, 4, 9], table, 2.0, (rows, 5, 7, 2))
    assert x[:, 0].tolist() == [5.0, (3 * 7 + 4 * 2) % 5, (4 * 7 + 9 * 2) % 5]
    assert [[P.visible(i, j, 3) for j in range(7)] for i in (2, 3, 6)] == [[True] * 3 + [False] * 4, [False] * 3 + [True] + [False] * 3,
                                                                          [False] * 6 + [True]]
    assert all(P.visible(5, j, 0) for j in range(6))


def test_plain_value_mixing_uses_the_first_mixing_layer():
    """Three attention layers, the second without v_mix: the third mixes with the first."""
    cfg = copy.deepcopy(H.CONFIGS["va"])
    cfg["layers"] = [cfg["layers"][0], cfg["layers"][3], cfg["layers"][4]]
    cfg["layers"][1]["mixer"]["v_mix"] = False
    rng = np.random.default_rng(2)
    D, n = cfg["width"], 6
    m = cfg["layers"][2]["mixer"]
    H_, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    W = {"q": rng.normal(size=(H_ * d, D)), "q.b": np.zeros(H_ * d), "k": rng.normal(size=(G * d, D)), "k.b": np.zeros(G * d),
         "v": rng.normal(size=(G * e, D)), "v.b": rng.normal(size=G * e), "q.norm": np.ones(d), "k.norm": np.ones(d),
         "rel": np.zeros((4, H_)), "g": np.zeros((H_, D)), "o": np.eye(H_ * e)[:D], "o.b": np.zeros(min(D, H_ * e)), "vmix": np.array(1.0)}
    h, first = rng.normal(size=(n, D)), rng.normal(size=(n, G, e))
    out, own = P.attention(h, W, m, 1e-6, first)
    assert np.allclose(own.reshape(n, -1), h @ W["v"].T + W["v.b"])
    assert np.allclose(out[0].reshape(-1), 0.5 * np.repeat(first[0], H_ // G, axis=0).reshape(-1)[:len(out[0])])   # the first token sees itself
