"""Nipizen without a GPU: the configuration and its errors, tensor names and shapes, the cache and state each layer asks for, the
scaled rotation, what the parts refuse, random model folders, and the plain implementation's mechanisms against closed forms."""
import copy
import dataclasses
import math

import numpy as np
import pytest
import torch

import nipizen_helpers as H
import plain_nipizen as P


def test_configuration_reads_every_key_and_round_trips():
    import zinfer_b200 as z
    for name, d in H.CONFIGS.items():
        c = z.config_from_dict(d)
        assert c.architecture == "Nipizen" and c.vocab_size == d["vocab"] and c.hidden_size == d["width"]
        assert c.norm_eps == d["norm"]["eps"] and len(c.layers) == len(d["layers"])
        again = c.to_json_dict()
        assert dataclasses.replace(z.config_from_dict(again), raw={}) == dataclasses.replace(c, raw={})
        assert again["layers"] == d["layers"], name
    c = z.config_from_dict(H.CONFIGS["na"])
    a, r = c.layers[0].left, c.layers[0].right
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.rot_base, a.rot_dims, a.yarn) == (4, 2, 16, 12, 0.3, 1000.0, 8, (4.0, 64, 8.0, 0.5))
    assert (r.heads, r.kv_heads, r.dim, r.vdim, r.conv) == (4, 2, 12, 10, 3)
    assert (c.layers[0].left_scale, c.layers[0].right_scale) == (0.7, 0.9) and c.layers[2].mlp is None and c.layers[2].left.yarn is None
    m = c.layers[1].mlstm
    assert (m.heads, m.dim, m.vdim, m.gate_cap) == (3, 8, 10, 5.0) and c.layers[1].mlp.top == 1
    d = copy.deepcopy(H.CONFIGS["na"])                     # what a file leaves out is the plain form
    for k in ("left_scale", "right_scale"):
        del d["layers"][0]["mixer"][k]
    del d["layers"][0]["mixer"]["left"]["kv_heads"], d["layers"][0]["mixer"]["left"]["vdim"], d["layers"][0]["mixer"]["left"]["scale"]
    L = z.config_from_dict(d).layers[0]
    assert (L.left_scale, L.right_scale, L.left.kv_heads, L.left.vdim, L.left.scale) == (1.0, 1.0, 4, 16, 0.25)


@pytest.mark.parametrize("change,message", [
    (lambda d: d["layers"][0].update(type="mamba"), "known types"),
    (lambda d: d["layers"][0]["mixer"]["left"].update(kv_heads=3), "not a multiple"),
    (lambda d: d["layers"][0]["mixer"]["right"].update(kv_heads=3), "not a multiple"),
    (lambda d: d["layers"][0]["mixer"]["left"]["rot"].update(dims=3), "even"),
    (lambda d: d["layers"][0]["mixer"]["left"]["rot"].update(dims=18), "at most dim"),
    (lambda d: d["layers"][0]["mixer"]["left"]["rot"].pop("base"), "base"),
    (lambda d: d["layers"][0]["mixer"]["left"]["rot"]["scaling"].pop("slow"), "slow"),
    (lambda d: d["layers"][0]["mixer"]["left"]["rot"]["scaling"].update(factor=0), "positive"),
    (lambda d: d["layers"][0]["mixer"]["right"].pop("conv"), "conv"),
    (lambda d: d["layers"][0]["mixer"]["right"].update(conv=0), "conv"),
    (lambda d: d["layers"][0]["mixer"].pop("right"), "mixer.right"),
    (lambda d: d["layers"][1]["mixer"].pop("gate_cap"), "gate_cap"),
    (lambda d: d["layers"][1]["mixer"].update(gate_cap=0), "gate_cap"),
    (lambda d: d["layers"][0]["mlp"]["router"].update(top=7), "experts per token"),
    (lambda d: d["layers"][1]["mlp"].update(kind="dense"), "moe"),
    (lambda d: d["norm"].update(eps=0), "eps"),
    (lambda d: d.pop("vocab"), "vocab"),
])
def test_configuration_errors_name_the_key(change, message):
    import zinfer_b200 as z
    d = copy.deepcopy(H.CONFIGS["na"])
    change(d)
    with pytest.raises(z.ConfigError, match=message):
        z.config_from_dict(d)


def test_model_asks_for_the_tensors_of_the_design_and_storage():
    import zinfer_b200 as z
    from zinfer_b200.config.registry import build_model
    m = build_model(z.config_from_dict(H.CONFIGS["na"]))
    specs = m.weight_specs()
    want = {"embed": (97, 48), "final.norm": (48,), "l0.norm1": (48,), "l0.norm2": (48,),
            "l0.mix.left.q": (64, 48), "l0.mix.left.q.b": (64,), "l0.mix.left.k": (32, 48), "l0.mix.left.k.b": (32,),
            "l0.mix.left.v": (24, 48), "l0.mix.left.v.b": (24,), "l0.mix.left.q.norm": (64,), "l0.mix.left.k.norm": (32,),
            "l0.mix.left.g": (48, 48), "l0.mix.left.o": (48, 48), "l0.mix.right.q": (24, 48), "l0.mix.right.q.conv": (24, 3),
            "l0.mix.right.k": (24, 48), "l0.mix.right.k.conv": (24, 3), "l0.mix.right.v": (40, 48), "l0.mix.right.v.conv": (40, 3),
            "l0.mix.right.b": (4, 48), "l0.mix.right.A_log": (4,), "l0.mix.right.norm": (10,), "l0.mix.right.a1": (-1, 48),
            "l0.mix.right.a2": (48, -1), "l0.mix.right.dt_bias": (48,), "l0.mix.right.g1": (-1, 48), "l0.mix.right.g2": (40, -1),
            "l0.mix.right.o": (48, 40), "l0.mlp.router": (6, 48), "l0.mlp.e5.up": (24, 48), "l0.mlp.e0.down": (48, 24),
            "l1.mix.q": (24, 48), "l1.mix.v": (30, 48), "l1.mix.g": (30, 48), "l1.mix.i": (3, 48), "l1.mix.i.b": (3,),
            "l1.mix.f.b": (3,), "l1.mix.norm": (30,), "l1.mix.o": (48, 30)}
    for name, shape in want.items():
        assert specs[name].shape == shape, name
    assert "l2.norm2" not in specs and not any(n.startswith("l2.mlp") or ".gate" in n for n in specs)
    assert len(specs) == 2 + (2 + 10 + 15 + 13) + (2 + 10 + 9) + (1 + 10 + 15)
    assert "l2.norm2" in m.ignorable_weights
    cs = m.cache_specs()
    assert cs[0].kv.n_kv_heads == 2 and cs[0].kv.head_dim == 16 and cs[0].kv.v_dim == 12 and cs[1].kv is None
    assert cs[0].state.shape == (176 + 4 * 10 * 12,) and cs[0].state.dtype == torch.float32       # 2 rows of 88 inputs, the matrices
    assert cs[2].state.shape == (104 + 3 * 14 * 12,)                                              # 102 inputs and ten channels, rounded up
    assert cs[1].state.shape == (3 * 8 * 11 + 3 + 1,)                                             # normaliser column, maxima, rounded up


def test_inner_widths_that_do_not_meet_are_refused(tmp_path):
    import zinfer_b200 as z
    cfg = H.CONFIGS["nd"]
    W = H.make_weights(cfg, 1, (3, 5))
    assert z.load(H.write_folder(tmp_path / "good", cfg, W), dtype="fp32", device="cpu").layers[0].mixer.second.rank == 8
    W["l0.mix.right.a1"] = W["l0.mix.right.a1"][:2]
    with pytest.raises(ValueError, match="a1"):
        z.load(H.write_folder(tmp_path / "bad", cfg, W), dtype="fp32", device="cpu")


@pytest.mark.parametrize("rot", [H._rot(1000.0, 8, (4.0, 64, 8.0, 0.5)), H._rot(10000.0, 64, (16.0, 256, 32.0, 1.0)),
                                 H._rot(10000.0, 96, (8.0, 100, 1.0, 1.0)), H._rot(30.0, 6, (3.0, 20, 2.0, 0.3)), H._rot(500.0, 16)])
def test_scaled_rotation_against_the_plain_one(rot):
    from zinfer_b200.parts import RotaryEncoding
    s = rot.get("scaling")
    enc = RotaryEncoding(rot["dims"], rot["base"], yarn=tuple(s[k] for k in ("factor", "original", "fast", "slow")) if s else None)
    freq, amp = P.rotation(rot)
    assert np.allclose(enc.inv_freq_host(), freq, rtol=1e-6) and abs(enc.amplitude - amp) < 1e-12
    if s:
        plain = rot["base"] ** (-2.0 * np.arange(rot["dims"] // 2) / rot["dims"])
        assert plain[-1] / s["factor"] * (1 - 1e-12) <= freq[-1] < 0.6 * plain[-1] and abs(amp - 1.0) > 0.05 and np.all(freq <= plain * (1 + 1e-12))


def test_parts_refuse_what_no_kernel_takes():
    from zinfer_b200.parts import GatedDelta, GqaAttention, MixerPair, MLstm, Retention, RotaryEncoding, RoutedMoE
    names = [f"w{i}" for i in range(20)]
    with pytest.raises(ValueError):
        GatedDelta(16, 3, 2, 4, 4, 2, *names[:15])
    with pytest.raises(ValueError):
        GatedDelta(16, 2, 2, 4, 4, 0, *names[:15])
    with pytest.raises(ValueError):
        MLstm(16, 2, 4, 4, 0.0, *names[:10])
    with pytest.raises(ValueError):
        RoutedMoE(16, 8, 4, 2, "r", lambda e: (f"u{e}", f"d{e}"), weight_input=True, n_identity=1, act="relu")
    with pytest.raises(ValueError):
        RoutedMoE(16, 8, 4, 2, "r", lambda e: (f"u{e}", f"d{e}"), score="tanh")
    with pytest.raises(ValueError):
        GqaAttention(16, 2, 2, 4, *names[:4], head_gate_name="g", value_gate_name="h")
    with pytest.raises(ValueError):
        Retention(16, 1, 8, 8, [0.9], *names[:5], position=RotaryEncoding(8, 100.0, yarn=(4.0, 64, 8.0, 0.5)))
    a, m = GqaAttention(16, 2, 2, 4, *names[:4]), MLstm(16, 2, 4, 4, 1.0, *names[:10])
    for kw in (dict(), dict(first_norm_name="n", scales=(1.0, 1.0)), dict(first_norm_name="n")):
        with pytest.raises(ValueError):
            MixerPair(16, a, m, **kw)
    with pytest.raises(ValueError):
        MixerPair(16, m, m, scales=(1.0, 1.0))


def test_random_model_folders_load_back(tmp_path):
    import zinfer_b200 as z
    from zinfer_b200.weights.safetensors_io import SafetensorsFile
    cfg = z.config_from_dict(H.CONFIGS["ne"])
    folder = z.write_random_model(tmp_path / "m", cfg, seed=3)
    assert dataclasses.replace(z.config_from_folder(folder), raw={}) == dataclasses.replace(cfg, raw={})
    with SafetensorsFile(folder / "model.safetensors") as f:
        from zinfer_b200.config.registry import build_model
        assert sorted(f.names()) == sorted(build_model(cfg).weight_specs())
    assert z.load(folder, dtype="fp32", device="cpu").layers[0].mixer.second.w_high.shape[0] == 2 * 7 + 2 * 5


# ------------------------------------------------------------------------------- the plain implementation's own mechanisms

def test_plain_delta_rule_writes_what_the_key_does_not_read():
    """With beta 1 and no decay a unit key read back gives exactly the value written last under it, and writing again under
    the same key replaces it; a decay of one channel scales that channel's share alone."""
    q = k = np.zeros((3, 1, 2))
    k[0, 0] = k[2, 0] = [1.0, 0.0]
    k[1, 0] = [0.0, 1.0]
    v = np.array([[[5.0, 1.0]], [[7.0, 2.0]], [[-3.0, 4.0]]])
    one = np.ones((3, 1, 2))
    o = P.delta_scan(q, k, v, one, np.ones((3, 1)))
    assert np.allclose(o[:, 0], v[:, 0])
    o = P.delta_scan(np.array([[[1.0, 0.0]]] * 3), k, v, one, np.ones((3, 1)))
    assert np.allclose(o[:, 0], [[5, 1], [5, 1], [-3, 4]])
    o = P.delta_scan(np.array([[[1.0, 1.0]]] * 3), k, v, one * np.array([0.5, 1.0]), np.ones((3, 1)))
    assert np.allclose(o[1, 0], [0.5 * 5 + 7, 0.5 * 1 + 2])


def test_plain_mlstm_is_its_unstabilised_form():
    """S and n without the running maximum: o = S^T q / (max(|n . q|, 1) + 1e-6 exp(m)), since every term carries exp(-m)."""
    rng = np.random.default_rng(0)
    n, d, e = 12, 4, 3
    q, k, v = rng.normal(size=(n, 1, d)), rng.normal(size=(n, 1, d)), rng.normal(size=(n, 1, e))
    i, f = rng.normal(size=(n, 1)), P.log_sigmoid(rng.normal(size=(n, 1)))
    o = P.mlstm_scan(q, k, v, i, f)
    S, z, m = np.zeros((d, e)), np.zeros(d), 0.0
    for t in range(n):
        m = max(f[t, 0] + m, i[t, 0])
        S = math.exp(f[t, 0]) * S + math.exp(i[t, 0]) * np.outer(k[t, 0], v[t, 0])
        z = math.exp(f[t, 0]) * z + math.exp(i[t, 0]) * k[t, 0]
        assert np.allclose(o[t, 0], S.T @ q[t, 0] / (max(abs(z @ q[t, 0]), 1.0) + 1e-6 * math.exp(m)))


def test_plain_router_weighs_the_input():
    """Squared relu of a weighted input is the squared weight times the expert's output; scores are not renormalised."""
    rng = np.random.default_rng(1)
    h = rng.normal(size=(5, 6))
    W = {"router": rng.normal(size=(3, 6))}
    for e in range(3):
        W[f"e{e}.up"], W[f"e{e}.down"] = rng.normal(size=(4, 6)), rng.normal(size=(6, 4))
    s = P.sigmoid(h @ W["router"].T)
    full = P.moe(h, W, {"experts": 3, "top": 3})
    want = np.stack([sum(s[t, e] ** 2 * P.expert(h[t], W, e) for e in range(3)) for t in range(5)])
    assert np.allclose(full, want)
    one = P.moe(h, W, {"experts": 3, "top": 1})
    best = s.argmax(1)
    assert np.allclose(one, np.stack([s[t, best[t]] ** 2 * P.expert(h[t], W, best[t]) for t in range(5)]))


def test_plain_layer_norm_and_convolution():
    x = np.array([[1.0, 2.0, 3.0, 6.0]])
    y = P.layer_norm(x, np.array([1.0, 1.0, 2.0, 1.0]), 0.5)
    assert np.allclose(y, (x - 3.0) / math.sqrt(3.5 + 0.5) * [1, 1, 2, 1])
    c = P.short_conv_silu(np.array([[1.0], [2.0], [4.0]]), np.array([[10.0, 0.5]]))
    z = np.array([0.5, 11.0, 22.0])
    assert np.allclose(c[:, 0], z * P.sigmoid(z))
