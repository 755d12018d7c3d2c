"""The Nebanex decoder on the CPU: its configuration, the model's description, the table of the distance bias, and the plain
implementation's own mechanisms against closed forms."""
import copy

import numpy as np
import pytest
import torch

import nebanex_models as M
import plain_nebanex as P


@pytest.mark.parametrize("which", sorted(M.CONFIGS))
def test_configuration_round_trip_and_declared_tensors(which):
    from hk_b200.config import NebanexConfig, config_from_dict, resolve_architecture
    raw = M.CONFIGS[which]
    cfg = config_from_dict(raw)
    assert isinstance(cfg, NebanexConfig) and config_from_dict(cfg.to_dict()).to_dict() == cfg.to_dict()
    _, build = resolve_architecture("Nebanex")
    model = build(cfg, 64)
    specs, d = model.param_specs(), raw["width"]
    assert specs["embed"].shape == specs["head"].shape == (raw["vocab"], d) and not specs["head"].optional
    assert specs["final.norm"].shape == specs["final.norm.b"].shape == (d,)
    assert model.head.softcap == raw.get("logit_softcap", 0.0) and model.embedding.scale == raw["embedding"]["scale"]
    for i, layer in enumerate(raw["layers"]):
        a, r, mlp, p = layer["mixer"]["left"], layer["mixer"]["right"], layer["mlp"], f"l{i}."
        H, G, dk, dv = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
        ml, mr = p + "mix.left.", p + "mix.right."
        assert specs[p + "norm1"].shape == specs[p + "norm1.b"].shape == (d,)
        for name, rows in (("q", H * dk), ("k", G * dk), ("v", G * dv)):
            assert specs[ml + name].shape == (rows, d) and specs[ml + name + ".b"].shape == (rows,)
        assert specs[ml + "q.norm"].shape == (H * dk,) and specs[ml + "k.norm"].shape == (G * dk,)
        assert specs[ml + "g"].shape == (H * dv, d) and specs[ml + "o"].shape == (d, H * dv) and specs[ml + "o.b"].shape == (d,)
        assert specs[ml + "rel"].shape == (a["bias_rows"], H) and specs[ml + "out"].shape == specs[mr + "out"].shape == (d,)
        K, V = r["heads"] * r["dim"], r["heads"] * r["vdim"]
        for name, shape in (("q", (K, d)), ("k", (K, d)), ("v", (V, d)), ("g", (V, d)), ("o", (d, V)), ("norm", (r["vdim"],)),
                            ("a1", (r["decay_rank"], d)), ("a2", (K, r["decay_rank"])), ("a2.b", (K,))):
            assert specs[mr + name].shape == shape, name
        if mlp is None:
            assert not any(n.startswith(p + "mlp.") or n.startswith(p + "norm2") for n in specs)
        else:
            E = mlp["router"]["experts"]
            assert specs[p + "mlp.router"].shape == (E, d) and specs[p + "mlp.router.b"].shape == (E,)
            assert p + f"mlp.e{E - 1}.down" in specs and p + f"mlp.e{E}.down" not in specs
            assert (p + "mlp.shared.up" in specs) == bool(mlp.get("shared"))
    # the caches: pages of the heads' width in the kernels beside a state
    for layer, (pages, state) in zip(raw["layers"], model.cache_specs()):
        a, r = layer["mixer"]["left"], layer["mixer"]["right"]
        assert pages.n_kv_heads == a["kv_heads"] and pages.window is None and pages.k_dim >= a["dim"] and pages.v_dim >= a["vdim"]
        assert state.shape == (r["heads"], r["vdim"], r["dim"])


def test_sizes_that_only_the_file_gives():
    """Without `bias_rows` and `decay_rank` the tensors' own sizes are taken, and random weights are refused."""
    from hk_b200.config import config_from_dict, resolve_architecture
    from hk_b200.weights import random_tensors
    raw = copy.deepcopy(M.CONFIGS["A"])
    for e in raw["layers"]:
        del e["mixer"]["left"]["bias_rows"], e["mixer"]["right"]["decay_rank"]
    cfg = config_from_dict(raw)
    assert config_from_dict(cfg.to_dict()) == cfg and "bias_rows" not in str(cfg.to_dict())
    specs = resolve_architecture("Nebanex")[1](cfg, 8).param_specs()
    assert specs["l0.mix.left.rel"].shape == (-1, 6) and specs["l0.mix.right.a1"].shape == (-1, 48) and specs["l0.mix.right.a2"].shape == (24, -1)
    with pytest.raises(ValueError, match="only a file"):
        random_tensors(specs, 0, 0.1, 0.1, "cpu")


def test_configuration_errors_name_the_key():
    from hk_b200.config import ConfigError, config_from_dict
    for path, value, word in ((("layers", 0, "mixer", "left", "kv_heads"), 4, "kv_heads"), (("layers", 0, "mixer", "left", "bias_max"), 0, "bias_max"),
                              (("layers", 0, "mixer", "left", "q_temp", "every"), 0, "every"), (("layers", 0, "mixer", "right", "tau"), -1.0, "tau"),
                              (("layers", 0, "mixer", "right"), None, "right"), (("layers", 0, "mlp", "router", "top"), 6, "top"),
                              (("layers", 0, "mlp", "kind"), "dense", "kind"), (("layers", 1, "type"), "attention", "type"),
                              (("logit_softcap",), -2.0, "logit_softcap"), (("norm", "eps"), 0.0, "eps"), (("layers",), [], "layers")):
        raw = copy.deepcopy(M.CONFIGS["A"])
        at = raw
        for key in path[:-1]:
            at = at[key]
        at[path[-1]] = value
        with pytest.raises(ConfigError, match=word):
            config_from_dict(raw)


def test_parts_refuse_what_they_cannot_do():
    from hk_b200.parts import GQAAttention, GatedLinearAttention, ParallelMixer, RMSNorm, RotaryEmbedding, RoutedFeedForward
    rope = RotaryEmbedding(100.0, 4, 8)
    for more in ({"qk_norm_rows": True}, {"qk_norm_rows": True, "qk_norm_eps": 1e-5, "position": rope}, {"q_factor": (1.0, 0)},
                 {"pad_to": 8}, {"pad_to": 64, "qk_norm_eps": 1e-5}, {"pad_to": 64, "value_from_key": True}):
        with pytest.raises(ValueError):
            GQAAttention(32, 2, 1, 16, "m.", **more)
    with pytest.raises(ValueError):
        GatedLinearAttention(32, 2, 8, 8, 0.0, "m.", 1e-5)
    left, right = GQAAttention(32, 2, 1, 16, "l."), GatedLinearAttention(32, 2, 8, 8, 2.0, "r.", 1e-5)
    with pytest.raises(ValueError):
        ParallelMixer(left, right, left_norm=RMSNorm(32, 1e-5, "n"))
    with pytest.raises(ValueError):
        RoutedFeedForward(32, 16, 4, 2, "f.", scores="sigmoid", shared=left, shared_gated=True, router_bias=True)


@pytest.mark.parametrize("buckets,reach", [(16, 200), (8, 64), (32, 128), (2, 9), (7, 50), (64, 1000), (12, 9), (6, 4.5), (1, 5), (10, 5 * 2 ** 5)])
def test_distance_table_is_the_bucket_formula(buckets, reach):
    from hk_b200.parts.attention import distance_table
    rel = torch.arange(buckets * 3, dtype=torch.float32).reshape(buckets, 3)
    table = distance_table(rel, reach)
    assert table.shape[0] == 3
    for n in range(1500):
        want = rel[P.bucket(n, buckets, reach)]
        assert torch.equal(table[:, min(n, table.shape[1] - 1)], want), n


def test_distances_that_fall_on_a_row_exactly_belong_to_it():
    """reach = half * 16 with four rows above half: 16^(k/4) = 2^k, so rows start at 4, 8, 16 and 32 exactly."""
    from hk_b200.parts.attention import distance_starts
    assert distance_starts(8, 64) == [4, 8, 16, 32]
    assert [P.bucket(n, 8, 64) for n in (3, 4, 7, 8, 15, 16, 31, 32, 63, 64, 1000)] == [3, 4, 4, 5, 5, 6, 6, 7, 7, 7, 7]
    with pytest.raises(ValueError):
        distance_starts(8, 4)


def test_heads_filled_up_with_zeros():
    from hk_b200.parts.attention import _filled, padded_head
    assert padded_head(64, 64) is None and padded_head(48, 48) is None and padded_head(130, 8) is None
    assert padded_head(10, 10) == 64 and padded_head(64, 40) == 64 and padded_head(72, 24) == 128 and padded_head(16, 65) == 128
    t = torch.arange(12.0).reshape(6, 2)
    out = _filled(t, 2, 4).reshape(2, 4, 2)
    assert torch.equal(out[:, :3], t.reshape(2, 3, 2)) and not out[:, 3:].any() and _filled(t, 2, 3) is t


def test_gated_linear_tables_part_long_requests_from_short_ones():
    from types import SimpleNamespace

    from hk_b200.parts import GatedLinearAttention
    part = GatedLinearAttention(16, 2, 8, 8, 2.0, "m.", 1e-5)
    ctx = SimpleNamespace(slots=[4, 1, 0, 2], q_starts=[0, 127, 255, 256], q_lens=[127, 128, 1, 150])
    np.testing.assert_array_equal(part.step_tables(ctx).arrays["segments"], [[4, 0, 127], [1, 127, 128], [0, 255, 1], [2, 256, 150]])
    part._chunks = True
    arrays = part.step_tables(ctx).arrays
    np.testing.assert_array_equal(arrays["short"], [[4, 0, 127], [0, 255, 1]])
    np.testing.assert_array_equal(arrays["chunks"], [[127, 64], [191, 64], [256, 64], [320, 64], [384, 22]])
    np.testing.assert_array_equal(arrays["requests"], [[1, 0, 2], [2, 2, 3]])
    ctx = SimpleNamespace(slots=[3], q_starts=[0], q_lens=[1])
    arrays = part.step_tables(ctx).arrays
    assert arrays["chunks"].shape == (0, 2) and arrays["requests"].shape == (0, 3) and arrays["short"].shape == (1, 3)


def test_plain_attention_against_the_sums_written_out():
    rng = np.random.default_rng(0)
    d, H, G, dk, dv, T, B, D = 7, 4, 2, 3, 5, 12, 4, 6
    w = {"q": rng.standard_normal((H * dk, d)), "q.b": rng.standard_normal(H * dk), "k": rng.standard_normal((G * dk, d)),
         "k.b": rng.standard_normal(G * dk), "v": rng.standard_normal((G * dv, d)), "v.b": rng.standard_normal(G * dv),
         "q.norm": rng.standard_normal(H * dk), "k.norm": rng.standard_normal(G * dk), "rel": rng.standard_normal((B, H)),
         "g": rng.standard_normal((H * dv, d)), "o": np.eye(H * dv), "o.b": rng.standard_normal(H * dv)}
    h = rng.standard_normal((T, d))
    m = {"heads": H, "kv_heads": G, "dim": dk, "vdim": dv, "scale": 0.4, "bias_max": D, "q_temp": {"coef": 0.7, "every": 4}}
    got = P.attention(h, w, "", m, 1e-3)
    norm = lambda v, wt: v / np.sqrt((v ** 2).mean() + 1e-3) * wt            # noqa: E731
    t = T - 1
    for head in range(H):
        q = norm(w["q"] @ h[t] + w["q.b"], w["q.norm"])[head * dk:(head + 1) * dk] * (1 + 0.7 * np.log((t + 1) // 4 + 1))
        scores, values = [], []
        for j in range(T):
            k = norm(w["k"] @ h[j] + w["k.b"], w["k.norm"]).reshape(G, dk)[head // 2]
            row = t - j if t - j < 2 else min(3, 2 + int(np.log((t - j) / 2) / np.log(3) * 2))
            scores.append(0.4 * q @ k + w["rel"][row, head])
            values.append((w["v"] @ h[j] + w["v.b"]).reshape(G, dv)[head // 2])
        p = np.exp(scores) / np.exp(scores).sum()
        gate = 1 / (1 + np.exp(-(w["g"] @ h[t])[head * dv:(head + 1) * dv]))
        np.testing.assert_allclose(got[t, head * dv:(head + 1) * dv], p @ np.array(values) * gate + w["o.b"][head * dv:(head + 1) * dv])


def test_plain_gated_linear_walk_is_its_closed_form():
    rng = np.random.default_rng(1)
    T, H, dk, dv = 11, 2, 3, 4
    q, k, v = rng.standard_normal((T, H, dk)), rng.standard_normal((T, H, dk)), rng.standard_normal((T, H, dv))
    la = P.log_sigmoid(rng.standard_normal((T, H, dk)) * 3) / 4.0
    want = np.zeros((T, H, dv))
    for h in range(H):
        for t in range(T):
            for s in range(t + 1):
                want[t, h] += (q[t, h] * np.exp(la[s + 1:t + 1, h].sum(axis=0))) @ k[s, h] * v[s, h]
    np.testing.assert_allclose(P.gated_linear_walk(q, k, v, la), want, rtol=1e-10, atol=1e-10)
    np.testing.assert_allclose(np.exp(P.log_sigmoid(np.array([0.3, -40.0]))), 1 / (1 + np.exp([-0.3, 40.0])))


def test_plain_norms_router_and_cap():
    rng = np.random.default_rng(2)
    x, w, b = rng.standard_normal((3, 6)) + 5.0, rng.standard_normal(6), rng.standard_normal(6)
    want = (x - x.mean(axis=1, keepdims=True)) / np.sqrt(x.var(axis=1, keepdims=True) + 1e-2) * w + b
    np.testing.assert_allclose(P.layer_norm(x, w, b, 1e-2), want)
    z = np.array([2.0, -1.0, 1.5, -0.4, 3.0])
    chosen, weights, margin = P.route(z, 3)
    assert chosen == [4, 0, 2] and np.isclose(margin, 1.9)
    np.testing.assert_allclose(weights, np.exp(z[chosen]) / np.exp(z[chosen]).sum())
    np.testing.assert_allclose(P.query_factor([0, 6, 7, 15], 0.5, 8), 1 + 0.5 * np.log([1, 1, 2, 3]))
    np.testing.assert_allclose(P.soft_cap(np.array([0.1, 100.0]), 3.0), [3 * np.tanh(0.1 / 3), 3.0])
