"""The Gezavik decoder on the CPU: its configuration, the model's description, and the plain implementation's own
mechanisms against closed forms."""
import copy

import numpy as np
import pytest

import gezavik_models as M
import plain_gezavik as P


@pytest.mark.parametrize("which", sorted(M.CONFIGS))
def test_configuration_round_trip_and_declared_tensors(which):
    from hk_b200.config import GezavikConfig, config_from_dict, resolve_architecture
    raw = M.CONFIGS[which]
    cfg = config_from_dict(raw)
    assert isinstance(cfg, GezavikConfig) and config_from_dict(cfg.to_dict()).to_dict() == cfg.to_dict()
    _, build = resolve_architecture("Gezavik")
    model = build(cfg, 64)
    specs = model.param_specs()
    d = raw["width"]
    assert specs["embed"].shape == specs["head"].shape == (raw["vocab"], d) and not specs["head"].optional and "final.norm" in specs
    for i, layer in enumerate(raw["layers"]):
        m, mlp, p = layer["mixer"], layer["mlp"], f"l{i}."
        assert specs[p + "norm1"].shape == (d,) and p + "norm2" not in specs
        if layer["type"] == "mamba2":
            inner, bc = m["heads"] * m["vdim"], 2 * m["groups"] * m["state"]
            assert specs[p + "mix.in"].shape == (2 * inner + bc + m["heads"], d)
            assert specs[p + "mix.conv"].shape == (inner + bc, m["conv"]) and specs[p + "mix.conv.b"].shape == (inner + bc,)
            for name in ("dt_bias", "A_log", "D"):
                assert specs[p + "mix." + name].shape == (m["heads"],)
            assert specs[p + "mix.norm"].shape == (inner,) and specs[p + "mix.o"].shape == (d, inner)
        else:
            H = m["heads"]
            assert specs[p + "mix.dq"].shape == (m["q_rank"], d) and specs[p + "mix.dq.norm"].shape == (m["q_rank"],)
            assert specs[p + "mix.uq"].shape == (H * (m["dim"] + m["rot_dim"]), m["q_rank"]) and p + "mix.q" not in specs
            assert specs[p + "mix.dkv"].shape == (m["kv_rank"] + m["rot_dim"], d) and specs[p + "mix.dkv.norm"].shape == (m["kv_rank"],)
            assert specs[p + "mix.uk"].shape == (H * m["dim"], m["kv_rank"]) and specs[p + "mix.uv"].shape == (H * m["vdim"], m["kv_rank"])
            assert specs[p + "mix.g"].shape == (H, d) and specs[p + "mix.o"].shape == (d, H * m["vdim"])
        if mlp is None:
            assert not any(n.startswith(p + "mlp.") for n in specs)
        elif mlp["kind"] == "moe":
            E, outputs = mlp["router"]["experts"], mlp["router"]["experts"] + mlp["router"]["identity"]
            assert specs[p + "mlp.router"].shape == (outputs, d) and specs[p + "mlp.correction"].shape == (outputs,)
            assert p + f"mlp.e{E - 1}.down" in specs and p + f"mlp.e{E}.down" not in specs
            assert (p + "mlp.shared.up" in specs) == bool(mlp.get("shared"))
        else:
            assert specs[p + "mlp.up"].shape == (mlp["ff"], d) and p + "mlp.gate" not in specs
    # the caches: a state and the convolution's tail per state-space layer, one row per token for the others
    for layer, caches in zip(raw["layers"], model.cache_specs()):
        m = layer["mixer"]
        if layer["type"] == "mamba2":
            assert caches[0].shape == (m["heads"], m["vdim"], m["state"]) and len(caches) == 2
            assert caches[1].shape == (max(m["conv"] - 1, 1), m["heads"] * m["vdim"] + 2 * m["groups"] * m["state"])
        else:
            assert caches[0].k_dim == m["kv_rank"] + m["rot_dim"] and caches[0].v_dim == 0
            assert caches[0].window == (m["mask"]["size"] if m.get("mask") else None)


def test_configuration_errors_name_the_key():
    from hk_b200.config import ConfigError, config_from_dict
    for path, value, word in ((("layers", 0, "mixer", "groups"), 4, "groups"), (("layers", 0, "mixer", "norm_groups"), 5, "norm_groups"),
                              (("layers", 0, "mlp", "router", "top"), 7, "top"), (("layers", 0, "mlp", "expert", "limit"), 0.0, "limit"),
                              (("layers", 3, "mlp", "shared", "limit"), -1.0, "limit"), (("layers", 1, "mixer", "rot", "dims"), 6, "dims"),
                              (("layers", 1, "type"), "attention", "type"), (("layers", 1, "mixer", "q_rank"), None, "q_rank"),
                              (("residual_mult",), "x", "residual_mult"), (("norm", "eps"), 0.0, "eps")):
        raw = copy.deepcopy(M.CONFIGS["A"])
        at = raw
        for key in path[:-1]:
            at = at[key]
        at[path[-1]] = value
        with pytest.raises(ConfigError, match=word):
            config_from_dict(raw)


def test_the_residual_factor_rides_on_the_sublayers():
    from hk_b200.config import config_from_dict, resolve_architecture
    from hk_b200.parts import ParallelBlock, RMSNorm, SquaredReLUFeedForward, SwiGLUFeedForward
    raw = M.CONFIGS["C"]
    model = resolve_architecture("Gezavik")[1](config_from_dict(raw), 8)
    for block in model.layers:
        assert isinstance(block, ParallelBlock) and block._carried
        assert block.mixer.out_scale == block.feed_forward.out_scale == raw["residual_mult"]
    # a sublayer that cannot carry it: neither is given it, and the block adds their sum itself
    mixer = SquaredReLUFeedForward(8, 16, "m.")
    block = ParallelBlock(RMSNorm(8, 1e-5, "n"), mixer, SwiGLUFeedForward(8, 16, "f."), 0.5)
    assert not block._carried and mixer.out_scale == 1.0


def test_state_space_tables_part_long_requests_from_short_ones():
    from hk_b200.parts import StateSpace
    from types import SimpleNamespace
    part = StateSpace(16, 2, 8, 8, 1, 3, "m.", 1e-5)
    ctx = SimpleNamespace(slots=[4, 1, 0, 2], q_starts=[0, 31, 63, 64], q_lens=[31, 32, 1, 200])
    np.testing.assert_array_equal(part.step_tables(ctx).arrays["segments"], [[4, 0, 31], [1, 31, 32], [0, 63, 1], [2, 64, 200]])
    part._chunks = True
    arrays = part.step_tables(ctx).arrays
    np.testing.assert_array_equal(arrays["short"], [[4, 0, 31], [0, 63, 1]])
    np.testing.assert_array_equal(arrays["long"], [[1, 31, 32], [2, 64, 200]])
    ctx = SimpleNamespace(slots=[3], q_starts=[0], q_lens=[1])
    assert part.step_tables(ctx).arrays["long"].shape == (0, 3)


def test_plain_state_space_walk_is_its_closed_form():
    rng = np.random.default_rng(0)
    T, H, G, N, dv = 14, 4, 2, 3, 5
    x, B, C = rng.standard_normal((T, H, dv)), rng.standard_normal((T, G, N)), rng.standard_normal((T, G, N))
    dt, a_log, skip = P.softplus(rng.standard_normal((T, H))), rng.standard_normal(H) * 0.3 - 1.0, rng.standard_normal(H)
    want = np.zeros((T, H, dv))
    for h in range(H):
        g = h // 2
        for t in range(T):
            want[t, h] = skip[h] * x[t, h]
            for s in range(t + 1):
                decay = np.exp(-np.exp(a_log[h]) * dt[s + 1:t + 1, h].sum())
                want[t, h] += decay * dt[s, h] * (C[t, g] @ B[s, g]) * x[s, h]
    np.testing.assert_allclose(P.state_space_walk(x, B, C, dt, a_log, skip), want, rtol=1e-10, atol=1e-10)


def test_plain_gated_norm_cuts_across_heads_and_gates_before_it():
    rng = np.random.default_rng(1)
    y, z, w = rng.standard_normal((3, 12)), rng.standard_normal((3, 12)), rng.standard_normal(12)
    got = P.gated_group_norm(y, z, w, 3, 1e-5)
    u = y * z / (1.0 + np.exp(-z))
    for part in range(3):
        c = slice(4 * part, 4 * part + 4)
        np.testing.assert_allclose(got[:, c], u[:, c] / np.sqrt((u[:, c] ** 2).mean(axis=1, keepdims=True) + 1e-5) * w[c])
    assert np.abs(P.gated_group_norm(y, z, w, 1, 1e-5) - got).max() > 0.1


def test_plain_router_weights_and_identities():
    z = np.array([2.0, -1.0, 1.5, -0.4, 3.0, 0.2])
    s = np.exp(z) / np.exp(z).sum()
    chosen, weights, margin = P.route(z, np.zeros(6), 3)
    assert chosen == [4, 0, 2] and np.isclose(margin, s[2] - s[5])
    np.testing.assert_allclose(weights, s[chosen])                       # as they are: their sum stays below 1
    corr = np.array([0.0, 5.0, 0.0, 0.0, -1.0, 0.0])                     # moves the choice, not the weights
    chosen, weights, _ = P.route(z, corr, 2)
    assert chosen == [1, 0]
    np.testing.assert_allclose(weights, s[[1, 0]])
    # experts 0 and 1 and one identity, all chosen: the identity gives back the input times its score
    rng = np.random.default_rng(2)
    d, F = 5, 4
    w = {"f.router": rng.standard_normal((3, d)), "f.correction": np.zeros(3)}
    for e in range(2):
        w.update({f"f.e{e}.gate": rng.standard_normal((F, d)), f"f.e{e}.up": rng.standard_normal((F, d)), f"f.e{e}.down": np.zeros((d, F))})
    h = rng.standard_normal((4, d))
    zz = h @ w["f.router"].T
    sc = np.exp(zz) / np.exp(zz).sum(axis=1, keepdims=True)
    mlp = {"kind": "moe", "expert": {"ff": F, "limit": 1.0}, "router": {"experts": 2, "identity": 1, "top": 3}}
    np.testing.assert_allclose(P.routed_feed_forward(h, w, "f.", mlp), sc[:, 2:] * h)


def test_plain_convolution_and_rotation():
    x = np.arange(12.0).reshape(6, 2)
    wt = np.array([[1.0, 0.0, 0.0], [0.0, 0.0, 2.0]])            # channel 0: the input two rows back; channel 1: twice the current one
    y = P.short_conv(x, wt, np.array([0.5, -1.0]))
    np.testing.assert_allclose(y[:, 0], np.array([0, 0, 0, 2, 4, 6]) + 0.5)
    np.testing.assert_allclose(y[:, 1], x[:, 1] * 2 - 1.0)
    q = np.random.default_rng(1).standard_normal((5, 2, 6))
    r = P.rotate(q, np.arange(5), 100.0, 4)
    np.testing.assert_allclose(r[..., 4:], q[..., 4:])                                   # the rest passes unchanged
    np.testing.assert_allclose(np.linalg.norm(r, axis=-1), np.linalg.norm(q, axis=-1))   # a rotation
    np.testing.assert_allclose(r[0], q[0])                                               # position 0: angle 0
    a = 3 * 100.0 ** (-2.0 / 4)
    np.testing.assert_allclose(r[3, 1, 2], q[3, 1, 2] * np.cos(a) - q[3, 1, 3] * np.sin(a))   # neighbours are a pair
    np.testing.assert_allclose(r[3, 1, 3], q[3, 1, 3] * np.cos(a) + q[3, 1, 2] * np.sin(a))
