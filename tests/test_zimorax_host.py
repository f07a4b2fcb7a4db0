"""Zimorax on the CPU: configuration, graph, registry, cache layout, weight arrangements, rotation tables, and the oracle's own
mechanisms against other statements of them."""
import copy
import json
import math

import numpy as np
import pytest
import torch

from oracle import zimorax as O
from zimorax_models import CONFIGS, attention, config, delta, mamba2, random_weights, save_model


def _config(name):
    from cacheir_b200.zimorax import ZimoraxConfig
    return ZimoraxConfig.from_dict(CONFIGS[name])


def test_registry_builds_the_family(tmp_path):
    from cacheir_b200 import CompileArtifact, ZimoraxConfig, load_model, models

    assert "Zimorax" in models.architectures() and models.family_for({"architecture": "Zimorax"}).kernel_groups == ("ragged", "recurrence", "talking", "delta")
    art = load_model(save_model(tmp_path / "z", CONFIGS["fast"], random_weights(CONFIGS["fast"])))
    assert isinstance(art.config, ZimoraxConfig) and (art.config.hidden_size, art.config.vocab_size, art.config.num_layers) == (136, 168, 8)
    again = CompileArtifact.load(art.save(tmp_path / "artifact.json"))
    assert again.config.layers == art.config.layers and again.config.runs == art.config.runs and again.to_dict() == art.to_dict()
    with pytest.raises(ValueError):
        load_model(tmp_path / "z", quant="int8")


def test_graph_follows_the_configuration():
    from cacheir_b200.topunex import UNBOUNDED
    from cacheir_b200.zimorax import build_zimorax_graph

    graph = build_zimorax_graph(_config("fast"))
    ops = [n.op for n in graph.nodes]
    assert [ops.count(o) for o in ("talking_attention", "delta_rule", "state_space", "short_conv", "join_embedding", "residual_add")] == [3, 3, 2, 5, 2, 14]
    joins = [i for i, n in enumerate(graph.nodes) if n.op == "join_embedding"]
    assert [graph.nodes[i].attrs["step"] for i in joins] == [0, 1]
    assert [(graph.nodes[i - 1].name, graph.nodes[i + 1].name) for i in joins] == [("r0.mlp_residual", "r1.norm1"), ("r2.mlp_residual", "r3.norm1")]
    shapes = {k: s.shape for k, s in graph.weights.items()}
    assert shapes["loop.in"] == (136, 272) and shapes["loop.step"] == (2, 136)
    assert shapes["l0.mix.in"] == (240 + 240 + 2 * 144 + 6, 136) and shapes["l0.mix.conv"] == (528, 4) and shapes["l0.mix.D"] == (6,)
    assert shapes["l1.mix.talk"] == (6, 6) and shapes["l1.mix.v.b"] == (48,) and shapes["l2.mix.q"] == (96, 136) and shapes["l2.mix.v.conv"] == (144, 3)
    assert shapes["l2.mix.norm"] == (24,) and shapes["l0.mix.norm"] == (240,) and "l3.norm2" not in shapes and "l3.ls2" not in shapes and "l2.mix.q.b" not in shapes
    at = [n.attrs for n in graph.nodes if n.op == "talking_attention"]
    assert [a["layer"] for a in at] == [1, 3, 5] and (at[0]["window"], at[2]["window"], at[0]["rot_dims"]) == (37, UNBOUNDED, 24)
    assert at[2]["yarn"] == [8.0, 128.0, 4.0, 1.0]
    plain = build_zimorax_graph(_config("wide"))
    assert [n.attrs["yarn"] for n in plain.nodes if n.name == "r7.attention"] == [None]


def test_every_pass_has_a_cache_and_state_of_its_own():
    from cacheir_b200.zimorax import state_floats

    cfg = _config("fast")
    pools, states = cfg.cache_layout(64, torch.bfloat16)
    assert sorted(pools) == [1, 3, 5] and sorted(states) == [0, 2, 4, 6, 7]
    assert pools[1] == pools[3] == {"key_rows": ((64, 80), torch.bfloat16), "value_rows": ((64, 48), torch.bfloat16)}
    assert states[0] == (6 * 40 * 48 + 3 * 528,) and states[2] == states[4] == (6 * 48 * 24 + 2 * 336,)
    offset, size = state_floats(_config("odd").layers[0].mixer)
    assert offset == 212 and size % 4 == 0 and size >= 212 + 4 * 41 and state_floats(_config("ones").layers[1].mixer) == (4, 4)


@pytest.mark.parametrize("loop,runs", [(None, [0, 1, 2]), ((0, 3, 2), [0, 1, 2, 0, 1, 2]), ((1, 2, 3), [0, 1, 1, 1, 2]), ((2, 3, 1), [0, 1, 2])])
def test_layer_runs(loop, runs):
    from cacheir_b200.zimorax import ZimoraxConfig, build_zimorax_graph

    cfg = config(16, 16, [(attention(1, 1, 8, 8), None)] * 3, loop=loop)
    parsed = ZimoraxConfig.from_dict(cfg)
    got = [(r.layer, r.begins) for r in parsed.runs]
    assert got == O.layer_runs(cfg) and [i for i, _ in got] == runs
    assert [(n, t) for n, (_, t) in enumerate(got) if t is not None] == {None: [], (0, 3, 2): [(0, 0), (3, 1)], (1, 2, 3): [(1, 0), (2, 1), (3, 2)],
                                                                        (2, 3, 1): [(2, 0)]}[loop]
    assert ("loop.in" in build_zimorax_graph(parsed).weights) == (loop is not None)


@pytest.mark.parametrize("change", [
    lambda c: c["layers"][1]["mixer"].update(kv_heads=4),
    lambda c: c["layers"][1]["mixer"].update(vdim=0),
    lambda c: c["layers"][1]["mixer"]["rot"].update(dims=42),
    lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7),
    lambda c: c["layers"][1]["mixer"]["rot"].update(base=1.0),
    lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].update(slow=0.0),
    lambda c: c["layers"][1]["mixer"].update(mask={"size": 0}),
    lambda c: c["layers"][0]["mixer"].update(groups=4),
    lambda c: c["layers"][0]["mixer"].update(norm_groups=7),
    lambda c: c["layers"][0]["mixer"].update(conv=0),
    lambda c: c["layers"][2]["mixer"].update(kv_heads=4),
    lambda c: c["layers"][2]["mixer"].update(dim=1.5),
    lambda c: c["layers"][0].update(type="linear"),
    lambda c: c["layers"][0]["mlp"].update(kind="moe"),
    lambda c: c["layers"][0]["mlp"].update(ff=0),
    lambda c: c.update(loop={"start": 2, "stop": 2, "times": 2}),
    lambda c: c.update(loop={"start": 0, "stop": 7, "times": 2}),
    lambda c: c.update(loop={"start": 0, "stop": 2, "times": 0}),
    lambda c: c.update(vocab=0),
])
def test_bad_configurations_are_refused(change):
    from cacheir_b200.zimorax import ZimoraxConfig

    cfg = copy.deepcopy(CONFIGS["fast"])
    change(cfg)
    with pytest.raises(ValueError):
        ZimoraxConfig.from_dict(cfg)


def test_json_configuration_round_trips():
    from cacheir_b200.zimorax import ZimoraxConfig

    for cfg in CONFIGS.values():
        parsed = ZimoraxConfig.from_dict(json.loads(json.dumps(cfg)))
        assert ZimoraxConfig.from_dict(parsed.to_dict()).layers == parsed.layers
    bare = config(8, 8, [(("attention", {"heads": 2, "kv_heads": 1, "dim": 8, "vdim": 4, "scale": 0.3}), None)])
    m = ZimoraxConfig.from_dict(bare).layers[0].mixer
    assert (m.rot_dims, m.rot_scaling, m.window) == (0, None, 1 << 30)


def test_derived_weights_are_shared_by_the_passes():
    from cacheir_b200.runtime import _Engine
    from cacheir_b200.weights import B200WeightStore, TensorSource
    from cacheir_b200.zimorax import build_zimorax_graph

    w = random_weights(CONFIGS["fast"], seed=2)
    eng = _Engine.__new__(_Engine)
    eng.graph, eng.device, eng.dtype, eng._derived, eng._largest = build_zimorax_graph(_config("fast")), torch.device("cpu"), torch.float32, {}, {}
    eng.weights = B200WeightStore(TensorSource(w), eng.graph.weights, None, device=eng.device, dtype=eng.dtype)
    nodes = {n.name: n for n in eng.graph.nodes}
    first, second = (eng.concat_weight(tuple(nodes[f"r{r}.in_proj"].inputs[1:])) for r in (2, 4))
    assert first is second and np.array_equal(first[-12:-6].numpy(), w["l2.mix.b"]) and np.array_equal(first[96:192].numpy(), w["l2.mix.k"])
    bias = eng.concat_bias(tuple(nodes["r1.in_proj"].attrs["bias"]), tuple(nodes["r1.in_proj"].inputs[1:]))
    assert np.array_equal(bias[240:320].numpy(), w["l1.mix.k.b"])
    taps = [eng.concat_f32(tuple(nodes[f"r{r}.conv"].inputs[2:])) for r in (2, 4)]
    assert taps[0] is taps[1] and np.array_equal(taps[0][192:].numpy(), w["l2.mix.v.conv"])


# ---- rotations ---------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dims,base,yarn", [(24, 10000.0, (4.0, 64.0, 8.0, 0.5)), (64, 500000.0, (16.0, 4096.0, 32.0, 1.0)), (2, 100.0, (2.0, 8.0, 1.0, 0.5)),
                                            (16, 7.0, (1.0, 100.0, 5.0, 2.0)), (32, 10000.0, (8.0, 32.0, 100.0, 50.0)), (8, 10.0, (40.0, 1e6, 4.0, 1.0))])
def test_yarn_frequencies(dims, base, yarn):
    from cacheir_b200.ragged import yarn_frequencies, yarn_table

    freq, factor = yarn_frequencies(dims, base, *yarn)
    want, by = O.yarn_frequencies(dims, base, dict(zip(("factor", "original", "fast", "slow"), yarn)))
    np.testing.assert_allclose(freq, want, rtol=1e-12)
    assert factor == pytest.approx(by) == pytest.approx(0.1 * math.log(yarn[0]) + 1.0)
    table = yarn_table(9, dims, base, yarn)
    assert table.dtype == np.float32 and table.shape == (9, dims // 2, 2)
    np.testing.assert_allclose(table[5, :, 0] / factor, np.cos(5 * want), atol=1e-6)
    # turning pairs keep their frequency, slow ones have it divided
    turns = yarn[1] * np.array([base ** (-2.0 * i / dims) for i in range(dims // 2)]) / (2 * math.pi)
    plain = np.array([base ** (-2.0 * i / dims) for i in range(dims // 2)])
    lo, hi = math.floor(dims * math.log(yarn[1] / (2 * math.pi * yarn[2])) / (2 * math.log(base))), math.ceil(
        dims * math.log(yarn[1] / (2 * math.pi * yarn[3])) / (2 * math.log(base)))
    for i in range(dims // 2):
        if i <= lo:
            assert freq[i] == pytest.approx(plain[i]) and turns[i] >= yarn[2] * 0.99
        if i >= hi > max(lo, 0):
            assert freq[i] == pytest.approx(plain[i] / yarn[0])


# ---- the oracle's mechanisms -----------------------------------------------------------------------------------------------
def test_oracle_state_space_equals_its_closed_form():
    rng = np.random.default_rng(1)
    n, heads, d, e = 11, 4, 3, 2
    x, b, c = rng.standard_normal((n, heads, e)), rng.standard_normal((n, 2, d)), rng.standard_normal((n, 2, d))
    dt, rate, skip = O.softplus(rng.normal(0, 1, (n, heads))), rng.normal(0, 1, heads), rng.standard_normal(heads)
    got = O.state_space(x, b, c, dt, rate, skip)
    total = np.cumsum(-np.exp(rate) * dt, axis=0)
    for t in range(n):
        for h in range(heads):
            g = h // 2
            a = np.exp(total[t, h] - total[:t + 1, h]) * dt[:t + 1, h] * (b[:t + 1, g] @ c[t, g])
            np.testing.assert_allclose(got[t, h], a @ x[:t + 1, h] + skip[h] * x[t, h], rtol=1e-9, atol=1e-12)


def test_oracle_delta_rule_equals_its_triangular_system():
    """All writes at once: (I + A) U = beta (V - exp(c) K S0) with S0 = 0."""
    rng = np.random.default_rng(2)
    n, heads, d, e = 12, 2, 5, 3
    q, k, v = rng.standard_normal((n, 1, d)), O.unit(rng.standard_normal((n, 1, d))), rng.standard_normal((n, heads, e))
    beta, decay = O.sigmoid(rng.normal(0, 1, (n, heads))), rng.uniform(0.3, 1.0, (n, heads))
    got = O.delta_rule(q, k, v, beta, decay)
    for h in range(heads):
        c = np.cumsum(np.log(decay[:, h]))
        d_ij = np.tril(np.exp(c[:, None] - c[None, :]))
        a = np.tril(beta[:, h:h + 1] * d_ij * (k[:, 0] @ k[:, 0].T), -1)
        u = np.linalg.solve(np.eye(n) + a, beta[:, h:h + 1] * v[:, h])
        np.testing.assert_allclose(got[:, h], (d_ij * (q[:, 0] @ k[:, 0].T)) @ u, rtol=1e-9, atol=1e-12)


def test_oracle_attention_mixes_scores_and_adds_one():
    q, k, v = np.zeros((2, 2, 4)), np.zeros((2, 1, 4)), np.ones((2, 1, 3))
    np.testing.assert_allclose(O.attend(q, k, v, 1.0, np.eye(2), O.seen(2))[:, 0, 0], [1 / 2, 2 / 3])
    q[:, 0, 0], k[:, 0, 0] = 1.0, np.log(2.0)
    talk = np.array([[0.0, 5.0], [3.0, 0.0]])                     # head 1 hears head 0 three times, head 0 hears nothing
    out = O.attend(q, k, v, 1.0, talk, O.seen(2, 1))
    np.testing.assert_allclose(out[:, :, 0], [[1 / 2, 8 / 9]] * 2)
    for i, row in enumerate(O.seen(9, 3)):
        assert list(np.flatnonzero(row)) == [j for j in range(i + 1) if i - j < 3]


def test_oracle_convolution_is_causal():
    x, taps = np.random.default_rng(3).standard_normal((6, 2)), np.array([[1.0, 10.0, 100.0], [0.0, 0.0, 1.0]])
    y = O.causal_conv(x, taps)
    want = 100 * x[:, 0] + 10 * np.r_[0, x[:-1, 0]] + np.r_[0, 0, x[:-2, 0]]
    np.testing.assert_allclose(y[:, 0], O.silu(want))
    np.testing.assert_allclose(y[:, 1], O.silu(x[:, 1]))


def test_oracle_causality_and_sensitivity_of_the_whole_model():
    cfg = CONFIGS["fast"]
    w = {k: a.astype(np.float64) for k, a in random_weights(cfg).items()}
    tokens = np.random.default_rng(2).integers(0, cfg["vocab"], 60)
    base, residuals = O.forward(cfg, w, tokens)
    assert len(residuals) == 8
    changed = tokens.copy()
    changed[41] = (changed[41] + 1) % cfg["vocab"]
    other, _ = O.forward(cfg, w, changed)
    assert np.array_equal(base[:41], other[:41]) and np.abs(base[41:] - other[41:]).max(axis=1).min() > 1e-6
    for name in w:
        shift = np.linspace(-0.4, 0.4, w[name].size).reshape(w[name].shape)
        assert np.abs(O.forward(cfg, dict(w, **{name: w[name] * 1.25 + shift}), tokens)[0] - base).max() > 1e-5, name

    def changed_config(change):
        c = copy.deepcopy(cfg)
        change(c)
        return c
    for change in (lambda c: c["layers"][1]["mixer"].update(mask={"size": 38}), lambda c: c["layers"][1]["mixer"].update(scale=0.3),
                   lambda c: c["layers"][1]["mixer"]["rot"].update(base=5000.0), lambda c: c["layers"][1]["mixer"]["rot"].update(dims=20),
                   lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].update(factor=5.0), lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].update(original=256.0),
                   lambda c: c["layers"][1]["mixer"]["rot"].pop("scaling"), lambda c: c["layers"][0]["mixer"].update(norm_groups=3),
                   lambda c: c["norm"].update(eps=1e-2)):
        assert np.abs(O.forward(changed_config(change), w, tokens)[0] - base).max() > 1e-5


def test_configurations_cover_every_branch():
    entries = [e for cfg in CONFIGS.values() for e in cfg["layers"]]
    att, ssm, dlt = ([e["mixer"] for e in entries if e["type"] == t] for t in ("attention", "mamba2", "delta"))
    assert any("rot" not in m for m in att) and any("mask" not in m for m in att) and any(m.get("rot", {}).get("dims") == m["dim"] for m in att)
    assert any("rot" in m and "scaling" not in m["rot"] for m in att) and any(m["mask"]["size"] == 1 for m in att if "mask" in m)
    assert any(m["heads"] == m["kv_heads"] for m in att) and any(m["kv_heads"] == 1 < m["heads"] for m in att)
    assert any(m["vdim"] > m["dim"] for m in att) and any(m["vdim"] < m["dim"] for m in att)
    assert {m["conv"] for m in ssm + dlt} >= {1, 2, 3, 4, 5, 6} and any(m["groups"] not in (1, m["heads"]) for m in ssm)
    assert any(m["kv_heads"] not in (1, m["heads"]) for m in dlt) and any(e["mlp"] is None for e in entries)
    assert {CONFIGS[n]["loop"]["start"] for n in CONFIGS} >= {0, 1} and mamba2(1, 1, 1)[0] == "mamba2" and delta(1, 1, 1, 1)[0] == "delta"
