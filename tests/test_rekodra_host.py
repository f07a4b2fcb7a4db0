"""Rekodra on the CPU: configuration, graph, registry, cache layout, weight arrangements, and the oracle's own mechanisms
against other statements of them."""
import copy
import json

import numpy as np
import pytest
import torch

from oracle import rekodra as O
from rekodra_models import CONFIGS, attention, config, moe, parallel, random_weights, save_model


def _config(name):
    from cacheir_b200.rekodra import RekodraConfig
    return RekodraConfig.from_dict(CONFIGS[name])


def test_registry_builds_the_family(tmp_path):
    from cacheir_b200 import CompileArtifact, RekodraConfig, load_model, models

    assert "Rekodra" in models.architectures()
    art = load_model(save_model(tmp_path / "r", CONFIGS["fast"], random_weights(CONFIGS["fast"])))
    assert isinstance(art.config, RekodraConfig) and (art.config.hidden_size, art.config.vocab_size, art.config.num_layers) == (136, 168, 7)
    again = CompileArtifact.load(art.save(tmp_path / "artifact.json"))
    assert again.config.layers == art.config.layers and again.config.runs == art.config.runs and again.to_dict() == art.to_dict()
    with pytest.raises(ValueError):
        load_model(tmp_path / "r", quant="int8")


def test_graph_follows_the_configuration():
    from cacheir_b200.rekodra import build_rekodra_graph
    from cacheir_b200.topunex import UNBOUNDED

    graph = build_rekodra_graph(_config("fast"))
    ops = [n.op for n in graph.nodes]
    assert ops.count("tied_attention") == 7 and ops.count("matrix_memory") == 4 and ops.count("expert_mixture") == 5
    assert ops.count("add_token_embedding") == 1 and ops.count("residual_rms_pair") == 4 and ops.count("residual_add") == 3
    rejoin = next(i for i, n in enumerate(graph.nodes) if n.op == "add_token_embedding")
    assert graph.nodes[rejoin - 1].name == "r2.mix_residual" and graph.nodes[rejoin + 1].name == "r3.norm1"
    shapes = {k: s.shape for k, s in graph.weights.items()}
    assert shapes["l0.mlp.router"] == (12, 136) and shapes["l0.mlp.correction"] == (12,) and shapes["l0.mlp.shared.sg"] == (1, 136)
    assert shapes["l1.mix.k.norm"] == (80,) and "l1.mix.v" not in shapes and shapes["l0.mix.left.v"] == (48, 136) and shapes["l0.mix.left.k.norm"] == (40,)
    assert "l1.mlp.shared.sg" not in shapes and "l2.norm2" not in shapes and "head" not in shapes and "l0.mix.left.sink" not in shapes
    at = [n.attrs for n in graph.nodes if n.op == "tied_attention"]
    assert [a["layer"] for a in at] == list(range(7))
    assert (at[0]["window"], at[0]["key_dim"], at[1]["window"], at[1]["whole_norm"], at[4]["rot_dims"]) == (37, 40, UNBOUNDED, True, 24)


def test_every_pass_has_a_cache_and_state_of_its_own():
    from cacheir_b200.hybrid_ops import memory_state_size

    cfg = _config("fast")
    pools, states = cfg.cache_layout(64, torch.bfloat16)
    assert sorted(pools) == list(range(7)) and sorted(states) == [0, 2, 3, 5]
    assert pools[0]["rows"] == pools[3]["rows"] == ((2, 64, 64), torch.bfloat16) and pools[4]["rows"] == ((2, 64, 64), torch.bfloat16)
    assert pools[6]["rows"] == ((1, 64, 128), torch.bfloat16) and pools[2]["inv_rms"] == ((3, 64), torch.float32)
    assert states[0] == (memory_state_size(3, 32, 72),) == ((3 * (32 * 72 + 32 + 1) + 3) // 4 * 4,)


@pytest.mark.parametrize("loop,runs", [(None, [0, 1, 2]), ((0, 3, 2), [0, 1, 2, 0, 1, 2]), ((1, 2, 3), [0, 1, 1, 1, 2]), ((2, 3, 1), [0, 1, 2])])
def test_layer_runs(loop, runs):
    from cacheir_b200.rekodra import RekodraConfig

    cfg = config(16, 16, [(attention(1, 1, 8), None)] * 3, loop=loop)
    got = [(r.layer, r.rejoin) for r in RekodraConfig.from_dict(cfg).runs]
    assert got == O.layer_runs(cfg) and [i for i, _ in got] == runs
    assert [n for n, (_, again) in enumerate(got) if again] == {None: [], (0, 3, 2): [3], (1, 2, 3): [2, 3], (2, 3, 1): []}[loop]


@pytest.mark.parametrize("change", [
    lambda c: c["layers"][1]["mixer"].update(kv_heads=4),
    lambda c: c["layers"][1]["mixer"].update(vdim=24),
    lambda c: c["layers"][1]["mixer"]["rot"].update(dims=42),
    lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7),
    lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=4),
    lambda c: c["layers"][0]["mixer"]["left"].update(mask={"size": 0}),
    lambda c: c["layers"][0]["mixer"]["right"].update(gate_cap=0.0),
    lambda c: c["layers"][0]["mixer"]["right"].update(dim=0),
    lambda c: c["layers"][0].update(type="linear"),
    lambda c: c["layers"][0]["mlp"].update(kind="dense"),
    lambda c: c["layers"][0]["mlp"]["router"].update(top=7),
    lambda c: c["layers"][0]["mlp"]["router"].update(identity=3),
    lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(keep=5),
    lambda c: c["layers"][0]["mlp"]["expert"].update(ff=0),
    lambda c: c.update(loop={"start": 2, "stop": 2, "times": 2}),
    lambda c: c.update(loop={"start": 0, "stop": 5, "times": 2}),
    lambda c: c.update(loop={"start": 0, "stop": 2, "times": 0}),
    lambda c: c.update(vocab=0),
])
def test_bad_configurations_are_refused(change):
    from cacheir_b200.rekodra import RekodraConfig

    cfg = copy.deepcopy(CONFIGS["fast"])
    change(cfg)
    with pytest.raises(ValueError):
        RekodraConfig.from_dict(cfg)


def test_json_configuration_round_trips():
    from cacheir_b200.rekodra import RekodraConfig

    for cfg in CONFIGS.values():
        parsed = RekodraConfig.from_dict(json.loads(json.dumps(cfg)))
        assert RekodraConfig.from_dict(parsed.to_dict()).layers == parsed.layers
    bare = {"kind": "moe", "expert": {"ff": 3}, "router": {"experts": 4, "top": 2}}
    cfg = config(8, 8, [(("attention", {"heads": 2, "kv_heads": 1, "dim": 8, "scale": 0.3}), bare)])
    layer = RekodraConfig.from_dict(cfg).layers[0]
    assert (layer.mixer.rot_dims, layer.mlp.identity, layer.mlp.groups, layer.mlp.keep, layer.mlp.shared_ff) == (0, 0, 1, 1, None)


def test_derived_weights_are_shared_by_the_passes():
    from cacheir_b200.rekodra import build_rekodra_graph
    from cacheir_b200.runtime import _Engine
    from cacheir_b200.weights import B200WeightStore, TensorSource

    w = random_weights(CONFIGS["fast"], seed=2)
    eng = _Engine.__new__(_Engine)
    eng.graph, eng.device, eng.dtype, eng._derived, eng._largest = build_rekodra_graph(_config("fast")), torch.device("cpu"), torch.float32, {}, {}
    eng.weights = B200WeightStore(TensorSource(w), eng.graph.weights, None, device=eng.device, dtype=eng.dtype)
    nodes = {n.name: n for n in eng.graph.nodes}
    first, second = (eng.concat_weight(tuple(nodes[f"r{r}.in_proj"].inputs[1:])) for r in (0, 3))
    assert first is second and np.array_equal(first[-3:].numpy(), w["l0.mix.right.f"]) and np.array_equal(first[:96].numpy(), w["l0.mix.right.q"])
    pairs = eng.paired_weight(("l0.mlp.shared.gate", "l0.mlp.shared.up"), ("l0.mlp.router", "l0.mlp.shared.sg")).numpy()
    assert np.array_equal(pairs[1:80:2], w["l0.mlp.shared.up"]) and np.array_equal(pairs[80:92], w["l0.mlp.router"])
    assert np.array_equal(pairs[92:], w["l0.mlp.shared.sg"])
    assert np.array_equal(eng.scaled_weight("final.norm", 0.5).numpy(), w["final.norm"] * 0.5)
    assert eng.largest_weight("l1.mix.q.norm") == float(np.abs(w["l1.mix.q.norm"]).max()) and eng.largest_weight("") == 1.0


# ---- the oracle's mechanisms -----------------------------------------------------------------------------------------------
def test_oracle_matrix_memory_equals_its_closed_form():
    """Unrolled: with F the running sum of forget gates, state weights are exp(F_t - F_s + i_s) over exp(m_t)."""
    rng = np.random.default_rng(1)
    n, heads, d, e = 13, 2, 4, 3
    q, k, v = rng.standard_normal((n, heads, d)), rng.standard_normal((n, heads, d)), rng.standard_normal((n, heads, e))
    gi, gf = rng.normal(0, 3, (n, heads)), O.log_sigmoid(rng.normal(1, 2, (n, heads)))
    got = O.matrix_memory(q, k, v, gi, gf)
    total = np.cumsum(gf, axis=0)
    for t in range(n):
        for h in range(heads):
            logs = total[t, h] - total[:t + 1, h] + gi[:t + 1, h]
            m = max(total[t, h], logs.max())
            a = np.exp(logs - m) * (k[:t + 1, h] @ q[t, h])
            want = (a @ v[:t + 1, h]) / (max(abs(a.sum()), np.exp(-m)) + 1e-6)
            np.testing.assert_allclose(got[t, h], want, rtol=1e-10)


def test_oracle_router_keeps_groups_and_weighs_without_the_correction():
    z = np.array([[0.0, 1.0, 2.0, 0.5, 1.5, 1.4]])
    s = O.softmax(z)
    np.testing.assert_allclose(s, np.exp(z) / np.exp(z).sum())
    correction = np.array([0.0, 0.0, -5.0, 0.0, 0.0, -0.3])
    chosen, weight = O.route(z, correction, 2, 3, 2)         # groups (0, 1), (2, 3), (4, 5): the best of the second is 3 at s[3]
    assert chosen.tolist() == [[4, 1]]
    np.testing.assert_allclose(weight, [[s[0, 4], s[0, 1]]])
    chosen, _ = O.route(z, correction, 3, 3, 2)              # the last one has a negative choice score and is still preferred to the dropped group
    assert chosen.tolist() == [[4, 1, 0]]
    assert O.route(z, np.zeros(6), 6)[0].tolist() == [[2, 4, 5, 1, 3, 0]]


def test_oracle_window_and_sink():
    got = O.seen(9, 3)
    for i in range(9):
        assert list(np.flatnonzero(got[i])) == [j for j in range(i + 1) if i - j < 3]
    q, k, v = np.zeros((2, 1, 4)), np.zeros((2, 1, 4)), np.ones((2, 1, 2))
    out = O.attend(q, k, v, 1.0, O.seen(2), np.array([np.log(2.0)]))
    np.testing.assert_allclose(out[:, 0, 0], [1 / 3, 2 / 4])
    np.testing.assert_allclose(O.attend(q, k, v, 1.0, O.seen(2, 1)), 1.0)


def test_oracle_causality_and_sensitivity_of_the_whole_model():
    cfg = CONFIGS["fast"]
    w = {k: a.astype(np.float64) for k, a in random_weights(cfg).items()}
    tokens = np.random.default_rng(2).integers(0, cfg["vocab"], 60)
    base, residuals = O.forward(cfg, w, tokens)
    assert len(residuals) == 7
    changed = tokens.copy()
    changed[41] = (changed[41] + 1) % cfg["vocab"]
    other, _ = O.forward(cfg, w, changed)
    assert np.array_equal(base[:41], other[:41]) and np.abs(base[41:] - other[41:]).max(axis=1).min() > 1e-6
    for name in ("l1.mix.sink", "l1.mix.q.norm", "l1.mix.k.norm", "l0.mix.left.k.norm", "l0.mix.right.i.b", "l0.mix.right.f", "l0.mix.right.norm",
                 "l0.mix.right.g", "l0.mix.left.out", "l2.mix.right.out", "l0.mlp.shared.sg", "l0.mlp.correction", "l3.mlp.router", "final.norm"):
        shift = np.linspace(-0.4, 0.4, w[name].size).reshape(w[name].shape)
        assert np.abs(O.forward(cfg, dict(w, **{name: w[name] * 1.25 + shift}), tokens)[0] - base).max() > 1e-4, name

    def changed_config(change):
        c = copy.deepcopy(cfg)
        change(c)
        return c
    for change in (lambda c: c["layers"][0]["mixer"]["left"].update(mask={"size": 38}), lambda c: c["layers"][0]["mixer"]["right"].update(gate_cap=4.0),
                   lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(keep=1), lambda c: c["loop"].update(times=3),
                   lambda c: c["layers"][1]["mixer"]["rot"].update(base=5000.0), lambda c: c["embedding"].update(scale=0.8),
                   lambda c: c.update(logit_scale=0.7)):
        assert np.abs(O.forward(changed_config(change), w, tokens)[0] - base).max() > 1e-4


def test_configurations_cover_every_branch():
    mixers = [e["mixer"] for cfg in CONFIGS.values() for e in cfg["layers"] if e["type"] == "attention"]
    lefts = [e["mixer"]["left"] for cfg in CONFIGS.values() for e in cfg["layers"] if e["type"] == "parallel"]
    mlps = [e["mlp"] for cfg in CONFIGS.values() for e in cfg["layers"]]
    assert any(m["rot"]["dims"] == 0 for m in mixers) and any(m["rot"]["dims"] == m["dim"] for m in mixers) and any(m["kv_heads"] == 1 for m in mixers)
    assert any(m["heads"] == m["kv_heads"] for m in lefts) and any(m["vdim"] > m["dim"] for m in lefts) and any(m["vdim"] < m["dim"] for m in lefts)
    assert None in mlps and any(m and "shared" not in m for m in mlps) and any(m and m["router"]["identity"] == 0 for m in mlps)
    assert any(m and m["router"]["groups"]["keep"] > 1 for m in mlps) and moe(2, 1, 3)["router"]["groups"]["count"] == 1
    assert parallel((1, 1, 2, 2, 1), (1, 1, 1, 1.0))[0] == "parallel"
