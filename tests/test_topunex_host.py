"""Topunex on the CPU: configuration, graph, registry, weight arrangements, rotation tables, and the oracle's own mechanisms
against other statements of them."""
import copy
import json

import numpy as np
import pytest
import torch

from oracle import topunex as O
from topunex_models import CONFIGS, attention, config, dense, moe, random_weights, save_model


def _config(name):
    from cacheir_b200.topunex import TopunexConfig
    return TopunexConfig.from_dict(CONFIGS[name])


def test_registry_builds_the_family(tmp_path):
    from cacheir_b200 import CompileArtifact, TopunexConfig, load_model, models

    assert "Topunex" in models.architectures()
    art = load_model(save_model(tmp_path / "t", CONFIGS["fast"], random_weights(CONFIGS["fast"])))
    assert isinstance(art.config, TopunexConfig) and (art.config.hidden_size, art.config.vocab_size, art.config.num_layers) == (136, 168, 4)
    again = CompileArtifact.load(art.save(tmp_path / "artifact.json"))
    assert again.config.layers == art.config.layers and again.to_dict() == art.to_dict()
    with pytest.raises(ValueError):
        load_model(tmp_path / "t", quant="int8")


def test_graph_follows_the_configuration():
    from cacheir_b200.topunex import UNBOUNDED, build_topunex_graph

    cfg = _config("fast")
    graph = build_topunex_graph(cfg)
    ops = [n.op for n in graph.nodes]
    assert ops.count("tied_attention") == 4 and ops.count("expert_mixture") == 2 and ops.count("residual_rms_norm") == 5
    assert ops.count("combine_residual_rms_norm") == 2 and ops.count("fused_glu") == 2
    shapes = {k: s.shape for k, s in graph.weights.items()}
    assert shapes["l1.mlp.e6.down"] == (136, 24) and shapes["l1.mlp.shared.up"] == (40, 136) and shapes["l1.mlp.router"] == (7, 136)
    assert shapes["l0.mix.k.b"] == (80,) and "l0.mix.g.b" not in shapes and "l0.mix.v" not in shapes and "l1.mlp.e0.up.b" not in shapes
    assert "l2.mlp.shared.up" not in shapes and "l3.norm2" not in shapes and shapes["l3.mix.sink"] == (5,)
    at = {n.attrs["layer"]: n.attrs for n in graph.nodes if n.op == "tied_attention"}
    assert (at[0]["window"], at[0]["keep_first"], at[2]["window"], at[2]["softcap"]) == (37, 3, UNBOUNDED, None)
    assert at[1]["rot_scaling"] == [8.0, 1.0, 4.0, 64.0] and at[0]["rot_scaling"] is None
    pools, states = cfg.cache_layout(64, torch.bfloat16)
    assert states == {} and pools[0]["rows"] == ((2, 64, 64), torch.bfloat16) and pools[3]["inv_rms"] == ((5, 64), torch.float32)


def test_every_graph_op_has_kernels_in_the_registry():
    from cacheir_b200 import _lib, registry
    from cacheir_b200.gutorax import GutoraxConfig, build_gutorax_graph
    from cacheir_b200.rekodra import RekodraConfig, build_rekodra_graph
    from cacheir_b200.topunex import build_topunex_graph
    from gutorax_models import CONFIGS as OTHERS
    from rekodra_models import CONFIGS as THIRD
    from cacheir_b200.zimorax import ZimoraxConfig, build_zimorax_graph
    from zimorax_models import CONFIGS as FOURTH

    used = {n.op for name in CONFIGS for n in build_topunex_graph(_config(name)).nodes}
    used |= {n.op for cfg in OTHERS.values() for n in build_gutorax_graph(GutoraxConfig.from_dict(cfg)).nodes}
    used |= {n.op for cfg in THIRD.values() for n in build_rekodra_graph(RekodraConfig.from_dict(cfg)).nodes}
    used |= {n.op for cfg in FOURTH.values() for n in build_zimorax_graph(ZimoraxConfig.from_dict(cfg)).nodes}
    assert used == set(registry.HYBRID_KERNELS_FOR_OP)
    exported = {name for table in _lib.GROUP_SIGNATURES.values() for name in table}
    assert {k for names in registry.HYBRID_KERNELS_FOR_OP.values() for k in names} <= exported


@pytest.mark.parametrize("change", [
    lambda c: c["layers"][0]["mixer"].update(kv_heads=4),
    lambda c: c["layers"][0]["mixer"].update(vdim=24),
    lambda c: c["layers"][0]["mixer"]["rot"].update(dims=42),
    lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7),
    lambda c: c["layers"][0]["mixer"].update(softcap=0.0),
    lambda c: c["layers"][0]["mixer"].update(mask={"size": 0}),
    lambda c: c["layers"][0]["mixer"].update(mask={"size": 4, "keep_first": -1}),
    lambda c: c["layers"][0].update(type="linear"),
    lambda c: c["layers"][0]["mlp"].update(kind="tree"),
    lambda c: c["layers"][1]["mlp"]["router"].update(top=8),
    lambda c: c["layers"][1]["mlp"]["expert"].update(ff=0),
    lambda c: c.update(vocab=0),
])
def test_bad_configurations_are_refused(change):
    from cacheir_b200.topunex import TopunexConfig

    cfg = copy.deepcopy(CONFIGS["fast"])
    change(cfg)
    with pytest.raises(ValueError):
        TopunexConfig.from_dict(cfg)


def test_json_configuration_round_trips():
    from cacheir_b200.topunex import TopunexConfig

    for cfg in CONFIGS.values():
        parsed = TopunexConfig.from_dict(json.loads(json.dumps(cfg)))
        assert TopunexConfig.from_dict(parsed.to_dict()).layers == parsed.layers
    bare = {"heads": 2, "kv_heads": 1, "dim": 8, "scale": 0.3}
    mixer = TopunexConfig.from_dict(config(8, 8, [(bare, None)])).layers[0].mixer
    assert (mixer.rot_dims, mixer.keep_first, mixer.softcap, mixer.rot_scaling) == (0, 0, None, None)


@pytest.mark.parametrize("scaling", [None, (8.0, 1.0, 4.0, 64), (4.0, 1.0, 4.0, 1024), (2.0, 0.5, 3.0, 17)])
def test_rotation_table_matches_the_oracle(scaling):
    from cacheir_b200.ragged import rotary_frequencies, rotate_half_table

    named = None if scaling is None else dict(zip(("factor", "low", "high", "original"), scaling))
    freq = O.frequencies(24, 777.0, named)
    np.testing.assert_allclose(rotary_frequencies(24, 777.0, scaling), freq, rtol=1e-12)
    if scaling == (8.0, 1.0, 4.0, 64):            # all three bands are there
        plain = O.frequencies(24, 777.0)
        assert (freq == plain).any() and (freq == plain / 8).any() and ((freq < plain) & (freq > plain / 8)).any()
    x = np.random.default_rng(0).standard_normal((50, 3, 30))
    table = rotate_half_table(50, 24, 777.0, scaling).astype(np.float64)[:, None]
    c, s = table[..., 0], table[..., 1]
    want = np.concatenate([x[..., :12] * c - x[..., 12:24] * s, x[..., 12:24] * c + x[..., :12] * s, x[..., 24:]], -1)
    np.testing.assert_allclose(O.rotate_half(x, freq), want, atol=1e-5)


def test_frequencies_at_a_real_model_s_constants():
    """At a real model's constants fast pairs are kept and slow ones divided by the factor."""
    from cacheir_b200.ragged import rotary_frequencies

    plain, scaled = rotary_frequencies(128, 500000.0), rotary_frequencies(128, 500000.0, (8.0, 1.0, 4.0, 8192.0))
    assert np.array_equal(scaled[:20], plain[:20]) and np.allclose(scaled[-20:], plain[-20:] / 8) and np.all(np.diff(scaled) < 0)


def test_derived_weights_interleave_and_stack():
    from cacheir_b200.runtime import _Engine
    from cacheir_b200.topunex import build_topunex_graph
    from cacheir_b200.weights import B200WeightStore, TensorSource

    w = random_weights(CONFIGS["fast"], seed=2)
    eng = _Engine.__new__(_Engine)
    eng.graph, eng.device, eng.dtype, eng._derived = build_topunex_graph(_config("fast")), torch.device("cpu"), torch.float32, {}
    eng.weights = B200WeightStore(TensorSource(w), eng.graph.weights, None, device=eng.device, dtype=eng.dtype)
    pairs = eng.paired_weight(("l1.mlp.shared.gate", "l1.mlp.shared.up"), ("l1.mlp.router",)).numpy()
    assert np.array_equal(pairs[0:80:2], w["l1.mlp.shared.gate"]) and np.array_equal(pairs[1:80:2], w["l1.mlp.shared.up"])
    assert np.array_equal(pairs[80:], w["l1.mlp.router"])
    experts = eng.expert_pairs(tuple(f"l1.mlp.e{e}.gate" for e in range(7)), tuple(f"l1.mlp.e{e}.up" for e in range(7))).numpy()
    for e in range(7):
        assert np.array_equal(experts[48 * e:48 * (e + 1)][0::2], w[f"l1.mlp.e{e}.gate"])
        assert np.array_equal(experts[48 * e:48 * (e + 1)][1::2], w[f"l1.mlp.e{e}.up"])
    bias = eng.concat_bias(("l0.mix.q.b", None, "l0.mix.k.b"), ("l0.mix.q", "l0.mix.g", "l0.mix.k")).numpy()
    assert np.array_equal(bias[:240], w["l0.mix.q.b"]) and not bias[240:480].any() and np.array_equal(bias[480:], w["l0.mix.k.b"])
    assert np.array_equal(eng.paired_bias(("l0.mlp.gate.b", "l0.mlp.up.b")).numpy()[1::2], w["l0.mlp.up.b"])


# ---- the oracle's mechanisms -----------------------------------------------------------------------------------------------
def test_oracle_mask_sees_its_window_and_the_first_tokens():
    got = O.seen(9, 3, 2)
    for i in range(9):
        assert list(np.flatnonzero(got[i])) == sorted({j for j in range(i + 1) if i - j < 3 or j < 2})
    assert np.array_equal(O.seen(5), np.tril(np.ones((5, 5), bool)))


def test_oracle_sink_takes_its_share():
    score = np.zeros((1, 4))
    got = O.sink_softmax(score, np.array([[True, True, False, True]]), np.log(2.0))
    np.testing.assert_allclose(got, [[0.2, 0.2, 0.0, 0.2]])
    np.testing.assert_allclose(O.sink_softmax(score, np.ones((1, 4), bool), None), [[0.25] * 4])


def test_oracle_router_and_experts():
    z = np.array([[0.0, 2.0, 1.0, 2.0], [3.0, -1.0, 5.0, 4.0]])
    chosen, weight = O.route(z, 2, 0.5)
    assert chosen.tolist() == [[1, 3], [2, 3]]
    np.testing.assert_allclose(weight, 0.5 / (1 + np.exp(-np.take_along_axis(z, chosen, 1))))
    w = {"gate": np.array([[10.0]]), "up": np.array([[-10.0]]), "down": np.array([[1.0]])}
    np.testing.assert_allclose(O.clamped_expert(np.array([[1.0], [-1.0]]), w, "", 0.5).ravel(),
                               [0.5 / (1 + np.exp(-1.702 * 0.5)) * 0.5, -10.0 / (1 + np.exp(17.02)) * 1.5])


def test_oracle_causality_and_sensitivity_of_the_whole_model():
    cfg = CONFIGS["fast"]
    w = {k: a.astype(np.float64) for k, a in random_weights(cfg).items()}
    tokens = np.random.default_rng(2).integers(0, cfg["vocab"], 60)
    base, residuals = O.forward(cfg, w, tokens)
    assert len(residuals) == 4
    changed = tokens.copy()
    changed[41] = (changed[41] + 1) % cfg["vocab"]
    other, _ = O.forward(cfg, w, changed)
    assert np.array_equal(base[:41], other[:41]) and np.abs(base[41:] - other[41:]).max(axis=1).min() > 1e-6
    for name in ("l0.mix.sink", "l0.mix.q.b", "l1.mix.k.b", "l1.mlp.shared.up", "l2.mix.o.b", "l0.mlp.down.b", "l2.norm2", "l3.mix.g", "final.norm",
                 "l1.mlp.router"):
        moved = dict(w, **{name: w[name] * 1.25 + 0.1})
        assert np.abs(O.forward(cfg, moved, tokens)[0] - base).max() > 1e-4, name

    def with_mixer(i, **change):
        c = copy.deepcopy(cfg)
        c["layers"][i]["mixer"].update(change)
        return c
    for c in (with_mixer(0, mask={"size": 38, "keep_first": 3}), with_mixer(0, mask={"size": 37, "keep_first": 4}), with_mixer(0, softcap=29.0),
              with_mixer(0, scale=0.2), with_mixer(1, rot={"base": 500.0, "dims": 64})):
        assert np.abs(O.forward(c, w, tokens)[0] - base).max() > 1e-4


def test_configuration_helpers_cover_every_branch():
    kinds = {None if f is None else f["kind"] for cfg in CONFIGS.values() for _, f in ((e["mixer"], e["mlp"]) for e in cfg["layers"])}
    assert kinds == {None, "dense", "moe"}
    mixers = [e["mixer"] for cfg in CONFIGS.values() for e in cfg["layers"]]
    assert any(m["heads"] == m["kv_heads"] for m in mixers) and any(m["kv_heads"] == 1 for m in mixers)
    assert any("size" not in m["mask"] for m in mixers) and any("softcap" not in m for m in mixers) and any("scaling" in m["rot"] for m in mixers)
    assert dense(3)["kind"] == "dense" and moe(2, 1, 3)["router"]["top"] == 1 and attention(1, 1, 2)["vdim"] == 2
