"""Gutorax on the CPU: configuration, graph, registry, safetensors reader, cache and state bookkeeping, mixed rounds, the
second library's ABI, and the oracle's own mechanisms against other statements of them."""
import copy
import ctypes
import json
import re
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

from gutorax_models import CONFIGS, config, latent, lightning, random_weights, save_model
from oracle import gutorax as G

ROOT = Path(__file__).resolve().parents[1]


@pytest.mark.parametrize("group", ["ragged", "hybrid", "recurrence", "experts"])
def test_libraries_export_every_declared_symbol(group):
    from cacheir_b200 import _lib, build

    build.build(groups=(group,))
    text = re.sub(r"/\*.*?\*/", "", (ROOT / "include" / f"cacheir_b200_{group}.h").read_text(), flags=re.S)
    declared = sorted(n for n in set(re.findall(r"\b(cacheir_b200_[a-z0-9_]+)\s*\(", text)))
    lib = ctypes.CDLL(str(_lib.GROUP_PATHS[group]))
    for name in declared + (list(_lib.SHARED_NAMES) if group == "ragged" else []):
        assert hasattr(lib, name), name
    assert sorted(_lib.GROUP_SIGNATURES[group]) == declared, "ctypes table and header disagree"


def test_what_the_tensor_core_kernels_take():
    from cacheir_b200 import _lib, build

    build.build(groups=("ragged", "hybrid", "recurrence"))
    ragged, hybrid, recurrence = (_lib.load_group(g) for g in ("ragged", "hybrid", "recurrence"))
    assert ragged.cacheir_b200_dense_supported(24, 24, 24, 1, 0) == 1
    assert ragged.cacheir_b200_dense_supported(20, 20, 24, 1, 0) == 0
    assert hybrid.cacheir_b200_latent_attention_supported(512, 64, 64, 2) == 1
    assert hybrid.cacheir_b200_latent_attention_supported(512, 64, 64, 0) == 0
    assert recurrence.cacheir_b200_recurrence_workspace_bytes(256, 3, 4, 16, 8) == 0
    assert recurrence.cacheir_b200_recurrence_workspace_bytes(512, 3, 4, 16, 8) == 11 * 4 * (16 * (8 + 1) + 1) * 4


def test_a_family_s_libraries_hold_only_what_it_needs():
    from cacheir_b200 import build, models

    files = {name: {src.stem for g in models.family_for({"architecture": name}).kernel_groups for src in build.group_sources(g)}
             for name in ("Gutorax", "Topunex", "Rekodra", "LlamaForCausalLM")}
    assert {"latent_attention", "linear_recurrence", "dense_gemm"} <= files["Gutorax"] and "tied_attention" not in files["Gutorax"]
    assert {"tied_attention", "grouped_gemm", "dense_gemm"} <= files["Topunex"] and not {"latent_attention", "qgemm_i8"} & files["Topunex"]
    assert {"tied_attention", "linear_recurrence", "grouped_gemm"} <= files["Rekodra"] and not {"latent_attention", "qgemm_i8"} & files["Rekodra"]
    assert "paged_attention_mma" in files["LlamaForCausalLM"] and "dense_gemm" not in files["LlamaForCausalLM"]
    assert {src.stem for g in build.LIB_PATHS for src in build.group_sources(g)} == {src.stem for src in build.CSRC.glob("*.cu")}


def test_argument_structs_have_the_compiler_s_layout(tmp_path):
    from cacheir_b200 import _lib

    names = {"cacheir_b200_dense_args": _lib.DenseArgs, "cacheir_b200_latent_args": _lib.LatentArgs,
             "cacheir_b200_recurrence_args": _lib.RecurrenceArgs, "cacheir_b200_tied_args": _lib.TiedArgs, "cacheir_b200_route_rule": _lib.RouteRule}
    lines = []
    for c_name, cls in names.items():
        lines.append(f'printf("%zu ", sizeof({c_name}));')
        lines += [f'printf("%zu ", offsetof({c_name}, {f[0]}));' for f in cls._fields_]
    src = tmp_path / "layout.c"
    src.write_text('#include <stdio.h>\n#include <stddef.h>\n#include "cacheir_b200_hybrid.h"\n#include "cacheir_b200_recurrence.h"\n#include "cacheir_b200_experts.h"\nint main(void){'
                   + "".join(lines) + "return 0;}")
    subprocess.run(["gcc", "-I", str(ROOT / "include"), str(src), "-o", str(tmp_path / "layout")], check=True)
    got = [int(v) for v in subprocess.run([str(tmp_path / "layout")], capture_output=True, text=True, check=True).stdout.split()]
    want = []
    for cls in names.values():
        want.append(ctypes.sizeof(cls))
        want += [getattr(cls, f[0]).offset for f in cls._fields_]
    assert got == want


def test_registry_chooses_the_family_by_architecture(tmp_path):
    from cacheir_b200 import CompileArtifact, GutoraxConfig, ModelConfig, load_model, models
    from cacheir_b200.tiny import create_tiny_model

    assert "Gutorax" in models.architectures()
    tiny = load_model(create_tiny_model(tmp_path / "tiny"))
    assert isinstance(tiny.config, ModelConfig) and tiny.graph().nodes[0].op == "token_embedding"
    art = load_model(save_model(tmp_path / "g", CONFIGS["fast"], random_weights(CONFIGS["fast"])))
    assert isinstance(art.config, GutoraxConfig) and art.config.vocab_size == 160
    again = CompileArtifact.load(art.save(tmp_path / "artifact.json"))
    assert again.config.layers == art.config.layers and again.to_dict() == art.to_dict()
    with pytest.raises(ValueError):
        load_model(tmp_path / "g", quant="int8")


def test_graph_follows_the_configuration():
    from cacheir_b200.gutorax import GutoraxConfig, build_gutorax_graph

    cfg = GutoraxConfig.from_dict(CONFIGS["fast"])
    graph = build_gutorax_graph(cfg)
    ops = [n.op for n in graph.nodes]
    assert ops.count("latent_attention") == 2 and ops.count("linear_recurrence") == 2 and ops.count("fused_geglu") == 3
    assert ops.count("token_side_gate") == 4 and "l2.mix.dkv" not in graph.weights and "l2.mlp.gate" not in graph.weights
    assert graph.weights["side.embed"].shape == (160, 24 * 4)
    pools, states = cfg.cache_layout(64, torch.bfloat16)
    assert list(pools) == [0] and pools[0]["latent"][0] == (64, 48 + 16)
    assert states == {1: (3, 32, 72), 3: (4, 16, 24)}
    shared = next(n for n in graph.nodes if n.name == "l2.attention")
    assert shared.attrs["cache_layer"] == 0 and len(shared.inputs) == 5
    assert "token_side_gate" not in [n.op for n in build_gutorax_graph(GutoraxConfig.from_dict(CONFIGS["no_side"])).nodes]


def test_every_graph_op_has_kernels_in_the_registry():
    from cacheir_b200 import _lib, registry
    from cacheir_b200.gutorax import GutoraxConfig, build_gutorax_graph

    used = {n.op for cfg in CONFIGS.values() for n in build_gutorax_graph(GutoraxConfig.from_dict(cfg)).nodes}
    assert used <= set(registry.HYBRID_KERNELS_FOR_OP)
    exported = {name for table in _lib.GROUP_SIGNATURES.values() for name in table}
    assert {k for names in registry.HYBRID_KERNELS_FOR_OP.values() for k in names} <= exported


@pytest.mark.parametrize("change", [
    lambda c: c["layers"][1]["mixer"]["decay"].append(0.5),
    lambda c: c["layers"][2]["mixer"].update(kv_from=1),
    lambda c: c["layers"][2]["mixer"].update(kv_from=2),
    lambda c: c["layers"][2]["mixer"].update(kv_rank=32),
    lambda c: c["layers"][0]["mixer"].update(mask={"size": 0}),
    lambda c: c["layers"][0].update(type="softmax"),
    lambda c: c["layers"][0]["mlp"].update(kind="experts"),
    lambda c: c.update(width=0),
])
def test_bad_configurations_are_refused(change):
    from cacheir_b200.gutorax import GutoraxConfig

    cfg = copy.deepcopy(CONFIGS["fast"])
    change(cfg)
    with pytest.raises(ValueError):
        GutoraxConfig.from_dict(cfg)


def test_safetensors_reader(tmp_path):
    from cacheir_b200.weights import SafetensorsFile, TensorSource

    w = random_weights(CONFIGS["no_side"], seed=3)
    folder = save_model(tmp_path / "m", CONFIGS["no_side"], w)
    f = SafetensorsFile(folder / "model.safetensors")
    assert set(f.entries) == set(w)
    for name, a in w.items():
        t = f.tensor(name)
        assert t.dtype == torch.bfloat16 and np.array_equal(t.float().numpy(), a)
    source = TensorSource(folder)
    assert np.array_equal(source.load("head", (), "model.safetensors").float().numpy(), w["head"])
    with pytest.raises(KeyError):
        source.load("absent", (), None)
    (tmp_path / "bad.safetensors").write_bytes(b"\xff" * 16)
    with pytest.raises(ValueError):
        SafetensorsFile(tmp_path / "bad.safetensors")


def _allocator(**kwargs):
    from cacheir_b200.kv_cache import B200KVPageAllocator

    alloc = B200KVPageAllocator(page_size=4, initial_slots=2, **kwargs)
    alloc.configure_layout(torch=torch, device="cpu", pools={0: {"latent": ((4, 6), torch.float32)}, 2: {"latent": ((4, 10), torch.float32)}},
                           states={1: (2, 3, 5)})
    return alloc


def test_latent_pools_and_state_slots():
    from cacheir_b200.kv_cache import B200PagedKVCache, KVPoolExhausted

    alloc = _allocator(max_slots=5, initial_states=1, max_states=2)
    assert alloc.pool_for_layer(0)["latent"].shape == (2, 4, 6) and alloc.pool_for_layer(1) is None
    assert alloc.page_bytes == 160
    a, b = B200PagedKVCache(alloc, 3), B200PagedKVCache(alloc, 3)
    a.extend(5)
    alloc.state_for_layer(1)[a.state_slot] = 7.0
    generation = alloc.generation
    b.extend(1)
    assert {a.state_slot, b.state_slot} == {0, 1} and alloc.generation > generation and float(alloc.state_for_layer(1)[0].min()) == 7.0
    assert alloc.pool_for_layer(2)["latent"].shape[0] >= 3 and alloc.free_slots() == 2 and alloc.free_states() == 0
    assert a.pages_needed(3) == 0 and a.pages_needed(4) == 1
    with pytest.raises(KVPoolExhausted):
        B200PagedKVCache(alloc, 3).extend(1)
    with pytest.raises(RuntimeError):
        B200PagedKVCache(alloc, 3).share_prefix(a, 4)
    slot, pages = a.state_slot, set(a.page_ids())
    a.clear()
    assert alloc.free_states() == 1 and a.state_slot is None
    c = B200PagedKVCache(alloc, 3)
    c.extend(8)
    assert c.state_slot == slot and set(c.page_ids()) == pages
    assert alloc.stats()["states_in_use"] == 2
    with pytest.raises(ValueError):
        alloc.configure_layout(torch=torch, device="cpu", pools={}, states={})


def test_steps_are_cut_into_passes():
    from cacheir_b200.runtime import cut_passes

    assert cut_passes([[0] * 5, [0], [0] * 6], 4) == [[(0, 0, 4)], [(0, 4, 5), (1, 0, 1), (2, 0, 2)], [(2, 2, 6)]]
    assert cut_passes([[0] * 4], 4) == [[(0, 0, 4)]]


class _FakeRuntime:
    """The next token is a function of the session's history, so any order of portions must give the same ids."""

    def __init__(self, alloc):
        self.kv_allocator, self.history, self.log = alloc, [], []
        self.artifact = type("A", (), {"config": type("C", (), {"vocab_size": 50})})

    def fork(self):
        from cacheir_b200.kv_cache import B200PagedKVCache
        child = _FakeRuntime(self.kv_allocator)
        child.log, child.kv_cache = self.log, B200PagedKVCache(self.kv_allocator, 1)
        return child

    def synchronize(self):
        pass

    def run_step_batch(self, sessions, batches, wanted):
        self.log.append([len(b) for b in batches])
        rows = []
        for s, b, want in zip(sessions, batches, wanted):
            s.kv_cache.extend(len(b))
            s.history += b
            rows += [torch.nn.functional.one_hot(torch.tensor((sum(s.history) * 7 + len(s.history)) % 50), 50).float() for _ in want]
        return torch.stack(rows) if rows else torch.empty(0, 50)


def test_mixed_rounds_generate_what_requests_alone_generate():
    from cacheir_b200.scheduler import BatchedDecodeLauncher

    prompts = {"a": list(range(1, 12)), "b": [4], "c": list(range(3, 26)), "d": [9, 9]}
    budget = {"a": 5, "b": 7, "c": 1, "d": 4}

    def run(step_tokens, batch, names):
        template = _FakeRuntime(_allocator(max_slots=12, max_states=3))
        launcher = BatchedDecodeLauncher(template, max_batch_size=batch, step_tokens=step_tokens)
        for n in names:
            launcher.submit(prompts[n], max_new_tokens=budget[n], request_id=n)
        out = launcher.run_until_complete()
        assert template.kv_allocator.slots_in_use == 0 and not template.kv_allocator.state_owners
        return out, template.log, launcher.metrics

    alone = {n: run(64, 1, [n])[0][n] for n in prompts}
    for step_tokens in (4, 6, 64):
        out, log, metrics = run(step_tokens, 4, prompts)
        assert out == alone and {n: len(t) for n, t in out.items()} == budget
        assert max(sum(step) for step in log) <= max(4, step_tokens)
        assert metrics.prefill_tokens == sum(map(len, prompts.values())) and metrics.generated_tokens == sum(budget.values())
    assert any(len(step) > 1 and max(step) > 1 and min(step) == 1 for step in run(6, 4, prompts)[1])     # portions beside decodes
    template = _FakeRuntime(_allocator(max_slots=2))
    launcher = BatchedDecodeLauncher(template, step_tokens=8)
    launcher.submit([1] * 9)
    with pytest.raises(RuntimeError):
        launcher.run_until_complete()


def test_command_lines_describe_themselves():
    for cmd in (["-m", "cacheir_b200", "--help"], [str(ROOT / "bin" / "trace_run"), "--help"]):
        out = subprocess.run([sys.executable] + cmd, cwd=ROOT, capture_output=True, text=True)
        assert out.returncode == 0 and "--model" in out.stdout


def test_rotation_table_matches_the_oracle():
    from cacheir_b200.ragged import rotate_half_table

    x = np.random.default_rng(0).standard_normal((50, 3, 10))
    table = rotate_half_table(50, 6, 777.0).astype(np.float64)
    c, s = table[:, None, :, 0], table[:, None, :, 1]
    want = np.concatenate([x[..., :3] * c - x[..., 3:6] * s, x[..., 3:6] * c + x[..., :3] * s, x[..., 6:]], -1)
    np.testing.assert_allclose(G.rotate_half(x, 777.0, 6), want, atol=1e-6)


def test_oracle_recurrence_equals_its_closed_form():
    rng = np.random.default_rng(1)
    q, k, v = rng.standard_normal((9, 2, 4)), rng.standard_normal((9, 2, 4)), rng.standard_normal((9, 2, 3))
    decay = [0.5, 0.9]
    out, state = G.decayed_outer_recurrence(q, k, v, decay)
    for h in range(2):
        i = np.arange(9)
        gap = i[:, None] - i[None, :]
        weights = np.where(gap >= 0, decay[h] ** np.maximum(gap, 0), 0.0) * (q[:, h] @ k[:, h].T)
        np.testing.assert_allclose(out[:, h], weights @ v[:, h], atol=1e-12)
    half, s = G.decayed_outer_recurrence(q[:4], k[:4], v[:4], decay)
    rest, s = G.decayed_outer_recurrence(q[4:], k[4:], v[4:], decay, s)
    np.testing.assert_allclose(np.concatenate([half, rest]), out)
    np.testing.assert_allclose(s, state)


def test_oracle_attention_sees_exactly_its_window_and_the_sink():
    n, window = 12, 4
    q = np.ones((n, 1, 1))
    k = np.zeros((n, 1, 1))
    v = np.eye(n)[:, None, :]
    out = G.windowed_sink_attention(q, k, v, 1.0, window, np.array([np.log(2.0)]))[:, 0]
    for i in range(n):
        seen = [j for j in range(n) if 0 <= i - j < window]
        want = np.zeros(n)
        want[seen] = 1.0 / (len(seen) + 2.0)
        np.testing.assert_allclose(out[i], want, atol=1e-12)


def test_oracle_causality_and_sensitivity_of_the_whole_model():
    cfg = CONFIGS["fast"]
    w = {k: a.astype(np.float64) for k, a in random_weights(cfg).items()}
    tokens = np.random.default_rng(2).integers(0, cfg["vocab"], 30)
    base, residuals = G.forward(cfg, w, tokens)
    assert len(residuals) == 4
    changed = tokens.copy()
    changed[17] = (changed[17] + 1) % cfg["vocab"]
    other, _ = G.forward(cfg, w, changed)
    assert np.array_equal(base[:17], other[:17]) and np.abs(base[17:] - other[17:]).max(axis=1).min() > 1e-6
    for name in ("l0.mix.sink", "l1.mix.norm", "l2.mix.uv", "l3.side.norm", "l0.norm1b.b", "final.norm.alpha"):
        moved = dict(w, **{name: w[name] * 1.25 + 0.1})
        assert np.abs(G.forward(cfg, moved, tokens)[0] - base).max() > 1e-4, name


def test_json_configuration_round_trips():
    from cacheir_b200.gutorax import GutoraxConfig

    for cfg in CONFIGS.values():
        parsed = GutoraxConfig.from_dict(json.loads(json.dumps(cfg)))
        assert GutoraxConfig.from_dict(parsed.to_dict()).layers == parsed.layers
    assert GutoraxConfig.from_dict(config(8, 8, [(lightning(1, 8, 8), 8), (latent(1, 8, 8, 8, 8, 8), 8)])).num_layers == 2
