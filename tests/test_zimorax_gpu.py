"""Zimorax through the runtime, scheduler, trace replay and command line, against the plain NumPy model."""
import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

from oracle import zimorax as O
from zimorax_models import CONFIGS, random_weights, row_errors, save_model

pytestmark = pytest.mark.gpu

ROOT = Path(__file__).resolve().parents[1]
TOL = {"float32": 2e-4, "bfloat16": 0.05}
_ORACLE: dict = {}


def _weights(name):
    if ("w", name) not in _ORACLE:
        _ORACLE["w", name] = random_weights(CONFIGS[name], seed=11)
    return _ORACLE["w", name]


def _want(name, tokens):
    """Logits of the plain model."""
    key = (name, tuple(tokens))
    if key not in _ORACLE:
        w = {k: a.astype(np.float64) for k, a in _weights(name).items()}
        _ORACLE[key] = O.forward(CONFIGS[name], w, tokens)[0]
    return _ORACLE[key]


def _tokens(name, n, seed):
    return [int(t) for t in np.random.default_rng(seed).integers(0, CONFIGS[name]["vocab"], n)]


def _runtime(name, dtype, *, pages=None, **kwargs):
    from cacheir_b200 import B200DecodeRuntime, ZimoraxConfig, build_zimorax_artifact
    from cacheir_b200.kv_cache import B200KVPageAllocator

    alloc = B200KVPageAllocator(page_size=64, initial_slots=pages or 4, max_slots=pages)
    return B200DecodeRuntime(build_zimorax_artifact(ZimoraxConfig.from_dict(CONFIGS[name])), tensor_source=_weights(name), dtype=dtype,
                             kv_allocator=alloc, max_seq_len=1024, **kwargs)


def _within(errors, dtype):
    """All rows in float32. In bfloat16 one in twenty may be over: a head of a few entries that nearly cancel (its norm makes them
    large again) turns operand roundings into more than that, also in a float64 model with rounded operands."""
    errors = np.asarray(errors)
    assert np.isfinite(errors).all()
    over, allowed = (errors > TOL[dtype]).sum(), 0 if dtype == "float32" else max(1, len(errors) // 20)
    assert over <= allowed and errors.max() <= (TOL[dtype] if dtype == "float32" else 0.6), (int(errors.argmax()), np.sort(errors)[-8:])


def _agree(got, want, dtype):
    _within(row_errors(got.float().cpu().numpy(), want), dtype)


@pytest.fixture(params=["float32", "bfloat16"])
def dtype(request):
    return request.param


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_prompt_logits_and_kernels_in_use(name, dtype):
    rt = _runtime(name, dtype)
    tokens = _tokens(name, 150, 1)
    _agree(rt.run([tokens])[0], _want(name, tokens), dtype)
    counts = rt.kernel_counts
    if dtype == "float32":
        assert not any("gemm" in k for k in counts) and "b200.dense_simple" in counts and "b200.delta_simple" in counts
    elif name in ("fast", "wide"):
        assert not any("simple" in k for k in counts), counts
        assert counts["b200.talking_prompt"] and counts["b200.delta_chunked"] and counts["b200.recurrence_chunked"]
    rt.check_device_status()


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_decoding_token_by_token_equals_the_prompt(name, dtype):
    rt = _runtime(name, dtype)
    tokens = _tokens(name, 140, 1)[:140]
    logits = [rt.run_decode_batch([rt], [t])[:, 0] for t in tokens]
    _agree(torch.cat(logits), _want(name, tokens), dtype)
    if dtype == "bfloat16" and name in ("fast", "wide"):
        assert all(rt.kernel_counts["b200." + k] for k in ("talking_step", "delta_step", "state_space_step")) and not any("simple" in k for k in rt.kernel_counts)
    assert rt.kv_cache.tokens == 140 and len(rt.kv_cache.pages) == 3 and rt.cache_stats()["graph_captures"] >= 1


@pytest.mark.parametrize("portion", [2, 3, 33, 64, 65])
@pytest.mark.parametrize("name", ["fast", "wide", "odd"])
def test_portions_of_any_size_give_the_same_logits(name, portion, dtype):
    rt = _runtime(name, dtype)
    tokens = _tokens(name, 137, 2)
    parts = [rt.run_step_batch([rt], [tokens[i:i + portion]], [list(range(len(tokens[i:i + portion])))]) for i in range(0, 137, portion)]
    _agree(torch.cat(parts), _want(name, tokens), dtype)


def _replay(rt, name, dtype, rng, requests, *, live, step_rows):
    """Random mixed steps: up to `live` requests at a time, each step some of them, portions and single tokens mixed."""
    waiting, active, errors = list(requests), {}, []
    while waiting or active:
        while waiting and len(active) < live:
            tokens = waiting.pop(0)
            active[id(tokens)] = [tokens, 0, rt.fork()]
        chosen = [a for a in active.values() if rng.random() < 0.8] or list(active.values())[:1]
        batches = []
        for tokens, at, _ in chosen:
            n = 1 if rng.random() < 0.4 else int(rng.integers(2, step_rows))
            batches.append(tokens[at:at + n])
        wanted = [sorted(set(int(p) for p in rng.integers(0, len(b), 3))) if rng.random() < 0.7 else [] for b in batches]
        logits = rt.run_step_batch([a[2] for a in chosen], batches, wanted)
        rows = [_want(name, a[0])[a[1] + p] for a, places in zip(chosen, wanted) for p in places]
        assert logits.shape[0] == len(rows)
        if rows:
            errors.extend(row_errors(logits.float().cpu().numpy(), np.stack(rows)))
        for a, b in zip(chosen, batches):
            a[1] += len(b)
            if a[1] == len(a[0]):
                a[2].kv_cache.clear()
                del active[id(a[0])]
    _within(errors, dtype)
    return len(errors)


@pytest.mark.parametrize("name", ["fast", "wide", "odd"])
def test_mixed_steps_with_pages_used_again(name, dtype):
    rng = np.random.default_rng(5)
    lengths = (190, 3, 64, 130, 65, 1, 128, 30, 70)
    requests = [_tokens(name, n, 20 + i) for i, n in enumerate(lengths)]
    rt = _runtime(name, dtype, pages=9)                     # fewer pages than the requests need in sum
    assert _replay(rt, name, dtype, rng, requests, live=3, step_rows=80) > 40
    stats = rt.kv_allocator.stats()
    assert stats["resident_pages"] == 0 and stats["allocated_pages_total"] > 9
    rt.check_device_status()


def test_a_long_prompt_spans_passes_and_long_decoding_follows(dtype):
    name = "fast"
    tokens = _tokens(name, 700, 3)
    rt = _runtime(name, dtype)
    rt._engine.prefill_chunk = 128                          # more passes than the default would take
    other = rt.fork()
    first = rt.run_step_batch([other, rt], [tokens[:5], tokens[:600]], [[4], [0, 127, 128, 383, 599]])
    want = _want(name, tokens)
    _agree(first, want[[4, 0, 127, 128, 383, 599]], dtype)
    got = [rt.run_step_batch([rt], [[t]]) for t in tokens[600:]]
    _agree(torch.cat(got), want[600:], dtype)
    _agree(torch.cat([rt.run_step_batch([other], [[t]]) for t in tokens[5:40]]), want[5:40], dtype)


def test_the_batch_does_not_change_a_sequence(dtype):
    name = "wide"
    prompts = [_tokens(name, n, 40 + n) for n in (100, 7, 66, 129)]
    rt = _runtime(name, dtype)
    together = [rt.fork() for _ in prompts]
    rt.run_step_batch(together, [p[:-6] for p in prompts])
    batch = torch.stack([rt.run_step_batch(together, [[p[i]] for p in prompts]) for i in range(-6, 0)])
    for j, p in enumerate(prompts):
        alone = rt.fork()
        alone.run_step_batch([alone], [p[:-6]])
        mine = torch.cat([alone.run_step_batch([alone], [[p[i]]]) for i in range(-6, 0)])
        _agree(batch[:, j], mine.double().cpu().numpy(), dtype)
        _agree(batch[:, j], _want(name, p)[-6:], dtype)


def test_nothing_is_reserved_when_a_step_does_not_fit():
    from cacheir_b200.kv_cache import KVPoolExhausted

    rt = _runtime("fast", "bfloat16", pages=3)
    a, b = rt.fork(), rt.fork()
    tokens = _tokens("fast", 200, 1)
    rt.run_step_batch([a], [tokens[:100]])
    with pytest.raises(KVPoolExhausted):
        rt.run_step_batch([a, b], [tokens[100:130], tokens[:65]])
    assert (a.kv_cache.tokens, b.kv_cache.tokens) == (100, 0)
    for bad in ([[10 ** 6]], [[-1]], [[]]):
        with pytest.raises(ValueError):
            rt.run_step_batch([a], bad)
    with pytest.raises(ValueError):
        rt.run_step_batch([a], [[1]], [[1]])
    with pytest.raises(ValueError):
        rt.run_step_batch([a, a], [[1], [1]])
    with pytest.raises(ValueError):
        _runtime("fast", "float16")
    _agree(rt.run_step_batch([a], [tokens[100:150]]), _want("fast", tokens)[[149]], "bfloat16")


def _greedy_alone(rt, prompt, steps):
    s = rt.fork()
    logits, ids = s.run_step_batch([s], [prompt]), []
    for _ in range(steps):
        ids.append(int(logits[-1].argmax()))
        logits = s.run_step_batch([s], [[ids[-1]]])
    s.kv_cache.clear()
    return ids


def test_greedy_generation_through_the_scheduler(dtype):
    from cacheir_b200.scheduler import BatchedDecodeLauncher

    name = "fast"
    rt = _runtime(name, dtype, pages=10)
    prompts = {f"r{n}": _tokens(name, n, 60 + n) for n in (90, 4, 65, 33)}
    alone = {k: _greedy_alone(rt, p, 12) for k, p in prompts.items()}
    if dtype == "float32":
        w = {k: a.astype(np.float64) for k, a in _weights(name).items()}
        p, ids = prompts["r33"], alone["r33"]
        logits = O.forward(CONFIGS[name], w, p + ids)[0]
        assert ids == [int(v) for v in logits[len(p) - 1:len(p) + 11].argmax(axis=1)]
    for step_tokens in (None, 6, 200):
        launcher = BatchedDecodeLauncher(rt, max_batch_size=3, step_tokens=step_tokens)
        for k, p in prompts.items():
            launcher.submit(p, max_new_tokens=12, request_id=k)
        out = launcher.run_until_complete()
        if dtype == "float32":
            assert out == alone
        else:       # roundings differ between batch shapes: ids may part where two logits are close
            same = sum(a == b for k in alone for a, b in zip(alone[k], out[k]))
            assert {k: len(v) for k, v in out.items()} == {k: 12 for k in alone} and same >= 30
        assert rt.kv_allocator.slots_in_use == 0


def test_device_feedback_decoding(dtype):
    rt = _runtime("fast", dtype, pages=8)
    prompts = [_tokens("fast", 60, 8), _tokens("fast", 9, 9)]
    alone = [_greedy_alone(rt, p, 70) for p in prompts]
    sessions = [rt.fork(), rt.fork()]
    logits = rt.run_step_batch(sessions, prompts)
    first = [int(v) for v in logits.argmax(dim=-1)]
    ids = rt.decode_greedy_batch(sessions, first, 69).cpu().numpy()
    got = [[f] + ids[:, j].tolist() for j, f in enumerate(first)]
    if dtype == "float32":
        assert got == alone
    else:
        assert sum(a == b for g, w in zip(got, alone) for a, b in zip(g, w)) >= 40


def test_trace_replay_and_command_line(tmp_path, dtype):
    name = "fast"
    folder = save_model(tmp_path / "m", CONFIGS[name], _weights(name))
    a, b, c = _tokens(name, 100, 1), _tokens(name, 50, 2), _tokens(name, 80, 4)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:70], "want": [0, 69]}, {"id": "b", "tokens": b[:2], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[2:49], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[70:71], "want": [0]}, {"id": "b", "tokens": b[49:], "want": [0]}], "end": ["b"]},
             {"step": 3, "entries": [{"id": "c", "tokens": c, "want": [79, 3]}, {"id": "a", "tokens": a[71:], "want": [28]}], "end": ["a", "c"]},
             {"step": 4, "entries": [{"id": "b", "tokens": b, "want": [49]}], "end": ["b"]}]
    out = tmp_path / "out"
    run = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(folder), "--dtype", dtype, "--out", str(out), "--max-tokens", "256"],
                         input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True)
    assert run.returncode == 0, run.stderr[-2000:]
    assert [line for line in run.stdout.splitlines() if line.startswith("done")] == [f"done {i}" for i in range(5)]
    want = {0: _want(name, a)[[0, 69]], 2: np.stack([_want(name, a)[70], _want(name, b)[49]]),
            3: np.stack([_want(name, c)[79], _want(name, c)[3], _want(name, a)[99]]), 4: _want(name, b)[[49]]}
    assert sorted(p.name for p in out.iterdir()) == [f"{i}.f32" for i in sorted(want)]
    for i, rows in want.items():
        _agree(torch.from_numpy(np.fromfile(out / f"{i}.f32", "<f4").reshape(rows.shape)), rows, dtype)
    gen = subprocess.run([sys.executable, "-m", "cacheir_b200", "--model", str(folder), "--tokens", ",".join(map(str, b)), "--prompt", "hello",
                          "--max-new-tokens", "5", "--dtype", dtype], cwd=ROOT, capture_output=True, text=True)
    assert gen.returncode == 0, gen.stderr[-2000:]
    lines = [json.loads(x) for x in gen.stdout.splitlines()]
    assert [x["prompt_tokens"] for x in lines] == [5, 50] and all(len(x["tokens"]) == 5 for x in lines)
    if dtype == "float32":
        assert lines[1]["tokens"][0] == int(_want(name, b)[49].argmax())


def test_prefixes_are_not_shared_without_their_state(dtype):
    rt = _runtime("fast", dtype)
    prompt = _tokens("fast", 140, 1)
    a, b = rt.fork(), rt.fork()
    a.prefill_tokens(prompt, use_prefix_cache=True, remember_prefix=True)
    logits, reused = b.prefill_tokens(prompt[:130] + [1, 2], use_prefix_cache=True)
    assert reused == () and rt.prefix_cache.stats()["entries"] == 0
    _agree(logits[0], _want("fast", prompt[:130] + [1, 2]), dtype)


def test_state_slots_run_out_and_are_used_again(dtype):
    from cacheir_b200 import B200DecodeRuntime, ZimoraxConfig, build_zimorax_artifact
    from cacheir_b200.kv_cache import B200KVPageAllocator, KVPoolExhausted

    alloc = B200KVPageAllocator(page_size=64, initial_slots=4, max_slots=4, initial_states=2, max_states=2)
    rt = B200DecodeRuntime(build_zimorax_artifact(ZimoraxConfig.from_dict(CONFIGS["fast"])), tensor_source=_weights("fast"), dtype=dtype,
                           kv_allocator=alloc, max_seq_len=256)
    tokens = [_tokens("fast", n, 70 + n) for n in (30, 45, 20)]
    a, b, c = (rt.fork() for _ in range(3))
    rt.run_step_batch([a, b], [tokens[0][:29], tokens[1][:40]])
    with pytest.raises(KVPoolExhausted):
        rt.run_step_batch([c], [tokens[2]])
    _agree(rt.run_step_batch([a], [tokens[0][29:]]), _want("fast", tokens[0])[29:], dtype)
    slot = a.kv_cache.state_slot
    a.kv_cache.clear()
    _agree(rt.run_step_batch([c, b], [tokens[2], tokens[1][40:]]), np.stack([_want("fast", tokens[2])[-1], _want("fast", tokens[1])[-1]]), dtype)
    assert c.kv_cache.state_slot == slot and alloc.stats()["states_in_use"] == 2


def test_residual_stream_after_every_layer_run():
    """The 32-bit residual, run by run: the graph cut behind each run, with everything before it."""
    from cacheir_b200 import B200DecodeRuntime, ZimoraxConfig, build_zimorax_artifact

    name = "fast"
    tokens = _tokens(name, 90, 5)
    w64 = {k: a.astype(np.float64) for k, a in _weights(name).items()}
    _, residuals = O.forward(CONFIGS[name], w64, tokens)
    for n in range(1, len(residuals) + 1):
        art = build_zimorax_artifact(ZimoraxConfig.from_dict(CONFIGS[name]))
        graph = art.graph("decode")
        last = max(i for i, node in enumerate(graph.nodes) if node.name.startswith(f"r{n - 1}."))
        final, head = graph.nodes[-2:]
        graph.nodes[last + 1:] = [final, head]
        final.inputs[0] = graph.nodes[last].outputs[0]
        rt = B200DecodeRuntime(art, tensor_source=_weights(name), dtype="float32", max_seq_len=128)
        rt.run([tokens])
        plan = next(p for p in rt._engine.plans.values() if not p.decode)
        got = plan._residual[:len(tokens)].double().cpu().numpy()
        err = np.abs(got - residuals[n - 1]).max() / np.abs(residuals[n - 1]).max()
        assert err <= 2e-5, (n, err)
