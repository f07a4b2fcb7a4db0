"""Gutorax through the runtime, scheduler, trace replay and command line, against the plain NumPy model."""
import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

from gutorax_models import CONFIGS, config, latent, random_weights, row_errors, save_model
from oracle import gutorax as G

pytestmark = pytest.mark.gpu

ROOT = Path(__file__).resolve().parents[1]
TOL = {"float32": 2e-4, "bfloat16": 0.06}
_ORACLE: dict = {}


def _weights(name):
    if ("w", name) not in _ORACLE:
        _ORACLE["w", name] = random_weights(CONFIGS[name], seed=11)
    return _ORACLE["w", name]


def _want(name, tokens):
    key = (name, tuple(tokens))
    if key not in _ORACLE:
        _ORACLE[key] = G.forward(CONFIGS[name], {k: a.astype(np.float64) for k, a in _weights(name).items()}, tokens)[0]
    return _ORACLE[key]


def _tokens(name, n, seed):
    return [int(t) for t in np.random.default_rng(seed).integers(0, CONFIGS[name]["vocab"], n)]


def _runtime(name, dtype, *, pages=None, states=None, **kwargs):
    from cacheir_b200 import B200DecodeRuntime, GutoraxConfig, build_gutorax_artifact
    from cacheir_b200.kv_cache import B200KVPageAllocator

    alloc = B200KVPageAllocator(page_size=64, initial_slots=pages or 4, max_slots=pages, initial_states=2, max_states=states)
    return B200DecodeRuntime(build_gutorax_artifact(GutoraxConfig.from_dict(CONFIGS[name])), tensor_source=_weights(name), dtype=dtype,
                             kv_allocator=alloc, max_seq_len=1024, **kwargs)


def _agree(got, want, dtype, what=""):
    err = row_errors(got.float().cpu().numpy(), want)
    if dtype == "bfloat16" and what == "ones":      # an RMS norm over one element is a sign: a rounding near zero flips a row
        err = np.where(err <= np.quantile(err, 0.9), err, 0.0)
    assert np.isfinite(err).all() and err.max() <= TOL[dtype], (what, int(err.argmax()), float(err.max()))


@pytest.fixture(params=["float32", "bfloat16"])
def dtype(request):
    return request.param


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_prompt_logits_and_kernels_in_use(name, dtype):
    rt = _runtime(name, dtype)
    tokens = _tokens(name, 150, 1)
    _agree(rt.run([tokens])[0], _want(name, tokens), dtype, name)
    counts = rt.kernel_counts
    if dtype == "float32":
        assert not any("dense_gemm" in k for k in counts) and "b200.dense_simple" in counts
    elif name in ("fast", "wide_latent"):
        assert not any("simple" in k for k in counts), counts
        assert counts["b200.latent_attention"] and counts["b200.recurrence_chunked"] and counts["b200.dense_gemm.residual_dyt"]
    rt.check_device_status()


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_decoding_token_by_token_equals_the_prompt(name, dtype):
    rt = _runtime(name, dtype)
    tokens = _tokens(name, 140, 1)[:140]
    logits = [rt.run_decode_batch([rt], [t])[:, 0] for t in tokens]
    _agree(torch.cat(logits), _want(name, tokens), dtype, name)
    assert rt.kv_cache.tokens == 140 and len(rt.kv_cache.pages) == 3 and rt.cache_stats()["graph_captures"] >= 1


@pytest.mark.parametrize("portion", [2, 3, 33, 64, 65])
@pytest.mark.parametrize("name", ["fast", "wide_latent", "odd"])
def test_portions_of_any_size_give_the_same_logits(name, portion, dtype):
    rt = _runtime(name, dtype)
    tokens = _tokens(name, 137, 2)
    parts = [rt.run_step_batch([rt], [tokens[i:i + portion]], [list(range(len(tokens[i:i + portion])))]) for i in range(0, 137, portion)]
    _agree(torch.cat(parts), _want(name, tokens), dtype)


def _replay(rt, name, dtype, rng, requests, *, live, step_rows):
    """Random mixed steps: up to `live` requests at a time, each step some of them, portions and single tokens mixed."""
    waiting, active, checked = list(requests), {}, 0
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
            scale = np.std(_want(name, chosen[0][0]))
            err = np.abs(logits.float().cpu().numpy() - np.stack(rows)).std(axis=1) / scale
            assert np.isfinite(err).all() and err.max() <= TOL[dtype], float(err.max())
            checked += len(rows)
        for a, b in zip(chosen, batches):
            a[1] += len(b)
            if a[1] == len(a[0]):
                a[2].kv_cache.clear()
                del active[id(a[0])]
    return checked


@pytest.mark.parametrize("name", ["fast", "wide_latent", "odd", "no_side"])
def test_mixed_steps_with_pages_and_slots_used_again(name, dtype):
    rng = np.random.default_rng(5)
    lengths = (190, 3, 64, 130, 65, 1, 128, 30, 70)
    requests = [_tokens(name, n, 20 + i) for i, n in enumerate(lengths)]
    rt = _runtime(name, dtype, pages=9, states=3)           # fewer pages and slots than the requests need in sum
    assert _replay(rt, name, dtype, rng, requests, live=3, step_rows=80) > 40
    stats = rt.kv_allocator.stats()
    assert stats["resident_pages"] == 0 and stats["allocated_pages_total"] > 9 and stats.get("states_in_use", 0) == 0
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


def test_segments_longer_than_one_recurrence_piece(dtype):
    name = "fast"
    tokens, short = _tokens(name, 700, 3), _tokens(name, 64, 21)
    rt = _runtime(name, dtype)
    a, b, c = rt.fork(), rt.fork(), rt.fork()
    b.run_step_batch([b], [short[:30]])
    logits = rt.run_step_batch([a, b, c], [tokens, short[30:31], short[:50]], [list(range(0, 700, 7)), [0], [49]])
    want = np.concatenate([_want(name, tokens)[::7], _want(name, short)[[30, 49]]])
    _agree(logits, want, dtype)
    _agree(rt.run_step_batch([b, c], [short[31:64], short[50:64]]), _want(name, short)[[63, 63]], dtype)


def test_the_batch_does_not_change_a_sequence(dtype):
    name = "wide_latent"
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

    rt = _runtime("fast", "bfloat16", pages=3, states=2)
    a, b, c = rt.fork(), rt.fork(), rt.fork()
    tokens = _tokens("fast", 200, 1)
    rt.run_step_batch([a], [tokens[:100]])
    with pytest.raises(KVPoolExhausted):
        rt.run_step_batch([a, b], [tokens[100:130], tokens[:65]])
    with pytest.raises(KVPoolExhausted):
        rt.run_step_batch([b, c], [[1], [2]])
    assert (a.kv_cache.tokens, b.kv_cache.tokens, b.kv_cache.state_slot) == (100, 0, None)
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
    rt = _runtime(name, dtype, pages=10, states=3)
    prompts = {f"r{n}": _tokens(name, n, 60 + n) for n in (90, 4, 65, 33)}
    alone = {k: _greedy_alone(rt, p, 12) for k, p in prompts.items()}
    if dtype == "float32":
        w = {k: a.astype(np.float64) for k, a in _weights(name).items()}
        p, ids = prompts["r33"], alone["r33"]
        logits = G.forward(CONFIGS[name], w, p + ids)[0]
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
        _agree(torch.from_numpy(np.fromfile(out / f"{i}.f32", "<f4").reshape(rows.shape)), rows, dtype, i)
    gen = subprocess.run([sys.executable, "-m", "cacheir_b200", "--model", str(folder), "--tokens", ",".join(map(str, b)), "--prompt", "hello",
                          "--max-new-tokens", "5", "--dtype", dtype], cwd=ROOT, capture_output=True, text=True)
    assert gen.returncode == 0, gen.stderr[-2000:]
    lines = [json.loads(x) for x in gen.stdout.splitlines()]
    assert [x["prompt_tokens"] for x in lines] == [5, 50] and all(len(x["tokens"]) == 5 for x in lines)
    if dtype == "float32":
        assert lines[1]["tokens"][0] == int(_want(name, b)[49].argmax())


def test_llama_shaped_models_take_mixed_steps_and_traces(tmp_path):
    from cacheir_b200 import B200DecodeRuntime, load_model
    from cacheir_b200.tiny import create_tiny_model
    from cacheir_b200.trace_run import TraceReplay

    folder = create_tiny_model(tmp_path / "tiny", seed=3)
    rt = B200DecodeRuntime(load_model(folder), dtype="float32")
    x, y = [int(t) for t in np.random.default_rng(0).integers(0, 64, 90)], [5, 9, 11]
    want_x, want_y = rt.fork().run([x])[0], rt.fork().run([y])[0]
    trace = TraceReplay(rt)
    first = trace.step([{"id": "x", "tokens": x[:80], "want": [0, 70, 79]}, {"id": "y", "tokens": y[:2], "want": [1]}], [])
    torch.testing.assert_close(first, torch.stack([want_x[0], want_x[70], want_x[79], want_y[1]]), rtol=1e-4, atol=1e-5)
    second = trace.step([{"id": "y", "tokens": y[2:], "want": [0]}, {"id": "x", "tokens": x[80:], "want": [9]}], ["x", "y"])
    torch.testing.assert_close(second, torch.stack([want_y[2], want_x[89]]), rtol=1e-4, atol=1e-5)


def test_prefix_reuse_is_refused_for_recurrent_layers_only():
    layers = [(latent(2, 16, 16, 16, 32, 500), 32), (latent(3, 16, 16, 16, 32, 20, kv_from=0), None)]
    CONFIGS["latent_only"] = config(64, 64, layers)
    try:
        rt = _runtime("latent_only", "float32")
        prompt = _tokens("latent_only", 140, 1)
        a, b = rt.fork(), rt.fork()
        a.prefill_tokens(prompt, use_prefix_cache=True, remember_prefix=True)
        logits, reused = b.prefill_tokens(prompt[:130] + [1, 2], use_prefix_cache=True)
        assert len(reused) == 128 and b.kv_cache.page_ids()[:2] == a.kv_cache.page_ids()[:2]
        _agree(logits[0, -1:], _want("latent_only", prompt[:130] + [1, 2])[-1:], "float32")
    finally:
        del CONFIGS["latent_only"]
    rt = _runtime("fast", "float32")
    prompt = _tokens("fast", 140, 1)
    rt.prefill_tokens(prompt, use_prefix_cache=True, remember_prefix=True)
    _, reused = rt.fork().prefill_tokens(prompt + [1], use_prefix_cache=True)
    assert reused == ()
