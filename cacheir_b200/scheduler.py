"""Batched-decode launch: the part of the reference's continuous-batching
scheduler that drives the decode hot path.

`BatchedDecodeLauncher` keeps what `ContinuousBatchScheduler._decode_batch`
and its run loop do for decode (cacheir/runtime/scheduler.py:160-208, 456-478,
535-543): fork one session per request, prefill it, then advance every active
request one token per round through `run_decode_batch`, take the row argmax,
`% vocab_size`, and retire requests that reached their token budget. Admission
policy (priorities, aging, preemption, back-pressure) is host policy outside the
hot path and is not reproduced; the reference's own scheduler can drive
`B200DecodeRuntime` directly since it only needs the runtime duck type.

With `step_tokens` the launcher runs mixed rounds instead: every round is one `run_step_batch` that carries the next
token of each decoding request and portions of waiting prompts up to that many rows, so a long prompt does not hold
back the requests that are already decoding. A request is admitted when the pool has pages (and a state slot) for its
prompt and its whole budget.
"""
from __future__ import annotations

import time
from dataclasses import dataclass, field
from typing import Any


@dataclass
class DecodeMetrics:
    """The decode counters of `SchedulerMetrics` (scheduler.py:36-72)."""

    completed_requests: int = 0
    generated_tokens: int = 0
    prefill_tokens: int = 0
    batched_decode_rounds: int = 0
    batched_decode_tokens: int = 0
    total_decode_batch_ms: float = 0.0
    total_decode_ms: float = 0.0
    total_prefill_ms: float = 0.0


@dataclass
class _Active:
    request_id: str
    runtime: Any
    prompt_ids: list[int]
    max_new_tokens: int
    next_id: int
    generated_ids: list[int] = field(default_factory=list)
    prefilled: int = 0          # prompt tokens already run (mixed rounds)


def argmax_tokens(logits: Any) -> list[int]:
    """`_argmax_tokens` (scheduler.py:535-543): row argmax of the last position, read back to
    the host. CUDA logits go through the library's argmax kernel; only the ids cross PCIe."""
    last = logits[:, -1]
    if getattr(last, "is_cuda", False):
        from . import ops
        return [int(v) for v in ops.argmax_rows(last.contiguous()).tolist()]
    return [int(v) for v in last.argmax(dim=-1).tolist()]


class BatchedDecodeLauncher:
    def __init__(self, template: Any, *, max_batch_size: int = 4, step_tokens: int | None = None):
        self.template = template
        self.max_batch_size = max(1, int(max_batch_size))
        self.step_tokens = None if step_tokens is None else max(self.max_batch_size, int(step_tokens))
        self.metrics = DecodeMetrics()
        self._pending: list[tuple[str, list[int], int]] = []
        self._counter = 0

    def submit(self, prompt_ids: list[int], *, max_new_tokens: int = 16, request_id: str | None = None) -> str:
        self._counter += 1
        rid = request_id or f"req-{self._counter}"
        self._pending.append((rid, [int(t) for t in prompt_ids], int(max_new_tokens)))
        return rid

    def _prefill(self, rid: str, prompt_ids: list[int], max_new_tokens: int) -> _Active:
        runtime = self.template.fork()
        start = time.perf_counter()
        logits, _ = runtime.prefill_tokens(prompt_ids)
        runtime.synchronize()
        self.metrics.total_prefill_ms += (time.perf_counter() - start) * 1000.0
        self.metrics.prefill_tokens += len(prompt_ids)
        vocab = int(runtime.artifact.config.vocab_size)
        next_id = int(logits[0, -1].argmax().item()) % vocab
        return _Active(rid, runtime, prompt_ids, max_new_tokens, next_id)

    def _decode_batch(self, states: list[_Active]) -> None:
        runtime = states[0].runtime
        sessions = [s.runtime for s in states]
        token_ids = [s.next_id for s in states]
        start = time.perf_counter()
        logits = runtime.run_decode_batch(sessions, token_ids)
        runtime.synchronize()
        elapsed_ms = (time.perf_counter() - start) * 1000.0
        next_ids = argmax_tokens(logits)
        self.metrics.batched_decode_rounds += 1
        self.metrics.batched_decode_tokens += len(states)
        self.metrics.total_decode_batch_ms += elapsed_ms
        self.metrics.total_decode_ms += elapsed_ms * len(states)
        vocab = int(runtime.artifact.config.vocab_size)
        for state, next_id in zip(states, next_ids):
            state.generated_ids.append(state.next_id)
            self.metrics.generated_tokens += 1
            state.next_id = int(next_id) % vocab

    # -- mixed rounds --------------------------------------------------------------------
    def _room_for(self, prompt_ids: list[int], max_new_tokens: int, active: list[_Active]) -> bool:
        """Pages and a state slot for a request's whole life, counting what the active ones may still open."""
        alloc = self.template.kv_allocator
        page = alloc.page_size

        def pages(tokens: int) -> int:
            return (tokens + page - 1) // page

        free = alloc.free_slots()
        if free is not None:
            promised = sum(pages(len(s.prompt_ids) + s.max_new_tokens) - len(s.runtime.kv_cache.pages) for s in active)
            if pages(len(prompt_ids) + max_new_tokens) > free - promised:
                return False
        free = alloc.free_states() if alloc.has_state else None
        return free is None or free - sum(s.runtime.kv_cache.state_slot is None for s in active) > 0

    def _mixed_round(self, active: list[_Active]) -> None:
        decoding = [s for s in active if s.prefilled == len(s.prompt_ids)]
        room = self.step_tokens - len(decoding)
        states, batches = list(decoding), [[s.next_id] for s in decoding]
        for s in active:
            n = min(room, len(s.prompt_ids) - s.prefilled)
            if n > 0:
                states.append(s)
                batches.append(s.prompt_ids[s.prefilled:s.prefilled + n])
                room -= n
        # a portion that does not reach the prompt's end needs no logits
        wanted = [[len(b) - 1] if s.prefilled + len(b) >= len(s.prompt_ids) else [] for s, b in zip(states, batches)]
        start = time.perf_counter()
        logits = states[0].runtime.run_step_batch([s.runtime for s in states], batches, wanted)
        states[0].runtime.synchronize()
        elapsed_ms = (time.perf_counter() - start) * 1000.0
        next_ids = iter(argmax_tokens(logits.unsqueeze(1)) if any(wanted) else [])
        vocab = int(self.template.artifact.config.vocab_size)
        for s, batch, want in zip(states, batches, wanted):
            if s.prefilled < len(s.prompt_ids):
                s.prefilled += len(batch)
                self.metrics.prefill_tokens += len(batch)
            else:
                s.generated_ids.append(s.next_id)
                self.metrics.generated_tokens += 1
            if want:
                s.next_id = int(next(next_ids)) % vocab
        if decoding:
            self.metrics.batched_decode_rounds += 1
            self.metrics.batched_decode_tokens += len(decoding)
            self.metrics.total_decode_batch_ms += elapsed_ms
            self.metrics.total_decode_ms += elapsed_ms * len(decoding)
        else:
            self.metrics.total_prefill_ms += elapsed_ms

    def _run_mixed(self) -> dict[str, list[int]]:
        results: dict[str, list[int]] = {}
        active: list[_Active] = []
        while self._pending or active:
            while self._pending and len(active) < self.max_batch_size:
                rid, prompt_ids, max_new = self._pending[0]
                if not self._room_for(prompt_ids, max_new, active):
                    if not active:
                        raise RuntimeError(f"request {rid!r} needs more cache than the pool has")
                    break
                self._pending.pop(0)
                active.append(_Active(rid, self.template.fork(), prompt_ids, max_new, -1))
            self._mixed_round(active)
            still = []
            for s in active:
                if s.prefilled == len(s.prompt_ids) and len(s.generated_ids) >= s.max_new_tokens:
                    results[s.request_id] = s.generated_ids
                    s.runtime.kv_cache.clear()
                    self.metrics.completed_requests += 1
                else:
                    still.append(s)
            active = still
        return results

    def run_until_complete(self) -> dict[str, list[int]]:
        if self.step_tokens is not None:
            return self._run_mixed()
        results: dict[str, list[int]] = {}
        active: list[_Active] = []
        while self._pending or active:
            while self._pending and len(active) < self.max_batch_size:
                active.append(self._prefill(*self._pending.pop(0)))
            ready = [s for s in active if len(s.generated_ids) < s.max_new_tokens]
            if ready:
                self._decode_batch(ready)
            still = []
            for s in active:
                if len(s.generated_ids) >= s.max_new_tokens:
                    results[s.request_id] = s.generated_ids
                    s.runtime.kv_cache.clear()
                    self.metrics.completed_requests += 1
                else:
                    still.append(s)
            active = still
        return results
