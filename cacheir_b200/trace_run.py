"""Replay a trace: token ids go through a model step by step, wanted logits go to files. Nothing is sampled.

Steps come from standard input, one JSON object a line:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

All entries of a step run as one batch through `B200DecodeRuntime.run_step_batch`: a request's first entry admits it, its
next tokens continue from its cache and state, "end" gives back what it holds. For a step with wanted places,
OUT/<step>.f32 receives their logits in order as little-endian float32; "done <step>" follows on standard output.
"""
from __future__ import annotations

import argparse
import json
import sys
from pathlib import Path
from typing import Any, TextIO


class TraceReplay:
    """The requests of a trace as sessions of one runtime."""

    def __init__(self, runtime: Any):
        self.template = runtime
        self.sessions: dict[str, Any] = {}

    def step(self, entries: list[dict], end: list[str]) -> Any | None:
        """Run one step; returns the wanted logits [n, vocab] or None when nothing is wanted."""
        names = [str(e["id"]) for e in entries]
        if len(set(names)) != len(names):
            raise ValueError("a request may appear only once in a step")
        logits = None
        if entries:
            for name in names:
                if name not in self.sessions:
                    self.sessions[name] = self.template.fork()
            wanted = [[int(p) for p in e.get("want", [])] for e in entries]
            logits = self.template.run_step_batch([self.sessions[n] for n in names], [[int(t) for t in e["tokens"]] for e in entries], wanted)
            if not any(wanted):
                logits = None
        for name in end:
            self.sessions.pop(str(name)).kv_cache.clear()
        return logits


def replay(runtime: Any, lines: TextIO, out_dir: Path, done: TextIO) -> None:
    trace = TraceReplay(runtime)
    for line in lines:
        if not line.strip():
            continue
        item = json.loads(line)
        logits = trace.step(item.get("entries", []), item.get("end", []))
        if logits is not None:
            (out_dir / f"{item['step']}.f32").write_bytes(logits.float().contiguous().cpu().numpy().astype("<f4").tobytes())
        else:
            runtime.synchronize()
        runtime.check_device_status()
        print(f"done {item['step']}", file=done, flush=True)


def main(argv: list[str] | None = None) -> int:
    parser = argparse.ArgumentParser(prog="trace_run", description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    parser.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    parser.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    parser.add_argument("--out", required=True, help="folder for the logits")
    parser.add_argument("--max-tokens", type=int, required=True, help="tokens that live requests hold at most, in whole pages")
    parser.add_argument("--max-requests", type=int, default=4, help="requests alive at any time (recurrent state slots)")
    args = parser.parse_args(argv)

    from . import build, models
    folder = Path(args.model)
    config = json.loads((folder / "config.json").read_text(encoding="utf-8"))
    build.build(groups=models.family_for(config).kernel_groups)

    from .kv_cache import B200KVPageAllocator
    from .runtime import B200DecodeRuntime
    artifact = models.load_model(folder)
    page = int(artifact.graph("decode").attrs["execution_hints"]["page_size"])
    pages = max(1, (args.max_tokens + page - 1) // page)
    allocator = B200KVPageAllocator(page_size=page, initial_slots=pages, max_slots=pages, initial_states=args.max_requests,
                                    max_states=args.max_requests)
    runtime = B200DecodeRuntime(artifact, dtype=args.dtype, kv_allocator=allocator, max_seq_len=pages * page)
    out = Path(args.out)
    out.mkdir(parents=True, exist_ok=True)
    replay(runtime, sys.stdin, out, sys.stdout)
    return 0


if __name__ == "__main__":
    sys.exit(main())
