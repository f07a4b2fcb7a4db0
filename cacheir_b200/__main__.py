"""Command line: greedy generation from a model folder.

    python -m cacheir_b200 --model DIR --prompt "text" [--prompt ...] --max-new-tokens 32
    python -m cacheir_b200 --model DIR --tokens 5,17,3 --dtype float32

The architecture in DIR/config.json picks the model family; prompts run together under `BatchedDecodeLauncher`.
"""
from __future__ import annotations

import argparse
import json
import sys


def main(argv: list[str] | None = None) -> int:
    parser = argparse.ArgumentParser(prog="cacheir_b200", description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    parser.add_argument("--model", required=True, help="folder with config.json and model.safetensors or weights.npz")
    parser.add_argument("--prompt", action="append", default=[], help="text prompt (byte tokenizer); may be repeated")
    parser.add_argument("--tokens", action="append", default=[], help="prompt as comma-separated token ids; may be repeated")
    parser.add_argument("--max-new-tokens", type=int, default=16)
    parser.add_argument("--dtype", default="auto", choices=["auto", "float32", "float16", "bfloat16"])
    parser.add_argument("--quant", default=None, help="weight format of Llama-shaped models (int8, int4_awq)")
    parser.add_argument("--max-batch-size", type=int, default=8)
    parser.add_argument("--step-tokens", type=int, default=512, help="rows of a mixed round (prompt portions beside decoded tokens)")
    parser.add_argument("--max-seq-len", type=int, default=None)
    args = parser.parse_args(argv)

    from . import build, models
    from .scheduler import BatchedDecodeLauncher
    artifact = models.load_model(args.model, quant=args.quant)
    build.build(groups=models.family_for({"architecture": artifact.config.architecture}).kernel_groups)
    from .runtime import B200DecodeRuntime
    runtime = B200DecodeRuntime(artifact, dtype=args.dtype, max_seq_len=args.max_seq_len)
    prompts = [runtime.tokenizer.encode(text) for text in args.prompt] + [[int(t) for t in ids.split(",")] for ids in args.tokens]
    if not prompts:
        parser.error("give at least one --prompt or --tokens")
    launcher = BatchedDecodeLauncher(runtime, max_batch_size=args.max_batch_size, step_tokens=args.step_tokens)
    names = [launcher.submit(ids, max_new_tokens=args.max_new_tokens) for ids in prompts]
    results = launcher.run_until_complete()
    for name, ids in zip(names, prompts):
        print(json.dumps({"id": name, "prompt_tokens": len(ids), "tokens": results[name], "text": runtime.tokenizer.decode(results[name])}))
    return 0


if __name__ == "__main__":
    sys.exit(main())
