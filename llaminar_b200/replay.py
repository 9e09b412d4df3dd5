"""Replay of recorded token ids through the engine, step by step, with logits written to files.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps

Each line of standard input is a step: {"step": n, "entries": [{"id", "tokens", "want"}], "end": [ids]}.  The entries run as
one batch through `LLMEngine.feed`; for the places in "want" the logits go to `<out>/<step>.f32` (little-endian float32,
[wanted, vocab], in the order of the entries), and `done <step>` follows on standard output.  Requests named in "end" give
their cache pages back.  Exit code 3: the model has no 32-bit mode.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

import torch

PAGE = 64
LIVE_REQUESTS = 4


def build_engine(model: str, dtype: torch.dtype, max_tokens: int, device: str):
    from .engine.engine import LLMEngine
    from .models.weights import ModelWeights
    weights = ModelWeights.from_path(model, device="cpu")
    if dtype == torch.float32 and device != "cpu" and not weights.config.has_mixers:
        return None
    pages = -(-max_tokens // PAGE)
    return LLMEngine(weights, device=device, max_batch=LIVE_REQUESTS, max_context=pages * PAGE, kv_pages=pages + 1,      # + the scratch page
                     max_prefill_tokens=pages * PAGE, dtype=dtype)


def run(engine, lines, out_dir: str, report) -> None:
    live: dict = {}
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        entries = []
        for e in step["entries"]:
            if e["id"] not in live:
                live[e["id"]] = engine.open_sequence()
            entries.append((live[e["id"]], e["tokens"], e["want"]))
        logits = engine.feed(entries) if entries else None
        if logits is not None:
            data = logits.float().cpu().contiguous().numpy().astype("<f4", copy=False).tobytes()
            with open(os.path.join(out_dir, f"{step['step']}.f32"), "wb") as f:
                f.write(data)
        for name in step.get("end", ()):
            engine.close_sequence(live.pop(name))
        report(step["step"])


def main(argv: list[str] | None = None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.split("\n")[0])
    ap.add_argument("--model", required=True, help="checkpoint directory (config.json and safetensors) or .gguf file")
    ap.add_argument("--dtype", choices=("bfloat16", "float32"), default="bfloat16")
    ap.add_argument("--out", required=True, help="existing directory for the logits")
    ap.add_argument("--max-tokens", type=int, required=True, help="tokens the cache pool holds, over all live requests")
    ap.add_argument("--device", default="cuda:0", help="cuda:N, or cpu for the PyTorch back end")
    a = ap.parse_args(argv)
    engine = build_engine(a.model, getattr(torch, a.dtype), a.max_tokens, a.device)
    if engine is None:
        print("this model has no 32-bit mode on the GPU", file=sys.stderr)
        return 3

    def report(n) -> None:
        sys.stdout.write(f"done {n}\n")
        sys.stdout.flush()

    run(engine, sys.stdin, a.out, report)
    return 0


if __name__ == "__main__":
    raise SystemExit(main())
