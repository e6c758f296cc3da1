"""Replays a trace of steps through an engine and writes the logits it asks for.

Standard input has one JSON object a line: {"step": n, "entries": [{"id", "tokens", "want"}], "end": [ids]}.
Logits at the wanted places go to <out>/<step>.f32 (little-endian, [wanted, vocab]) and a line
"done <step>" follows.  Nothing is sampled.
"""
from __future__ import annotations

import json
import os
import sys

import torch


def replay(engine, lines, out_dir: str, report) -> None:
    live = {}
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        rows = []
        for entry in step["entries"]:
            if entry["id"] not in live:
                live[entry["id"]] = engine.open()
            logits = engine.step(live[entry["id"]], entry["tokens"], entry["want"])
            if logits is not None:
                rows.append(logits.to("cpu", torch.float32).contiguous())
        if rows:
            data = torch.cat(rows).numpy().astype("<f4").tobytes()
            part = os.path.join(out_dir, f".{step['step']}.part")
            with open(part, "wb") as f:
                f.write(data)
            os.replace(part, os.path.join(out_dir, f"{step['step']}.f32"))
        for ident in step.get("end", ()):
            if ident in live:
                engine.close(live.pop(ident))
        report(f"done {step['step']}")


def main(args) -> int:
    from . import registry
    dtype = {"bfloat16": torch.bfloat16, "float32": torch.float32}[args.dtype]
    engine = registry.load(args.model, dtype=dtype, max_tokens=args.max_tokens)

    def report(text):
        sys.stdout.write(text + "\n")
        sys.stdout.flush()

    replay(engine, iter(sys.stdin.readline, ""), args.out, report)
    return 0
