"""Trace replay: steps of given token ids through an engine's step function, logits to files (the program behind ``bin/trace_run``)."""
from __future__ import annotations

import argparse
import json
import sys
from pathlib import Path
from typing import IO, Iterable

import torch

DTYPES = {"bfloat16": torch.bfloat16, "float32": torch.float32}


def replay(engine, lines: Iterable[str], out_dir, report: IO[str]) -> int:
    """Runs every step of ``lines`` and returns their number."""
    from .serving import StepEntry
    out, n = Path(out_dir), 0
    for line in lines:
        if not line.strip():
            continue
        s = json.loads(line)
        logits = engine.step([StepEntry(e["id"], e["tokens"], e.get("want", ())) for e in s.get("entries", ())], s.get("end", ()))
        if logits is not None:
            (out / f"{s['step']}.f32").write_bytes(logits.float().contiguous().cpu().numpy().astype("<f4").tobytes())
        report.write(f"done {s['step']}\n")
        report.flush()
        n += 1
    if hasattr(engine, "check"):
        engine.check()
    return n


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay token steps through a model and write logits.")
    ap.add_argument("--model", required=True, help="directory with config.json and model.safetensors")
    ap.add_argument("--dtype", choices=sorted(DTYPES), default="bfloat16")
    ap.add_argument("--out", required=True, help="directory for <step>.f32")
    ap.add_argument("--max-tokens", type=int, default=4096, help="most tokens that live sequences hold together")
    ap.add_argument("--device", default="cuda")
    a = ap.parse_args(argv)
    from .registry import load_engine
    torch.backends.cuda.matmul.allow_tf32 = False
    replay(load_engine(a.model, a.device, DTYPES[a.dtype], a.max_tokens), sys.stdin, a.out, sys.stdout)
    return 0


if __name__ == "__main__":
    sys.exit(main())
