"""Trace replay: given token ids go through a model's engine step by step and the
logits at the places asked for are written out (bin/trace_run).  The model, its
slots, caches and steps are the ones generation uses; nothing is sampled."""
from __future__ import annotations

import argparse
import json
import sys
from pathlib import Path
from typing import Dict, Iterable, Optional, TextIO

import numpy as np


def replay(engine, lines: Iterable[str], out_dir: Path, done: TextIO) -> None:
    """Every line is one step: {"step", "entries": [{"id", "tokens", "want"}], "end": [ids]}."""
    slots: Dict[str, int] = {}
    for line in lines:
        if not line.strip():
            continue
        st = json.loads(line)
        parts = []
        for e in st["entries"]:
            if e["id"] not in slots:
                slots[e["id"]] = engine.states.acquire()
            lg = engine.forward_tokens(e["tokens"], slots[e["id"]], e["want"])
            if len(e["want"]):
                parts.append(lg.float().cpu().numpy())
        engine.check_status()
        for i in st.get("end", []):
            if i in slots:
                engine.states.release(slots.pop(i))
        if parts:
            np.ascontiguousarray(np.concatenate(parts), dtype="<f4").tofile(out_dir / f"{st['step']}.f32")
        print(f"done {st['step']}", file=done, flush=True)


def main(argv: Optional[list] = None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay a trace of token ids and write logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and safetensors")
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for <step>.f32")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens held by live sequences at any time")
    ap.add_argument("--max-sequences", type=int, default=4, help="most sequences alive at any time")
    a = ap.parse_args(argv)
    from ..models.registry import architecture_of, build_engine
    if a.dtype not in architecture_of(a.model).dtypes:
        print(f"this model does not run in {a.dtype}", file=sys.stderr)
        return 3
    engine, _ = build_engine(a.model, max_seq_len=max(16, a.max_tokens), max_batch=a.max_sequences, dtype=a.dtype)
    replay(engine, sys.stdin, Path(a.out), sys.stdout)
    return 0
