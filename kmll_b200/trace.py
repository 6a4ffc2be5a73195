"""Replays a trace: reads steps (JSON lines) from standard input, feeds their tokens to a model through the session layer and
writes the logits of the wanted places.

  {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

After a step whose entries want logits, OUT/<step>.f32 holds them as little-endian float32 [wanted, vocab]; then "done <step>"
goes to standard output.  The decoder holds one sequence: a request ends before the next begins."""
from __future__ import annotations

import argparse
import json
import os
import sys

import numpy as np

from . import build


def replay(session, lines, out_dir: str, stdout) -> None:
    current = None  # id of the request whose tokens the decoder holds
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        logits = []
        for entry in step.get("entries", []):
            if entry["id"] != current:
                if current is not None:
                    raise ValueError(f"step {step['step']}: request {entry['id']!r} begins before {current!r} has ended")
                session.reset_sequence()
                current = entry["id"]
            want = [int(w) for w in entry.get("want", [])]
            order = sorted(set(want))
            rows = session.extend(entry["tokens"], order)
            if want:
                logits.append(rows[[order.index(w) for w in want]])
        if current in step.get("end", []):
            session.reset_sequence()
            current = None
        if logits:
            data = np.ascontiguousarray(np.concatenate(logits), dtype="<f4").tobytes()
            with open(os.path.join(out_dir, f"{step['step']}.f32"), "wb") as f:
                f.write(data)
        print(f"done {step['step']}", file=stdout, flush=True)


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, default=0, help="the most tokens a request holds (0: as many as the model has positions)")
    a = ap.parse_args(argv)
    build.build()  # compiles the library at the first call
    from .registry import load_model
    from .session import Session
    os.makedirs(a.out, exist_ok=True)
    session = Session(load_model(a.model, a.dtype, a.max_tokens or None))
    replay(session, sys.stdin, a.out, sys.stdout)
    return 0


if __name__ == "__main__":
    sys.exit(main())
