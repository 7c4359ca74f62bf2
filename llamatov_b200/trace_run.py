"""Replay a trace of token portions through a model and write the logits it asks for (bin/trace_run).

  trace_run --model DIR --dtype bfloat16|float32 --out DIR [--max-tokens N]

Steps come from standard input, one JSON object a line:
  {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}
Each entry's tokens continue its sequence; `want` are the places among them whose logits go to DIR/<step>.f32 (fp32,
little endian, in order); sequences in `end` are finished after the step.  "done <step>" follows every step.
"""
import argparse
import json
import os
import sys


def main(argv=None):
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay token portions through a model and write logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for the <step>.f32 files")
    ap.add_argument("--max-tokens", type=int, default=None, help="most tokens live sequences hold at any time")
    a = ap.parse_args(argv)

    from . import build
    build.build(groups=("dense",))
    import numpy as np
    from . import _lib, llamatov_run
    from .sequences import Sequences
    cfg, w = llamatov_run.load_model(a.model, dtype=a.dtype)
    seqs = Sequences(w, cfg, a.max_tokens)
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        rows = []
        for e in step["entries"]:
            lg = seqs.step(e["id"], e["tokens"], e.get("want", ()))
            if lg is not None:
                rows.append(lg.numpy())
        for sid in step.get("end", ()):
            seqs.end(sid)
        status = _lib.device_status()
        if status:
            raise RuntimeError(f"device status after step {step['step']}: {', '.join(sorted(status))}")
        if rows:
            path = os.path.join(a.out, f"{step['step']}.f32")
            np.concatenate(rows).astype("<f4").tofile(path)
        print(f"done {step['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
