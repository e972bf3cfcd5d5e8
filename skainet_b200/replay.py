"""Replays a trace of token steps through a model and writes the logits it asks for (bin/trace_run).

Steps come as JSON lines on standard input: {"step": n, "entries": [{"id", "tokens", "want"}], "end": [ids]}.  A
request takes a slot of the decoder with its first entry and gives it back when it ends; the logits of a step's wanted
places go to <out>/<step>.f32 ([wanted, vocab], little-endian fp32), and `done <step>` is printed after every step."""
from __future__ import annotations

import argparse
import json
import os
import sys

import numpy as np


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.split("\n")[0])
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    ap.add_argument("--max-seqs", type=int, default=4, help="most requests alive at a time")
    ap.add_argument("--device", type=int, default=0)
    a = ap.parse_args(argv)
    from . import _ffi, build, registry
    _ffi.use(build.build_family(registry.architecture_of(registry.read_config(a.model)).family))
    from .tensor import Context
    ctx = Context(a.device)
    model = registry.load_model(ctx, a.model, max_seqs=a.max_seqs, max_tokens=max(1, min(a.max_tokens, 2048), a.max_seqs),
                                max_ctx=max(1, a.max_tokens), dtype=a.dtype)
    slots: dict = {}
    free = list(range(a.max_seqs))
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        rows = []
        for e in step["entries"]:
            if e["id"] not in slots:
                if not free:
                    raise RuntimeError(f"more than {a.max_seqs} live requests")
                slots[e["id"]] = free.pop(0)
                model.reset(slots[e["id"]])
            _, logits = model.forward(e["tokens"], seq=slots[e["id"]], want=e["want"], want_next=False)
            if logits is not None:
                rows.append(logits)
        if rows:
            np.concatenate(rows).astype("<f4").tofile(os.path.join(a.out, f"{step['step']}.f32"))
        for r in step.get("end", []):
            if r in slots:
                model.reset(slots[r])
                free.append(slots.pop(r))
        print(f"done {step['step']}", flush=True)
    model.close()
    ctx.close()
    return 0


if __name__ == "__main__":
    sys.exit(main())
