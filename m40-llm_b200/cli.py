"""Command line of the framework: bin/generate and bin/trace_run call generate_main and trace_main."""
from __future__ import annotations

import argparse
import json
import os
import sys

import numpy as np


def _open(model_dir: str, dtype: str, sequences: int, max_len: int):
    from . import build, models, native
    build.build()
    nat = native.Native(native.lib())
    return nat, models.load(nat, model_dir, dtype=dtype, sequences=sequences, max_len=max_len)


def generate_main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="generate", description="Greedy generation from token ids.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    ap.add_argument("--max-new", type=int, default=32)
    ap.add_argument("--stop", type=int, help="token id that ends a request")
    ap.add_argument("--sequences", type=int, default=8, help="requests that run at the same time")
    ap.add_argument("--max-len", type=int, default=4096, help="longest sequence, prompt and output together")
    ap.add_argument("--portion", type=int, default=512, help="prompt tokens per step")
    ap.add_argument("prompt", nargs="+", help="one prompt each: comma-separated token ids")
    a = ap.parse_args(argv)
    from .engine import Engine
    _, model = _open(a.model, a.dtype, a.sequences, a.max_len)
    engine = Engine(model, portion=a.portion)
    ids = [engine.submit([int(t) for t in p.split(",")], a.max_new, a.stop) for p in a.prompt]
    out = engine.run()
    for i in ids:
        print(json.dumps(out[i]))
    model.close()
    return 0


def trace_main(argv=None) -> int:
    ap = argparse.ArgumentParser(
        prog="trace_run",
        description="Feeds given token ids through a model step by step and writes logits. Reads one JSON object a line from "
                    "standard input: {step, entries: [{id, tokens, want}], end: [id]}; writes OUT/<step>.f32 for the wanted "
                    "places and prints 'done <step>'.")
    ap.add_argument("--model", required=True)
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    ap.add_argument("--out", required=True)
    ap.add_argument("--max-tokens", type=int, default=4096, help="most tokens that live requests hold at any time")
    a = ap.parse_args(argv)
    nat, model = _open(a.model, a.dtype, 4, max(a.max_tokens, 1))
    slots: dict[str, int] = {}
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        entries, want, order, at = [], [], [], 0
        for e in step["entries"]:
            if e["id"] not in slots:
                slots[e["id"]] = model.acquire()
            entries.append((slots[e["id"]], e["tokens"]))
            order += [at + int(k) for k in e["want"]]
            at += len(e["tokens"])
        if entries:
            want = sorted(set(order))
            logits = model.step(entries, want)["logits"]
            if order:
                rows = logits[[want.index(k) for k in order]]
                with open(os.path.join(a.out, f"{step['step']}.f32"), "wb") as f:
                    f.write(np.ascontiguousarray(rows, "<f4").tobytes())
        for i in step.get("end", []):
            if i in slots:
                model.release(slots.pop(i))
        print(f"done {step['step']}", flush=True)
    model.close()
    nat.free_all()
    return 0
