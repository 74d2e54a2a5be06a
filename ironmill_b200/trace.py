"""Replays a trace of requests: token ids come in steps on standard input, logits go to files.

A step is one JSON line {"step": n, "entries": [{"id", "tokens", "want"}], "end": [ids]}: every entry appends its tokens to
that request's sequence; `want` names the places among them whose logits are written to <out>/<n>.f32 (f32, one row per
place, entries in order); `end` lists the requests that give their cache slot back.  "done <n>" is printed after each step.
The tokens go through the engine's sequence interface: a cache slot per request, prompt portions through the chunked
prefill, single tokens through the captured decode step.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

import numpy as np


def replay(engine, lines, out_dir: str, report) -> None:
    seqs: dict = {}
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        rows = []
        for e in step["entries"]:
            if e["id"] not in seqs:
                seqs[e["id"]] = engine.open_sequence()
            want = [int(w) for w in e.get("want", ())]
            places = sorted(set(want))
            got = engine.extend_sequence(seqs[e["id"]], e["tokens"], places)
            rows += [got[places.index(w)] for w in want]
        if rows:
            path = os.path.join(out_dir, f"{step['step']}.f32")
            with open(path + ".part", "wb") as fh:
                fh.write(np.stack(rows).astype("<f4").tobytes())
            os.replace(path + ".part", path)
        for rid in step.get("end", ()):
            if rid in seqs:
                engine.remove_sequence(seqs.pop(rid))
        report(f"done {step['step']}")


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay a trace of requests and write logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and *.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, default=0, help="most tokens that live requests hold at any time")
    ap.add_argument("--max-requests", type=int, default=4, help="most requests alive at any time")
    a = ap.parse_args(argv)
    from . import _lib, build
    from .architectures import family_of
    from .checkpoint import CheckpointProvider
    provider = CheckpointProvider(a.model)
    family = family_of(provider.config())
    _lib.use(build.ensure(family.library) if family.library else build.build())
    from .engine import CudaConfig, CudaInference
    engine = CudaInference(CudaConfig(max_seq_len=max(1, a.max_tokens or 4096), max_batch=max(1, min(64, a.max_requests)), dtype=a.dtype))
    engine.load_weights(provider)

    def report(text):
        print(text, flush=True)

    replay(engine, sys.stdin, a.out, report)
    engine.close()
    return 0


if __name__ == "__main__":
    sys.exit(main())
