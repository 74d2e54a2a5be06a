"""Command line: python -m ironmill_b200 generate | trace.

  generate   greedy continuation of prompts of token ids with a model folder (a checkpoint or an `.ironml-gpu` bundle); the
             prompts run as sequences of one batch and one line of token ids is printed per prompt
  trace      replay of a trace of requests (trace.py)
"""
from __future__ import annotations

import argparse
import os
import sys


def generate(argv) -> int:
    ap = argparse.ArgumentParser(prog="python -m ironmill_b200 generate")
    ap.add_argument("--model", required=True)
    ap.add_argument("--tokens", required=True, action="append", help="prompt as token ids with commas between them; may be given several times")
    ap.add_argument("--max-new-tokens", type=int, default=16)
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"], help="list-of-layers models only")
    a = ap.parse_args(argv)
    prompts = [[int(t) for t in p.split(",")] for p in a.tokens]
    from . import _lib, build
    from .architectures import family_of
    from .bundle import CudaBundleProvider
    from .checkpoint import CheckpointProvider
    provider = (CudaBundleProvider if os.path.exists(os.path.join(a.model, "manifest.json")) else CheckpointProvider)(a.model)
    family = family_of(provider.config())
    _lib.use(build.ensure(family.library) if family.library else build.build())
    from .engine import CudaConfig, CudaInference
    engine = CudaInference(CudaConfig(max_seq_len=max(map(len, prompts)) + a.max_new_tokens, max_batch=len(prompts), dtype=a.dtype))
    engine.load_weights(provider)
    for row in engine.generate(prompts, a.max_new_tokens):
        print(",".join(map(str, row)))
    engine.close()
    return 0


def main(argv=None) -> int:
    argv = list(sys.argv[1:] if argv is None else argv)
    if argv[:1] == ["generate"]:
        return generate(argv[1:])
    if argv[:1] == ["trace"]:
        from .trace import main as trace_main
        return trace_main(argv[1:])
    print(__doc__.strip(), file=sys.stderr)
    return 2


if __name__ == "__main__":
    sys.exit(main())
