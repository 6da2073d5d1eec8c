"""Replays a trace of token ids through a model, step by step, and writes logits: ``bin/trace_run``.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps.jsonl

A step is one JSON object a line: ``{"step": 0, "entries": [{"id": "a", "tokens": [5, 17], "want": [0, 1]}], "end": []}``.
All entries of a step run as one batch of the engine, portions of prompts beside decoded tokens; a request is admitted at
its first entry, and the requests under ``end`` give back their cache pages and state slot after the step.  The logits at
the wanted places go to ``<out>/<step>.f32`` (little-endian FP32, [wanted, vocab], in the order of the entries), and
``done <step>`` is printed after every step.

``--max-tokens`` is what live requests hold at most, each rounded up to a multiple of 64; the cache pool is made for that
many tokens, and there are ``--max-seqs`` sequence slots.
"""
from __future__ import annotations

import argparse
import json
import os
import sys


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="replay a trace of token ids and write logits")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="existing folder for <step>.f32")
    ap.add_argument("--max-tokens", type=int, required=True)
    ap.add_argument("--max-seqs", type=int, default=4)
    args = ap.parse_args(argv)

    from .. import _build
    _build.ensure_serving()
    import numpy as np

    from ..infer import Chunk, EngineConfig, open_engine
    from ..ops import _cuda as K

    engine = open_engine(args.model, EngineConfig(precision="bf16" if args.dtype == "bfloat16" else "fp32",
                                                  max_seqs=args.max_seqs, max_tokens=args.max_tokens,
                                                  kv_tokens=args.max_tokens))
    vocab = engine.vocab()
    seqs = {}
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        chunks = []
        for e in step["entries"]:
            if e["id"] not in seqs:
                seqs[e["id"]] = engine.add_sequence()
            chunks.append(Chunk(seqs[e["id"]], e["tokens"], places=e["want"]))
        if any(len(c.tokens) for c in chunks):
            logits = engine.forward(chunks)
            if logits.shape[0]:
                data = logits[:, :vocab].float().cpu().numpy().astype("<f4", copy=False)
                K.check_status()
                path = os.path.join(args.out, f"{step['step']}.f32")
                with open(path + ".part", "wb") as f:
                    f.write(np.ascontiguousarray(data).tobytes())
                os.replace(path + ".part", path)
        for name in step["end"]:
            if name in seqs:
                engine.free_sequence(seqs.pop(name))
        print("done", step["step"], flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
