"""Generates from a model on disk: token ids in, token ids out, all prompts served together.

    python -m nexus_b200.tools.generate --model DIR --prompt 5,17,3 --prompt 12,9 --max-new 32
        [--precision bf16|fp32] [--temperature 0.8 --top-k 50 --top-p 0.95 --seed 7] [--stop ID]

The model is a folder with ``config.json`` (its ``architecture`` picks the family) or a GPT-2 archive; one JSON line per
prompt, in the order given."""
from __future__ import annotations

import argparse
import json
import sys


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="generate", description=__doc__.splitlines()[0])
    ap.add_argument("--model", required=True)
    ap.add_argument("--prompt", action="append", required=True, help="comma-separated token ids; repeat for more requests")
    ap.add_argument("--max-new", type=int, default=32)
    ap.add_argument("--precision", default="bf16", choices=["bf16", "fp32"])
    ap.add_argument("--temperature", type=float, default=0.0)
    ap.add_argument("--top-k", type=int, default=0)
    ap.add_argument("--top-p", type=float, default=1.0)
    ap.add_argument("--seed", type=int, default=0)
    ap.add_argument("--stop", type=int, default=None, help="token id that ends a request")
    ap.add_argument("--device", default="cuda")
    args = ap.parse_args(argv)

    from .. import _build
    _build.ensure_serving()
    from ..infer import EngineConfig, SamplingParams, create_engine, load_model
    from ..serve import Config, Request, Server

    prompts = [[int(t) for t in p.split(",")] for p in args.prompt]
    weights = load_model(args.model)
    vocab = weights.vocab
    for p in prompts:
        if any(t < 0 or t >= vocab for t in p):
            raise SystemExit(f"token ids must lie in 0 .. {vocab - 1}")
    longest = max(len(p) for p in prompts)
    block = 16
    held = sum(-(-(len(p) + args.max_new) // block) * block for p in prompts)
    seqs = min(64, len(prompts))
    engine = create_engine(weights, EngineConfig(device=args.device, precision=args.precision, max_seqs=seqs, kv_tokens=held,
                                                 context=longest + args.max_new, max_tokens=max(2048, longest + seqs),
                                                 block_size=block))
    server = Server(engine, Config(max_batch_tokens=engine.cfg.max_tokens, max_running=seqs))
    sampling = SamplingParams(temperature=args.temperature, top_k=args.top_k, top_p=args.top_p, seed=args.seed)
    futures = [server.submit(Request(p, args.max_new, sampling=sampling, stop_token=args.stop)) for p in prompts]
    server.run_until_idle()
    for p, f in zip(prompts, futures):
        r = f.result()
        print(json.dumps({"prompt": p, "tokens": r.tokens, "ttft_ms": round(r.ttft_ms, 3), "tpot_ms": round(r.tpot_ms, 3)}))
    return 0


if __name__ == "__main__":
    sys.exit(main())
