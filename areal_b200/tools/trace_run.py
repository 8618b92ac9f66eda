"""Replays a token trace through the rollout engine and writes logits.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N  < steps.jsonl

Every line of standard input is one step:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

The requests of a step either all start (``tokens`` is the whole prompt so far) or all go on by one token; ``want`` are
the places among a request's tokens whose logits are asked for, ``end`` the requests that are finished after the step.
When something is wanted, ``DIR/<step>.f32`` receives the logits ``[wanted, vocab]`` as little-endian 32-bit floats.
After every step a line ``done <step>`` is printed. Native libraries that are missing are built first.
"""

from __future__ import annotations

import argparse
import json
import os
import sys


def parse_args(argv=None) -> argparse.Namespace:
    ap = argparse.ArgumentParser(description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    ap.add_argument("--max-requests", type=int, default=256, help="most requests that are live at any time")
    ap.add_argument("--device", default=None)
    return ap.parse_args(argv)


def build_engine(args):
    from ..api.cli_args import InferenceEngineConfig, NativeRolloutConfig
    from ..engine.rollout_engine import NativeRolloutEngine

    bs, n = 16, max(args.max_tokens, 1)
    seqs = max(1, min(args.max_requests, n))
    native = NativeRolloutConfig(model_path=args.model, dtype=args.dtype, kv_block_size=bs, context_length=n + bs,
                                 max_num_seqs=seqs, max_num_batched_tokens=n,
                                 # every request may leave one page partly used and holds one ahead
                                 num_kv_blocks=-(-n // bs) + 2 * seqs, cuda_graph_batch_sizes=[1, 2, 4, 8, 16, 32])
    eng = NativeRolloutEngine(InferenceEngineConfig(backend="native:d1", native=native))
    return eng.initialize(start_loop=False, **({"device": args.device} if args.device else {}))


def main(argv=None) -> int:
    args = parse_args(argv)
    from .. import build

    build.build()
    from ..engine.trace_replay import TraceEntry, TraceReplay

    engine = build_engine(args)
    replay = TraceReplay(engine)
    try:
        for line in sys.stdin:
            if not line.strip():
                continue
            st = json.loads(line)
            logits = replay.step([TraceEntry(str(x["id"]), list(x["tokens"]), list(x.get("want", [])))
                                  for x in st.get("entries", [])], [str(x) for x in st.get("end", [])])
            if logits is not None:
                logits.numpy().astype("<f4").tofile(os.path.join(args.out, f"{st['step']}.f32"))
            print(f"done {st['step']}", flush=True)
    finally:
        engine.destroy()
    return 0


if __name__ == "__main__":
    sys.exit(main())
