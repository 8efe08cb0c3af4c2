"""Feeds given token ids through a model, step by step, and writes logits.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Steps come from standard input, one JSON object a line:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

All entries of a step form one batch.  Logits at the wanted places go to OUT/<step>.f32 (little-endian
fp32, [wanted, vocab]); after every step the line "done <step>" is printed.  What has to be compiled is
compiled at the first call."""
from __future__ import annotations

import argparse
import json
import os
import sys


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__, formatter_class=argparse.RawTextHelpFormatter)
    ap.add_argument("--model", required=True, help="folder with config.json and *.safetensors")
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    ap.add_argument("--out", required=True, help="folder the logits are written to")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    ap.add_argument("--max-requests", type=int, default=4, help="most requests alive at any time")
    ap.add_argument("--device", choices=["cuda", "cpu"], default="cuda")
    args = ap.parse_args(argv)
    if args.max_tokens < 1:
        ap.error("--max-tokens must be positive")
    if args.device == "cuda":
        from .. import build
        with open(os.path.join(args.model, "config.json")) as f:
            d = json.load(f)
        build.ensure(d.get("architecture") or (d.get("architectures") or [""])[0])
    from ..engine.replay import TraceReplayer, make_replay_engine
    rp = TraceReplayer(make_replay_engine(args.model, args.dtype, args.max_tokens, args.max_requests,
                                          device=args.device))
    os.makedirs(args.out, exist_ok=True)
    for line in sys.stdin:
        if not line.strip():
            continue
        s = json.loads(line)
        logits = rp.step(s.get("entries", []), s.get("end", []))
        if logits is not None:
            path = os.path.join(args.out, f"{s['step']}.f32")
            with open(path + ".part", "wb") as f:
                f.write(logits.contiguous().numpy().astype("<f4").tobytes())
            os.replace(path + ".part", path)
        print(f"done {s['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
