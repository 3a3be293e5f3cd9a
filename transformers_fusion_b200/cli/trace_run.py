"""trace_run: replay given token ids through a model folder, step by step, and write the logits that are asked for.

    trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N  < steps.jsonl

One JSON object a line on standard input:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

``entries``: the next tokens of each request and the places among them whose logits are wanted; ``end``: requests that are
finished after the step.  The logits of a step go to DIR/<step>.f32 (little-endian fp32, [wanted, vocab], in the order of the
entries and their ``want``), then the line "done <step>" is printed.  Nothing is sampled; the tokens run through
``InferenceEngine.feed``, i.e. the prefill and decode passes, cache and CUDA graphs that generation uses.  Exit code 3: the
model's class does not run in that dtype."""
from __future__ import annotations

import argparse
import json
import os
import sys


def main(argv=None):
    ap = argparse.ArgumentParser(prog="trace_run")
    ap.add_argument("--model", required=True)
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True)
    ap.add_argument("--max-tokens", type=int, default=4096, help="the most tokens that live requests hold at any time")
    ap.add_argument("--device", default="cuda")
    a = ap.parse_args(argv)
    import torch

    from ..inference.engine import EngineConfig, InferenceEngine, Request
    from ..inference.kv_cache import PAGE
    from ..models import registry
    from ..ops import _lib
    if a.device.startswith("cuda") and not torch.cuda.is_available():
        print("Error: no CUDA device", file=sys.stderr)
        return 1
    dev = torch.device(a.device)
    registry.limit_build(a.model)
    model = registry.load_folder(a.model, dev, getattr(torch, a.dtype))
    if a.dtype == "float32" and not getattr(model, "runs_fp32", False):
        print(f"Error: {type(model).__name__} does not run in 32-bit", file=sys.stderr)
        return 3
    max_batch = max(1, min(256, a.max_tokens))
    eng = InferenceEngine(model, None, EngineConfig(max_batch=max_batch, num_pages=a.max_tokens // PAGE + 2 * max_batch + 2,
                                                    max_seq_len=a.max_tokens + 1, enable_prefix_cache=False))
    live = {}
    for line in sys.stdin:
        if not line.strip():
            continue
        s = json.loads(line)
        entries = [(live.setdefault(e["id"], Request([])), e["tokens"], e.get("want", [])) for e in s["entries"]]
        got = [x for x in eng.feed(entries) if x is not None]
        if got:
            rows = torch.cat(got).float().cpu().contiguous().numpy().astype("<f4")
            path = os.path.join(a.out, f"{s['step']}.f32")
            with open(path + ".part", "wb") as f:
                f.write(rows.tobytes())
            os.replace(path + ".part", path)
        for i in s.get("end", []):
            eng.end(live.pop(i))
        if dev.type == "cuda":
            _lib.check_status(dev)
        print(f"done {s['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
