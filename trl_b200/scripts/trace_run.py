"""Trace replay: given token ids are fed through a model step by step, logits are written.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Steps come on standard input, one JSON object a line:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

``want``: places among the entry's tokens whose logits go to ``OUT/<step>.f32`` (little-endian fp32 [wanted, vocab], in
the order of the entries); ``end``: requests that are released after the step.  After every step ``done <step>`` is
printed.  The model runs on the serving engine that generation uses (rollout/engine.py: ``make_engine``), without
sampling.  Native libraries are built first if they are missing.  Exit code 3: the model is not served in float32."""
from __future__ import annotations

import argparse
import json
import os
import sys


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="replay a trace of token steps and write logits")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    ap.add_argument("--max-seqs", type=int, default=16, help="slots of the engine (a larger first batch raises it)")
    a = ap.parse_args(argv)

    from .._native import lib_path
    from ..csrc.build import build
    from ..models.layered import is_layered_dir, layered_kinds

    # a fresh checkout compiles what the model needs; an existing complete library is kept up to date
    if is_layered_dir(a.model) and not os.path.exists(lib_path("libtrl_b200_kernels.so")):
        build(part="layered", kinds=layered_kinds(a.model))
    else:
        build()
    import torch

    from ..models.hf_io import load_model
    from ..rollout.engine import make_engine
    from ..rollout.feed import TokenFeed

    dtype = getattr(torch, a.dtype)
    model = load_model(a.model, dtype=dtype, device="meta")
    if dtype == torch.float32 and not getattr(model, "serves_float32", False):
        print("this model is served in bfloat16 only", file=sys.stderr)
        return 3
    model = load_model(a.model, dtype=dtype, device="cuda").eval().requires_grad_(False)
    feed = None
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        entries = [(e["id"], e["tokens"], e["want"]) for e in step["entries"]]
        if feed is None or (feed.live == 0 and len(entries) > feed.e.max_seqs):
            slots = max(a.max_seqs, len(entries))
            block = 64 if a.dtype == "bfloat16" else 32
            feed = TokenFeed(make_engine(model, max_num_seqs=slots, max_model_len=a.max_tokens, block_size=block,
                                         num_blocks=-(-a.max_tokens // block) + slots))
        logits = feed.step(entries, step.get("end", []))
        rows = torch.cat(logits) if logits else torch.empty(0)
        if rows.numel():
            with open(os.path.join(a.out, f"{step['step']}.f32"), "wb") as f:
                f.write(rows.float().cpu().contiguous().numpy().astype("<f4").tobytes())
        else:
            torch.cuda.synchronize()
        from ..ops import cuda as K

        K.check_status()
        print(f"done {step['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
