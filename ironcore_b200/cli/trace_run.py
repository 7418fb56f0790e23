"""``bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N``: replay recorded token ids on the
rollout engine and write logits (no sampling).

Standard input holds one JSON object per line::

    {"step": 7, "entries": [{"id": "q1", "tokens": [12, 4], "want": [1]}, {"id": "q2", "tokens": [9]}], "end": ["q2"]}

The entries of a line form one batch: each continues (or opens) request ``id`` by ``tokens``, and ``want`` indexes the
tokens to report. Requests under ``end`` are closed once the step has run. Reported logits go to ``DIR/<step>.f32``
(little-endian fp32, [reported, vocab], entry order); ``done <step>`` on standard output follows every step.
``--max-tokens`` and ``--max-seqs`` size the cache."""

from __future__ import annotations

import argparse
import json
import os
import sys

PAGE = 64       # tokens


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.split("\n\n")[0],
                                 formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--model", required=True, help="directory with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="directory that receives <step>.f32")
    ap.add_argument("--max-tokens", type=int, default=65536, help="upper bound of the tokens in the cache")
    ap.add_argument("--max-seqs", type=int, default=256, help="upper bound of the open requests")
    args = ap.parse_args(argv)

    import torch

    from ..checkpoint.pretrained import load_pretrained
    from ..ops import native
    from ..parallel import mesh
    from ..rl import RolloutEngine

    # float32 means 32-bit products
    torch.backends.cuda.matmul.allow_tf32 = False
    torch.set_float32_matmul_precision("highest")
    dev = torch.device("cpu")
    if torch.cuda.is_available():
        dev = torch.device("cuda", torch.cuda.current_device())
    model, config = load_pretrained(args.model, precision=args.dtype, device=dev)
    if dev.type == "cuda":
        native.require(model.native_symbols())
    limit = max(1, args.max_tokens)
    seqs = max(1, min(args.max_seqs, limit))
    # every live request may leave its last page partly filled
    engine = RolloutEngine(model, config, max_seqs=seqs, max_seq_len=limit, block_size=PAGE,
                           num_blocks=(limit + PAGE - 1) // PAGE + seqs)
    if mesh.is_rank_zero():
        os.makedirs(args.out, exist_ok=True)
    for line in sys.stdin:
        if not line.strip():
            continue
        doc = json.loads(line)
        number, entries = int(doc["step"]), doc.get("entries") or []
        if entries:
            logits = engine.step([(e["id"], e["tokens"], e.get("want") or []) for e in entries])
            if any(e.get("want") for e in entries):
                rows = logits[:, :model.vocab_size].float().cpu().contiguous().numpy().astype("<f4")
                with open(os.path.join(args.out, f"{number}.f32"), "wb") as f:
                    f.write(rows.tobytes())
        engine.end(doc.get("end") or [])
        if dev.type == "cuda":
            native.check_status()
        print(f"done {number}", flush=True)
    return 0
