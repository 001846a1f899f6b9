"""trace_run: replay given token ids through a model, step by step, and write the logits asked for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

DIR is a checkpoint folder (``config.json``, ``model.safetensors``). Steps come on standard input, one
JSON object a line: ``{"step": n, "entries": [{"id": ..., "tokens": [...], "want": [...]}], "end": [...]}``.
The entries of a step form one batch of the engine: a request's tokens continue what earlier steps left
in its pages and state slot. ``want`` lists places among the entry's tokens; their logits go to
``OUT/<step>.f32`` (little-endian fp32, entry order). Requests in ``end`` give back what they hold.
After every step ``done <step>`` is printed. Nothing is sampled.

``--max-tokens`` sizes the page pool (tokens of all live requests together, each rounded up to 64) and
there are four state slots. Kernels that are not built yet are compiled first.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

SLOTS = 4
PAGE = 16


def build_parser() -> argparse.ArgumentParser:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--model", required=True)
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True)
    ap.add_argument("--max-tokens", type=int, required=True)
    ap.add_argument("--device", default="cuda")
    return ap


class TraceReplay:
    """Requests by name on top of an engine's step."""

    def __init__(self, engine):
        self.engine = engine
        self.seqs: dict = {}

    def run(self, step: dict):
        """Logits [wanted, vocab] of one step, or None when nothing is wanted."""
        eng, entries = self.engine, [e for e in step["entries"] if e["tokens"]]
        for e in entries:
            if e["id"] not in self.seqs:
                self.seqs[e["id"]] = eng.cache.new_sequence()
        out = None
        if entries:
            out = eng.step([self.seqs[e["id"]] for e in entries], [e["tokens"] for e in entries],
                           [e.get("want", []) for e in entries])
        for rid in step.get("end", []):
            if rid in self.seqs:
                eng.release(self.seqs.pop(rid))
        return out


def main(argv=None) -> int:
    args = build_parser().parse_args(argv)
    import torch

    from .. import build
    from ..models import registry

    build.ensure_hybrid()
    from ..infer.engine import InferenceEngine
    from ..ops import native

    model = registry.load_checkpoint(args.model, device=args.device)
    pages = (args.max_tokens + PAGE - 1) // PAGE
    engine = InferenceEngine.from_model(model, device=args.device, dtype=args.dtype, max_batch=SLOTS,
                                        max_seq_len=min(model.cfg.context_limit, pages * PAGE), page_size=PAGE, kv_pages=pages)
    del model
    replay = TraceReplay(engine)
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        logits = replay.run(step)
        if logits is not None:
            data = logits.float().cpu().numpy().astype("<f4")
            with open(os.path.join(args.out, f"{step['step']}.f32"), "wb") as f:
                f.write(data.tobytes())
        else:
            torch.cuda.synchronize()
        native.check_status(args.device)
        print(f"done {step['step']}", flush=True)
    return 0
