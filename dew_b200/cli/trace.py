"""``bin/trace_run``: feed given token ids through a released model, step by step, and write logits; nothing is sampled.

Standard input holds one JSON object a line::

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": ["a"]}

The entries of a step are one batch: rows that all start, or all go on from the cache and the state earlier steps left.  The logits at the
``want`` places go to ``OUT/<step>.f32`` (little-endian fp32 ``[wanted, vocab]``, in the order of the entries), and ``done <step>`` is printed
after every step.  Requests under ``end`` give back what they hold.  The steps run through ``sampling.text.RowBatch``, the loop ``generate``
itself uses.
"""
from __future__ import annotations

import argparse
import json
import sys
from pathlib import Path
from typing import Dict, List, Optional, Sequence


class TraceSession:
    """The requests of a trace as rows of a ``RowBatch``; a batch that needs more rows than the last one gets a new cache."""

    def __init__(self, model, max_tokens: int):
        self.model, self.max_tokens = model, max(1, int(max_tokens))
        self.batch = None
        self.row_of: Dict[str, int] = {}

    def step(self, entries: Sequence[dict], end: Sequence[str]):
        """-> logits ``[wanted, vocab]`` or None."""
        from ..sampling.text import RowBatch
        fresh = [e for e in entries if e["id"] not in self.row_of]
        if self.batch is None or len(self.row_of) + len(fresh) > self.batch.rows:
            if self.row_of:
                raise ValueError("a running batch has no free row for another request")
            limit = getattr(self.model.config, "max_seq_len", self.max_tokens)
            self.batch = RowBatch(self.model, max(1, len(fresh)), min(limit, self.max_tokens), pool_tokens=self.max_tokens)
        free = [r for r in range(self.batch.rows) if r not in self.row_of.values()]
        for e in fresh:
            self.row_of[e["id"]] = free.pop(0)
        pieces: List[List[int]] = [[] for _ in range(self.batch.rows)]
        want: List[List[int]] = [[] for _ in range(self.batch.rows)]
        order = []
        for e in entries:
            r = self.row_of[e["id"]]
            pieces[r], want[r] = list(e["tokens"]), list(e.get("want") or [])
            order.append(r)
        logits = self.batch.feed(pieces, want)
        if logits is not None:
            # ``feed`` returns the rows' logits in row order; the trace wants them in the order of its entries
            first, at = [0] * self.batch.rows, 0
            for r in range(self.batch.rows):
                first[r], at = at, at + len(want[r])
            logits = logits[[first[r] + j for r in order for j in range(len(want[r]))]]
        for i in end:
            self.batch.release(self.row_of.pop(i))
        return logits


def main(argv: Optional[Sequence[str]] = None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay a trace of token ids through a model and write the logits it asks for.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder the logits are written to")
    ap.add_argument("--max-tokens", type=int, required=True, help="the most tokens live requests hold at any time (sizes the cache)")
    ap.add_argument("--device", default="cuda", help="cuda (default); cpu runs the plain PyTorch forms of the operations")
    args = ap.parse_args(argv)

    import torch

    from ..interop.hf import Pretrained
    from ..ops import library
    if args.device == "cuda":
        if not torch.cuda.is_available():
            print("trace_run: no CUDA device", file=sys.stderr)
            return 2
        library.load_part("decoder")
    torch.backends.cuda.matmul.allow_tf32 = False
    torch.backends.cudnn.allow_tf32 = False
    model = Pretrained.load(args.model, dtype=getattr(torch, args.dtype), device=args.device).eval()
    for p in model.parameters():
        p.requires_grad_(False)
    session = TraceSession(model, args.max_tokens)
    out = Path(args.out)
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        logits = session.step(step["entries"], step.get("end") or [])
        if logits is not None:
            (out / f"{step['step']}.f32").write_bytes(logits.float().cpu().contiguous().numpy().astype("<f4").tobytes())
        if args.device == "cuda":
            library.check_status()
        print(f"done {step['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
