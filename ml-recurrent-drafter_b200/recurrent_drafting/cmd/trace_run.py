"""Replays given token ids through a model, step by step, and writes the logits asked for.  Nothing is sampled.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N  < steps.jsonl

Standard input has one JSON object per line:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

entries: the next tokens of each named request and the places among them whose logits are wanted; end: the requests that
are finished after the step.  When something is wanted, OUT/<step>.f32 receives the logits [wanted, vocab] as
little-endian 32-bit floats, in the order of the entries and of `want`; then `done <step>` is printed.  The model is any
of the registry's, the steps run through the session that autoregressive generation uses.
"""
import argparse
import json
import os
import sys
from typing import Dict, List, Optional

import torch


class TraceRunner:
    """Requests by name over a Session; every live request owns a row of its batch."""

    def __init__(self, llm, max_tokens: int, rows: int = 1):
        from ..session import Session

        self.session = Session(llm, rows, max_tokens)
        self.device = llm.device
        self.row_of: Dict[str, int] = {}
        self.free: List[int] = list(range(rows))[::-1]

    def step(self, entries: List[dict], end: List[str]) -> Optional[torch.Tensor]:
        """Logits [wanted, vocab] on the device, or None when nothing is wanted."""
        live = [e for e in entries if e["tokens"]]
        for e in live:
            if e["id"] not in self.row_of:
                if not self.free:
                    raise RuntimeError(f"more live requests than the {self.session.batch} rows of the batch")
                self.row_of[e["id"]] = self.free.pop()
        counts = [0] * self.session.batch
        for e in live:
            counts[self.row_of[e["id"]]] += len(e["tokens"])
        by_row = sorted(live, key=lambda e: self.row_of[e["id"]])
        start, at = {}, 0
        for e in by_row:
            start[e["id"]] = at
            at += len(e["tokens"])
        out = None
        if live:
            ids = torch.tensor([t for e in by_row for t in e["tokens"]], dtype=torch.int64, device=self.device)
            hidden = self.session.extend(ids, counts)
            places = [start[e["id"]] + p for e in live for p in e.get("want", [])]
            if places:
                out = self.session.logits(hidden[torch.tensor(places, device=self.device)])
        for name in end:
            row = self.row_of.pop(name, None)
            if row is not None:
                self.session.release(row)
                self.free.append(row)
        return out


def main(argv: Optional[List[str]] = None) -> int:
    ap = argparse.ArgumentParser(description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--model", required=True)
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True)
    ap.add_argument("--max-tokens", type=int, required=True)
    ap.add_argument("--rows", type=int, default=1, help="requests that may be live at the same time")
    args = ap.parse_args(argv)

    from .. import registry

    if not torch.cuda.is_available():
        print("no CUDA device: this implementation has no CPU path", file=sys.stderr)
        return 2
    device = torch.device("cuda", torch.cuda.current_device())
    llm = registry.load_model(args.model, torch_dtype=getattr(torch, args.dtype), device=device)
    runner = TraceRunner(llm, max(args.max_tokens, 1), args.rows)
    for line in sys.stdin:
        if not line.strip():
            continue
        msg = json.loads(line)
        logits = runner.step(msg["entries"], msg.get("end", []))
        if logits is not None:
            data = logits.float().cpu().numpy().astype("<f4", copy=False)
            runner.session.check()
            path = os.path.join(args.out, f"{msg['step']}.f32")
            with open(path + ".part", "wb") as f:
                f.write(data.tobytes())
            os.replace(path + ".part", path)
        print(f"done {msg['step']}", flush=True)
    torch.cuda.synchronize()
    runner.session.check()
    return 0


if __name__ == "__main__":
    sys.exit(main())
