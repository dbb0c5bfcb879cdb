"""Trace replay: feeds given token ids through a decoder stack, step by step, and writes logits. Nothing is sampled. It
drives the decoder that serves the model (`StackDecoder`: its forward pass, paged cache and kernels).

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps.jsonl

A line of standard input is one step:
    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": ["a"]}
`entries`: the next tokens of requests (several per step if wanted) and the places among them whose logits are asked for;
`end`: requests that are finished after the step, whose pages go back to the pool. A step that asks for something writes
<out>/<step>.f32 (little-endian fp32 [wanted, vocab], in the order of the entries); after every step the line `done <step>`
is printed. float32 runs everything in true 32-bit.
"""
from __future__ import annotations

import argparse
import json
import os
import sys
from pathlib import Path
from typing import Dict, List, Optional

import torch


class TraceRunner:
    def __init__(self, model_dir, dtype: torch.dtype, device, max_tokens: int, page_size: int = 32):
        from ..models.stack import load_stack
        from .decoder import StackDecoder

        self.model = load_stack(model_dir, dtype, device)
        pages = (max_tokens + page_size - 1) // page_size + 64   # every live request may leave its last page part-filled
        self.dec = StackDecoder(self.model, page_size, max_batch=1, max_len=max(1, max_tokens), num_pages=pages)
        self.seq_of: Dict[str, int] = {}
        self.have: Dict[str, int] = {}
        self._next = 0

    def step(self, entries: List[dict], end: List[str]) -> Optional[torch.Tensor]:
        """-> wanted logits [m, vocab] fp32 on the host, or None when the step asks for none."""
        run = []
        for e in entries:
            rid, toks = e["id"], e["tokens"]
            if rid not in self.seq_of:
                self.seq_of[rid], self.have[rid] = self._next, 0
                self._next += 1
            if not toks:
                continue
            if not self.dec.cache.reserve(self.seq_of[rid], len(toks)):
                raise RuntimeError("the cache is full: --max-tokens is too small for this trace")
            run.append((self.seq_of[rid], toks, self.have[rid], e.get("want", [])))
            self.have[rid] += len(toks)
        out = None
        if run:
            logits = self.dec.run_portions(run)
            if any(e[3] for e in run):
                out = logits.float().cpu()
        for rid in end:
            if rid in self.seq_of:
                self.dec.cache.release(self.seq_of.pop(rid))
                del self.have[rid]
        return out


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, default=8192, help="most tokens that live requests hold at any time")
    ap.add_argument("--page-size", type=int, default=32)
    ap.add_argument("--device", default="cuda", help="cuda, or cpu for the plain definitions (tests)")
    args = ap.parse_args(argv)
    from .. import ops

    device = torch.device(args.device)
    if device.type == "cuda":
        if not torch.cuda.is_available():
            raise RuntimeError("no CUDA device (use --device cpu for the plain definitions)")
        torch.backends.cuda.matmul.allow_tf32 = False
        torch.backends.cudnn.allow_tf32 = False
        torch.cuda.set_device(device.index or 0)
        if not ops.load_extension():
            raise RuntimeError(f"the kernel library failed to build or load: {ops._load_error}")
    runner = TraceRunner(args.model, getattr(torch, args.dtype), device, args.max_tokens, args.page_size)
    out = Path(args.out)
    out.mkdir(parents=True, exist_ok=True)
    for line in sys.stdin:
        if not line.strip():
            continue
        doc = json.loads(line)
        logits = runner.step(doc.get("entries", []), doc.get("end", []))
        ops.check_status()
        if logits is not None:
            tmp = out / f".{doc['step']}.tmp"
            logits.contiguous().numpy().astype("<f4").tofile(tmp)
            os.replace(tmp, out / f"{doc['step']}.f32")
        print(f"done {doc['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
