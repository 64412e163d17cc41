"""Replays a recorded request trace through a model and writes logits instead of sampling.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps.jsonl

Every input line is a step: ``{"step": n, "entries": [{"id", "tokens", "want"}], "end": [ids]}``.  All entries of a step run as one batch
through :class:`~torchtune_b200.generation.BatchDecoder`: either every request is new (its whole prompt), or every live request goes on by
one token.  ``want`` lists places among an entry's tokens; their logits go to ``DIR/<n>.f32`` (little-endian fp32, ``[wanted, vocab]``, in
the order given).  ``done <n>`` is printed after each step; requests named in ``end`` give their cache rows back."""
from __future__ import annotations

import argparse
import json
import sys
from pathlib import Path
from typing import Any, Dict, List, Optional

import torch

from ._rows import BatchDecoder

DTYPES = {"bfloat16": torch.bfloat16, "float32": torch.float32}


class TraceReplay:
    def __init__(self, decoder: BatchDecoder, out: Path) -> None:
        self.decoder, self.out = decoder, out
        self.live: List[str] = []  # requests by cache row

    def run(self, step: Dict[str, Any]) -> None:
        entries = step["entries"]
        ids = [e["id"] for e in entries]
        if entries and not self.live:
            hidden = self.decoder.begin([e["tokens"] for e in entries])
            self.live = ids
            at = [hidden.shape[1] - len(e["tokens"]) for e in entries]  # first own place of a left-padded row
        elif entries:
            if sorted(ids) != sorted(self.live) or any(len(e["tokens"]) != 1 for e in entries):
                raise ValueError(f"step {step['step']}: a running batch goes on with one token of each of its requests")
            token = {e["id"]: e["tokens"][0] for e in entries}
            hidden = self.decoder.advance([token[i] for i in self.live])
            at = [0] * len(entries)
        rows = [(self.live.index(e["id"]), at[k] + w) for k, e in enumerate(entries) for w in e["want"]]
        if rows:
            picked = hidden[[r for r, _ in rows], [c for _, c in rows]]
            logits = self.decoder.logits(picked).float().cpu().numpy().astype("<f4")
            (self.out / f"{step['step']}.f32").write_bytes(logits.tobytes())
        ended = [self.live.index(i) for i in step.get("end", [])]
        if ended:
            self.decoder.end(ended)
            self.live = [i for k, i in enumerate(self.live) if k not in set(ended)]


def main(argv: Optional[List[str]] = None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay a request trace and write logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and *.safetensors")
    ap.add_argument("--dtype", required=True, choices=sorted(DTYPES))
    ap.add_argument("--out", required=True, help="folder for <step>.f32 files")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    args = ap.parse_args(argv)

    from ..models._registry import load_pretrained
    from ..ops import build
    from ..ops._lib import check_device_errors

    if not torch.cuda.is_available():
        raise RuntimeError("no CUDA device: the trace runner drives the GPU kernels")
    build.build()
    torch.set_float32_matmul_precision("highest")
    torch.backends.cuda.matmul.allow_bf16_reduced_precision_reduction = False
    device, dtype = torch.device("cuda"), DTYPES[args.dtype]
    out = Path(args.out)
    with torch.inference_mode():
        model = load_pretrained(args.model, dtype=dtype, device=device, max_seq_len=max(args.max_tokens, 1))
        replay = TraceReplay(BatchDecoder(model, device, dtype, args.max_tokens), out)
        for line in sys.stdin:
            if not line.strip():
                continue
            step = json.loads(line)
            replay.run(step)
            torch.cuda.synchronize()
            check_device_errors()
            print(f"done {step['step']}", flush=True)
    return 0
