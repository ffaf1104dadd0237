"""Trace replay: feeds given token ids through the serving engine step by step and writes the logits asked for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps

Every input line is one step, ``{"step": n, "entries": [{"id", "tokens", "want"}], "end": [ids]}``: the next tokens of
some requests and the places among them whose logits are wanted.  For a step in which something is wanted
``OUT/<step>.f32`` receives the logits (little-endian fp32, [wanted, vocab]); after every step ``done <step>`` is
printed.  A request's cache pages are given back when it is named in ``end``.  Nothing is sampled: this is the
engine's own ``run_tokens`` over its cache, decode graphs and kernels."""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import Any, Dict, List, Optional, TextIO

import torch

from .engine import YvEngineConfig, YvInferenceEngine

DTYPES = {"bfloat16": torch.bfloat16, "float32": torch.float32}


class YvTraceReplayer:
    def __init__(self, engine: YvInferenceEngine, out_dir: str):
        self.engine, self.out_dir = engine, out_dir
        self.ids: Dict[str, int] = {}
        self._next = 0

    def step(self, spec: Dict[str, Any]) -> Optional[torch.Tensor]:
        """Run one step; returns the wanted logits [wanted, vocab] on the host (None when nothing is wanted)."""
        eng, rows = self.engine, []
        for e in spec["entries"]:
            if not e["tokens"]:
                continue
            if e["id"] not in self.ids:
                self.ids[e["id"]] = self._next
                eng.cache.add_sequence(self._next)
                self._next += 1
            logits = eng.run_tokens(self.ids[e["id"]], [int(t) for t in e["tokens"]], [int(w) for w in e["want"]])
            if logits is not None:
                rows.append(logits.float().cpu())
        for rid in spec.get("end", []):
            if rid in self.ids:
                eng.cache.free_sequence(self.ids.pop(rid))
        if eng.device.type == "cuda":
            from ..ops import check_status
            check_status(eng.device)
        return torch.cat(rows, 0) if rows else None

    def run(self, lines: TextIO, report: TextIO) -> None:
        for line in lines:
            if not line.strip():
                continue
            spec = json.loads(line)
            got = self.step(spec)
            if got is not None:
                with open(os.path.join(self.out_dir, f"{spec['step']}.f32"), "wb") as f:
                    f.write(got.contiguous().numpy().astype("<f4").tobytes())
            report.write(f"done {spec['step']}\n")
            report.flush()


def pages_for(max_tokens: int, block_size: int) -> int:
    """Cache pages for live requests of ``max_tokens`` tokens in all, with room for partly filled pages."""
    return -(-max_tokens // block_size) + 64


def main(argv: Optional[List[str]] = None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="replay a trace of token ids and write logits")
    ap.add_argument("--model", required=True, help="checkpoint folder (config.json, model.safetensors)")
    ap.add_argument("--dtype", choices=sorted(DTYPES), default="bfloat16")
    ap.add_argument("--out", required=True, help="folder for the logits files")
    ap.add_argument("--max-tokens", type=int, default=65536, help="most tokens held by live requests at any time")
    args = ap.parse_args(argv)
    if not torch.cuda.is_available():
        print("trace_run needs a GPU", file=sys.stderr)
        return 2
    from ..engine.loader import folder_config, load_model_for_inference
    from ..models.registry import kernel_families
    from ..ops import load_extension
    named = folder_config(args.model)
    load_extension(build_if_missing=True, families=kernel_families(named) if named is not None else ())
    dtype = DTYPES[args.dtype]
    if dtype == torch.float32:
        torch.backends.cuda.matmul.allow_tf32 = torch.backends.cudnn.allow_tf32 = False
    model = load_model_for_inference(ckpt=args.model, device="cuda", dtype=dtype)
    cfg = YvEngineConfig(num_blocks=pages_for(args.max_tokens, YvEngineConfig.block_size), eos_token_id=-1)
    YvTraceReplayer(YvInferenceEngine(model, cfg=cfg), args.out).run(sys.stdin, sys.stdout)
    return 0
