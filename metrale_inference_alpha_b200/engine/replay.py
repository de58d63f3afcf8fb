"""Replays a trace of given token ids through a model, step by step, and writes logits.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Steps arrive on standard input, one JSON object a line:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

The entries of a step are one batch: portions of prompts run beside single decoded tokens. "want" names the
places among an entry's tokens whose logits are asked for; a step with any writes <out>/<step>.f32, little-endian
32-bit floats [wanted, vocab] in the order of the entries. "end" lists the requests that are finished after the
step. After every step a line "done <step>" is printed. Nothing is sampled; everything else is the engine's own:
its model and weights, its cache blocks and state slots, its batch staging, step functions and decode graphs.
"""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import Dict, List, Optional

import torch

from ..scheduler.types import StepPlan
from .llm_engine import EngineArgs, LLMEngine

MAX_LIVE = 4
DTYPES = {"bfloat16": "bf16", "float32": "fp32"}


class TraceReplay:
    """An engine whose pools hold ``max_tokens`` tokens and MAX_LIVE states, fed from outside."""

    def __init__(self, model, dtype: str = "bf16", max_tokens: int = 2048, device: str = "cuda:0", block_size: int = 16,
                 use_cuda_graphs: bool = True, max_live: int = MAX_LIVE):
        blocks = (max_tokens + block_size - 1) // block_size + 1          # and the null block
        self.engine = LLMEngine(EngineArgs(
            model=model, device=device, dtype=dtype, max_num_seqs=max_live, max_model_len=max_tokens, max_prefill_tokens=max_tokens,
            block_size=block_size, num_kv_blocks=blocks, enable_prefix_caching=False, use_cuda_graphs=use_cuda_graphs,
            state_snapshots=1))
        self.live: Dict[str, object] = {}

    def step(self, entries: List[dict], end: List[str]) -> Optional[torch.Tensor]:
        """Runs one step; returns the wanted logits [wanted, vocab] (fp32, host) or None."""
        sch = self.engine.scheduler
        items = []
        for e in entries:
            if e["id"] not in self.live:
                self.live[e["id"]] = sch.open_fed(e["id"])
            items.append(sch.feed(self.live[e["id"]], e["tokens"], e.get("want") or []))
        out = None
        if items:
            plan = StepPlan("mixed", items)
            out = self.engine.runner.execute_fed(plan)
            sch.fed(plan)
        for rid in end:
            sch.close_fed(self.live.pop(rid))
        return out


def add_arguments(ap: argparse.ArgumentParser) -> None:
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=sorted(DTYPES))
    ap.add_argument("--out", required=True, help="folder for the logits, <step>.f32")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    ap.add_argument("--device", default="cuda:0")


def run(ns, lines=None) -> int:
    replay = TraceReplay(ns.model, DTYPES[ns.dtype], ns.max_tokens, ns.device)
    for line in lines if lines is not None else sys.stdin:
        if not line.strip():
            continue
        s = json.loads(line)
        out = replay.step(s["entries"], s.get("end", []))
        if out is not None:
            with open(os.path.join(ns.out, f"{s['step']}.f32"), "wb") as f:
                f.write(out.contiguous().numpy().astype("<f4").tobytes())
        print(f"done {s['step']}", flush=True)
    return 0


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.splitlines()[0])
    add_arguments(ap)
    return run(ap.parse_args(argv))


if __name__ == "__main__":
    sys.exit(main())
