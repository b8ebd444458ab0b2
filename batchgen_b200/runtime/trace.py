"""Trace replay: feed given token ids through a model step by step and write the logits that are asked for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps.jsonl

Every line of standard input is one step, ``{"step": 0, "entries": [{"id", "tokens", "want"}], "end": [ids]}``: the entries
are one batch of the engine (``Engine.extend``), ``want`` lists the places among an entry's tokens whose logits are written,
and the requests in ``end`` give their pages and state slots back after the step.  The logits of step n go to
``DIR/n.f32`` (little-endian fp32, [wanted, vocab], entry by entry); a line ``done n`` on standard output ends every step.

Nothing is sampled.  The engine's page pool holds ``--max-tokens`` tokens (requests rounded up to whole pages) and its state
pool four requests, so pages and slots are used again as requests come and go.
"""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import Dict, List, Optional

PAGE = 64
LIVE_REQUESTS = 4


class TraceReplay:
    """The step loop over an engine; ``run_step`` takes one parsed step."""

    def __init__(self, engine, out_dir: str):
        self.engine, self.out_dir = engine, out_dir
        self.live: Dict[str, object] = {}

    def run_step(self, step: dict) -> Optional[str]:
        """Runs one step; returns the path of its logits file, or None when nothing was wanted."""
        pieces = []
        for e in step["entries"]:
            if e["id"] not in self.live:
                self.live[e["id"]] = self.engine.open_sequence(custom_id=str(e["id"]))
            pieces.append((self.live[e["id"]], e["tokens"], e.get("want", [])))
        logits = self.engine.extend(pieces)
        path = None
        if logits.shape[0]:
            path = os.path.join(self.out_dir, f"{step['step']}.f32")
            data = logits.float().cpu().numpy().astype("<f4")
            with open(path, "wb") as f:
                f.write(data.tobytes())
        elif self.engine.device.type == "cuda":
            self.engine._sync()
        for rid in step.get("end", []):
            seq = self.live.pop(rid, None)
            if seq is not None:
                self.engine.close_sequence(seq)
        return path


def build_engine(model_dir: str, dtype: str, max_tokens: int, device: str = "cuda"):
    from ..config import EngineConfig, get_model_config
    from ..models import build_model
    from .engine import Engine
    cfg = get_model_config(model_dir)
    dt = {"bfloat16": "bf16", "float32": "fp32"}[dtype]
    model = build_model(cfg, device=device, dtype=dt)
    ecfg = EngineConfig(page_size=PAGE, device=device, dtype=dt, max_decode_batch=LIVE_REQUESTS,
                        max_state_slots=LIVE_REQUESTS, enable_cuda_graph=False)
    return Engine(model, ecfg, num_gpu_pages=max(1, -(-max_tokens // PAGE)))


def main(argv: Optional[List[str]] = None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="replay a trace of token ids and write logits")
    ap.add_argument("--model", required=True, help="directory with config.json and .safetensors files")
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    ap.add_argument("--out", required=True, help="directory the logits files are written to")
    ap.add_argument("--max-tokens", type=int, required=True, help="tokens the page pool holds")
    ap.add_argument("--device", default="cuda", help="cuda, or cpu with --dtype float32")
    a = ap.parse_args(argv)
    if a.device == "cuda":
        from .. import build
        from ..ops import _ext
        _ext.use_library(build.layered_library())
    replay = TraceReplay(build_engine(a.model, a.dtype, a.max_tokens, a.device), a.out)
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        replay.run_step(step)
        print(f"done {step['step']}", flush=True)
    if a.device == "cuda":
        from ..ops import _ext
        _ext.check_status()
    return 0
