"""Replay a trace of token ids through a model, step by step, and write logits: `bin/trace_run`.

    trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N [--device cuda|cpu]

Logits only: every token comes from the trace. Steps go through the engine that the server and the command line use
(`Engine.forward` over segments, its paged cache and slots), so a recorded schedule (portions of prompts beside single decoded tokens,
requests that pause and go on) can be repeated and its logits compared between builds, schedules or precisions. Standard input holds
one JSON object per line:

    {"step": 7, "entries": [{"id": "q", "tokens": [11, 4], "want": [1]}, {"id": "p", "tokens": [9], "want": []}], "end": ["p"]}

An entry feeds a request its next tokens and names the ones (by place in `tokens`) whose logits to write; a request takes a slot with
its first entry. Requests listed under `end` give back their pages and slot when the step is done. Wanted logits go to
DIR/<step>.f32 (little-endian fp32 rows of the vocabulary, entries in order, places in order); after each step `done <step>` is
printed. `--max-tokens` is the size of the page pool in tokens, counted in whole pages of 64 per request.
"""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import Dict, List

SLOTS = 4
PAGE = 64


class TraceRunner:
    """Requests of a trace on the slots of an engine."""

    def __init__(self, engine):
        self.eng = engine
        self.slot: Dict[str, int] = {}
        self.free: List[int] = list(range(engine.ecfg.n_slots))

    def step(self, entries: List[dict], end: List[str]):
        """Run one step; returns the wanted logits [wanted, vocab] on the host, or None."""
        from ..engine.executor import Segment
        segs = []
        for e in entries:
            if e["id"] not in self.slot:
                if not self.free:
                    raise RuntimeError(f"more than {self.eng.ecfg.n_slots} live requests")
                self.slot[e["id"]] = self.free.pop(0)
            s = self.slot[e["id"]]
            if e["tokens"]:
                segs.append(Segment(s, self.eng.slot_len[s], [int(t) for t in e["tokens"]], [int(i) for i in e["want"]]))
        out = None
        if segs:
            logits, _, _ = self.eng.forward(segs, commit=True, greedy=False)
            if logits is not None:
                out = logits.float().cpu()
            self.eng.check()
        for rid in end:
            s = self.slot.pop(rid)
            self.eng.reset_slot(s)
            self.free.append(s)
        return out


def open_engine(model: str, dtype: str, max_tokens: int, device: str):
    import torch

    from ..config import EngineConfig, ModelConfig
    from ..engine.engine import Engine
    from ..formats.loader import load_model_weights
    if device == "cuda" and not torch.cuda.is_available():
        raise SystemExit("trace_run: no CUDA device (--device cpu runs the fp32 CPU engine)")
    cfg = ModelConfig.from_hf(os.path.join(model, "config.json"))
    weights = load_model_weights(model, cfg)
    tokens = (max_tokens + PAGE - 1) // PAGE * PAGE
    ecfg = EngineConfig(n_slots=SLOTS, kv_block=PAGE, max_ctx=tokens, kv_pool_tokens=tokens, max_step_rows=max(tokens, PAGE),
                        compute_dtype="fp32" if dtype == "float32" else "bf16")
    return Engine(cfg, weights, ecfg, device=device)


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.splitlines()[0])
    ap.add_argument("--model", required=True, help="folder with config.json and safetensors weights")
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder the logits go to")
    ap.add_argument("--max-tokens", type=int, required=True, help="tokens the page pool holds")
    ap.add_argument("--device", default="cuda", choices=["cuda", "cpu"])
    a = ap.parse_args(argv)
    run = TraceRunner(open_engine(a.model, a.dtype, a.max_tokens, a.device))
    for line in sys.stdin:
        if not line.strip():
            continue
        st = json.loads(line)
        out = run.step(st["entries"], st.get("end", []))
        if out is not None:
            out.numpy().astype("<f4").tofile(os.path.join(a.out, f"{st['step']}.f32"))
        print(f"done {st['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
