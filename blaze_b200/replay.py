"""Replay a trace: token ids go through a model step by step, and chosen logits come out.  Nothing is sampled; the steps are the
engine's own (``Engine.plan`` / ``Engine.forward``), over its paged cache, as the scheduler issues them.

Steps are JSON lines on standard input::

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": ["b"]}

``entries`` bring the next tokens of requests (one batch), ``want`` names the places among them whose logits are written to
``<out>/<step>.f32`` (little-endian fp32, ``[wanted, vocab]``); ``end`` closes requests after the step.  ``done <step>`` is
printed after each.
"""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import Dict, Optional, Sequence

MAX_LIVE = 4                # requests that may be live at a time


def build_parser() -> argparse.ArgumentParser:
    ap = argparse.ArgumentParser(prog="trace_run", description="replay token ids through a model step by step and write logits")
    ap.add_argument("--model", required=True, help="checkpoint directory")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="directory of the logits")
    ap.add_argument("--max-tokens", type=int, required=True, help="tokens the cache holds, over all live requests")
    ap.add_argument("--device", default="cuda")
    return ap


def main(argv: Optional[Sequence[str]] = None) -> int:
    a = build_parser().parse_args(argv)
    import torch

    from .batch import PAGE
    from .config import ModelConfig
    from .llm import LLM
    from .models import model_class
    dtype = {"bfloat16": torch.bfloat16, "float32": torch.float32}[a.dtype]
    cfg = ModelConfig.load(a.model)
    if a.device != "cpu" and dtype not in model_class(cfg).cuda_dtypes:
        print(f"{cfg.architecture} does not run in {a.dtype}", file=sys.stderr)
        return 3
    tokens = -(-a.max_tokens // PAGE) * PAGE
    llm = LLM(a.model, device=a.device, dtype=dtype, kv_tokens=tokens, max_seqs=MAX_LIVE, max_model_len=tokens,
              enable_prefix_caching=False)
    os.makedirs(a.out, exist_ok=True)
    eng, live = llm.engine, {}
    for line in sys.stdin:
        if line.strip():
            step = json.loads(line)
            run_step(eng, live, step, a.out)
            print(f"done {step['step']}", flush=True)
    return 0


def run_step(eng, live: Dict[str, object], step: dict, out_dir: str) -> None:
    """One step: ``live`` maps request ids to their sequences."""
    items, wanted = [], 0
    for e in step["entries"]:
        if e["id"] not in live:
            live[e["id"]] = eng.open_from()
        if e["tokens"]:
            items.append((live[e["id"]], e["tokens"], list(e.get("want") or ())))
            wanted += len(items[-1][2])
    if items:
        logits = eng.forward(eng.plan(items), "logits" if wanted else "none")
        if wanted:
            rows = logits.float().cpu().contiguous().numpy().astype("<f4", copy=False)
            part = os.path.join(out_dir, f"{step['step']}.f32.part")
            rows.tofile(part)
            os.replace(part, part[:-5])
        elif eng.device.type == "cuda":
            import torch
            torch.cuda.synchronize(eng.device)
        eng.check_status()
    for rid in step.get("end") or ():
        eng.close(live.pop(rid))


if __name__ == "__main__":
    sys.exit(main())
