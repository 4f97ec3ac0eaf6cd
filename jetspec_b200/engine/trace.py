"""Replay a trace: feed given token ids through a model step by step and write the logits that are asked for.

Nothing is sampled.  Requests enter through the scheduler, every step is one ragged batch through
:meth:`JetSpecEngine.step` (the engine's own step function, cache and kernels), and finished requests give their pages
and slot-map rows back.  Steps arrive on standard input, one JSON object a line::

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": ["a"]}

For a step with wanted logits ``<out>/<step>.f32`` gets them as little-endian floats ``(wanted, vocab)``; after every
step the line ``done <step>`` is printed.  ``bin/trace_run`` is the command.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

import torch

LIVE_REQUESTS = 4        # slot-map rows of the replay's pool: no more requests are live at any time


class TraceReplay:
    """Drives one engine through the steps of a trace."""

    def __init__(self, engine, max_tokens: int):
        from ..runtime import Scheduler
        self.eng = engine
        pool = engine.reserve_pool(max_tokens, LIVE_REQUESTS)
        self.sched = Scheduler(pool, max_batch_size=LIVE_REQUESTS, prefill_batch_size=LIVE_REQUESTS,
                               admission_evicts=False)
        self.live: dict = {}

    def admit(self, name: str, tokens: list) -> None:
        from ..runtime import SequenceRequest
        sid = self.eng._new_seq_id()
        self.sched.admit_request(SequenceRequest(seq_id=sid, input_ids=list(tokens), max_new_tokens=0))
        self.live[name] = sid

    def step(self, entries: list, end: list):
        """One step; returns the wanted logits ``(wanted, vocab)`` as 32-bit floats, or ``None``."""
        for e in entries:
            if e["id"] not in self.live:
                self.admit(e["id"], e["tokens"])
        if self.sched.waiting_queue:
            out = self.sched.step()
            if self.sched.waiting_queue or out.evicted:
                raise RuntimeError("the pool is too small for the requests of this trace")
        logits = None
        if entries:
            logits = self.eng.step([(self.live[e["id"]], e["tokens"], e.get("want") or []) for e in entries])
        for name in end:
            sid = self.live.pop(name, None)
            if sid is not None:
                self.sched.mark_finished(sid)
        return None if logits is None else logits.float()


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay a trace of token ids and write logits.")
    ap.add_argument("--model", required=True, help="directory with config.json and model.safetensors")
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="directory the logits are written to")
    ap.add_argument("--max-tokens", required=True, type=int, help="most tokens live requests hold at any time")
    ap.add_argument("--device", default="cuda", help="cuda (default), or cpu for the reference ops")
    args = ap.parse_args(argv)
    from .engine import JetSpecEngine
    dtype = getattr(torch, args.dtype)
    torch.set_float32_matmul_precision("highest")          # true 32-bit products, no TF32
    torch.backends.cuda.matmul.allow_tf32 = False
    if args.device != "cpu" and not torch.cuda.is_available():
        raise RuntimeError("no CUDA device")
    eng = JetSpecEngine(args.model, device=args.device, dtype=dtype)
    replay = TraceReplay(eng, args.max_tokens)
    for line in sys.stdin:
        if not line.strip():
            continue
        s = json.loads(line)
        logits = replay.step(s["entries"], s.get("end") or [])
        if logits is not None:
            part = os.path.join(args.out, f".{s['step']}.part")
            logits.cpu().contiguous().numpy().astype("<f4").tofile(part)
            os.replace(part, os.path.join(args.out, f"{s['step']}.f32"))
        elif args.device != "cpu":
            torch.cuda.synchronize()
        print(f"done {s['step']}", flush=True)
    if args.device != "cpu" and eng.use_kernels:
        from ..ops import cuda_ext
        cuda_ext.check_status(eng.device)
    return 0


if __name__ == "__main__":
    sys.exit(main())
