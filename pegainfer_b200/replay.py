"""Replay a trace: given token ids go through an engine step by step, and logits come out; nothing is sampled.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps.jsonl

Each input line is one step, ``{"step": n, "entries": [{"id": ..., "tokens": [...], "want": [...]}, ...], "end": [...]}``:
the next tokens of some requests, the places among them whose logits are wanted, and the requests that are finished after
the step.  The entries of a step are one ragged batch of the engine's executor, prompt portions in front of single tokens as
the scheduler lists them; a step of single tokens replays the decode graph.  The logits at the wanted places go to
``DIR/<step>.f32`` (little-endian f32, entries in the order given), then ``done <step>`` is printed.

The KV pool holds ``--max-tokens`` tokens and there are state slots for ``--max-requests`` live requests, so pages and
slots are used again as requests end.  ``--dtype float32`` exits with code 3 on a line without 32-bit kernels.
"""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import Optional

PAGE = 16


class Replayer:
    """Feeds steps to an engine's executor with the engine's own pool, request bookkeeping and state slots."""

    def __init__(self, engine):
        self.ex, self.pool = engine.executor, engine.pool
        self.live: dict = {}  # request id -> (executor request id, RequestKv)
        self._next = 0

    def step(self, entries):
        """One batch; ``entries``: ``(id, tokens, want)``.  Returns f32 logits ``[wanted, vocab]`` in the order of the
        entries, or ``None``."""
        import torch

        from .kv.request_kv import RequestKv
        from .sched.executor import SeqStep, StepBatch

        seqs = []
        for rid, tokens, _ in entries:
            if rid not in self.live:
                self.live[rid] = (self._next, RequestKv(self.pool, []))
                self._next += 1
            num, kv = self.live[rid]
            start = kv.committed
            kv.extend_prompt(tokens)
            kv.schedule_prefill(len(tokens))
            seqs.append(SeqStep(rid=num, input_tokens=list(tokens), start_pos=start, view=kv.view(), fresh_state=start == 0))
        order = sorted(range(len(entries)), key=lambda i: len(entries[i][1]) == 1)  # portions first, stable
        batch = StepBatch([seqs[i] for i in order], kind="decode" if all(len(e[1]) == 1 for e in entries) else "unified")
        logits = self.ex.step_logits(batch, [entries[i][2] for i in order])
        for rid, _, _ in entries:
            self.live[rid][1].apply_prefill_chunk()
        if logits is None:
            return None
        first, n = {}, 0
        for i in order:
            first[i] = n
            n += len(entries[i][2])
        back = [first[i] + j for i in range(len(entries)) for j in range(len(entries[i][2]))]
        return logits.float()[torch.tensor(back, device=logits.device)]

    def end(self, rid) -> None:
        num, kv = self.live.pop(rid)
        kv.release()
        self.ex.release_request(num)


def open_engine(model: str, dtype: str, max_tokens: int, max_requests: int, device: Optional[str] = None):
    """An engine of that many tokens of KV pool and that many state slots (no scheduler thread)."""
    import torch

    from .config import EngineConfig, load_model_config
    from .engine.build import build_engine

    mcfg = load_model_config(model)
    ecfg = EngineConfig(model_path=model, kv_page_size=PAGE, num_kv_blocks=(max_tokens + PAGE - 1) // PAGE + 1, max_decode_batch=max_requests, state_slots=max_requests,
                        no_prefix_cache=True, run_ahead=False, dtype=dtype, max_model_len=min(mcfg.max_position, max(max_tokens, 2)))
    return build_engine(ecfg, mcfg, device=device, dtype=getattr(torch, dtype), start=False)


def main(argv: Optional[list] = None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="replay given tokens through a model and write logits")
    ap.add_argument("--model", required=True, help="directory with config.json and safetensors")
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    ap.add_argument("--out", required=True, help="directory for <step>.f32")
    ap.add_argument("--max-tokens", type=int, required=True, help="tokens that live requests hold at most")
    ap.add_argument("--max-requests", type=int, default=4, help="requests live at a time")
    ap.add_argument("--device", default=None, help="default: the first GPU")
    a = ap.parse_args(argv)

    from . import _native
    from .config import load_model_config
    from .engine.build import F32_FAMILIES
    from .models.registry import kernel_units

    family = load_model_config(a.model).family
    if a.dtype == "float32" and family not in F32_FAMILIES:
        print(f"the {family} line has no 32-bit kernels", file=sys.stderr)
        return 3
    import torch

    device = a.device or "cuda:0"
    if device.startswith("cuda"):
        if not torch.cuda.is_available():
            print("no GPU", file=sys.stderr)
            return 1
        _native.use_units(kernel_units(family))
    replay = Replayer(open_engine(a.model, a.dtype, a.max_tokens, a.max_requests, device))
    for line in sys.stdin:
        if not line.strip():
            continue
        s = json.loads(line)
        logits = replay.step([(e["id"], e["tokens"], e.get("want", [])) for e in s["entries"]]) if s["entries"] else None
        if logits is not None:
            logits.cpu().numpy().astype("<f4").tofile(os.path.join(a.out, f"{s['step']}.f32"))
        for rid in s.get("end", []):
            replay.end(rid)
        print(f"done {s['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
