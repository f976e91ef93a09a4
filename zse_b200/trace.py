"""Replays a trace of token ids through a model and writes logits: ``bin/trace_run`` or ``zse trace-run``.

    trace_run --model MODEL --dtype bfloat16|float32 --out DIR --max-tokens N

Steps come from standard input, one JSON object a line:

    {"step": 7, "entries": [{"id": "chat-1", "tokens": [901, 44], "want": [1]}], "end": ["chat-1"]}

An entry continues (or starts) a request by its tokens; ``want`` picks the places among them whose logits the caller needs.
Requests named in ``end`` free their cache blocks once the step has run.  A step is one call of ``ModelRunner.run_batch`` on
the engine's cache, whatever mixture of prompt portions and single tokens it carries.  Its logits go to ``DIR/<step>.f32``
(little-endian fp32, one row of the vocabulary per wanted place), then ``done <step>`` is printed.  No token is chosen.

``--max-tokens`` sizes the cache: the sum of the live requests' tokens at its peak, each counted in whole blocks of 64.
"""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import Dict, List, Optional

import numpy as np

MAX_LIVE = 4            # requests that hold cache blocks at the same time


class TraceRunner:
    def __init__(self, model: str, dtype: str, max_tokens: int, max_live: int = MAX_LIVE, device: Optional[str] = None):
        from .config import EngineConfig
        from .engine import ZStreamerEngine
        block = 64
        tokens = (max(1, max_tokens) + block - 1) // block * block
        self.engine = ZStreamerEngine(model, config=EngineConfig(
            dtype=dtype, device=device, block_size=block, kv_tokens=tokens, max_seq_len=tokens,
            max_batch_seqs=max_live, max_batch_tokens=tokens, prefill_chunk_size=0, logits_rows=tokens,
            enable_prefix_cache=False, state_slots=max_live))
        self._seq: Dict[str, int] = {}
        self._next = 0

    def step(self, entries: List[dict], end: List[str]) -> Optional[np.ndarray]:
        """Runs one step; the wanted logits [wanted, vocab] fp32, or None when nothing is wanted."""
        cache, runner = self.engine.kv_cache, self.engine.runner
        items, want = [], []
        for e in entries:
            rid, toks = str(e["id"]), [int(t) for t in e["tokens"]]
            if not toks:
                continue
            if rid in self._seq:
                sid = self._seq[rid]
                start = cache.num_tokens(sid)
                cache.extend_sequence(sid, len(toks))
            else:
                sid, self._next = self._next, self._next + 1
                cache.allocate_sequence(sid, num_tokens=len(toks))
                cache.mark_active(sid)
                self._seq[rid], start = sid, 0
            items.append((sid, toks, start))
            want.append([int(k) for k in e.get("want", ())])
        out = None
        if items:
            logits = runner.run_batch(items, want)
            if any(want):
                out = np.array(logits.float().cpu().numpy())       # the buffer belongs to the next pass
        for rid in end:
            sid = self._seq.pop(str(rid), None)
            if sid is not None:
                cache.free_sequence(sid)
        return out

    def close(self) -> None:
        self.engine.destroy()


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Feed token ids through a model step by step, write logits")
    ap.add_argument("--model", required=True, help="a .zse file or a model directory")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True)
    ap.add_argument("--max-tokens", type=int, required=True)
    ap.add_argument("--device", default=None, help="'cpu': the plain PyTorch path")
    a = ap.parse_args(argv)
    runner = TraceRunner(a.model, a.dtype, a.max_tokens, device=a.device)
    for line in sys.stdin:
        line = line.strip()
        if not line:
            continue
        s = json.loads(line)
        out = runner.step(s.get("entries", []), s.get("end", []))
        if out is not None:
            tmp = os.path.join(a.out, f"{s['step']}.tmp")
            out.astype("<f4").tofile(tmp)
            os.replace(tmp, os.path.join(a.out, f"{s['step']}.f32"))
        print(f"done {s['step']}", flush=True)
    runner.close()
    return 0


if __name__ == "__main__":
    sys.exit(main())
