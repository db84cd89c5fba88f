"""Replays given token ids step by step and writes the logits at chosen places.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N  < steps.jsonl

Every line of standard input is one step, ``{"step": n, "entries": [{"id", "tokens", "want"}, ...], "end": [ids]}``:
the next tokens of some requests and the places among them whose logits are wanted, then the requests that are
finished.  A step is one batch of the serving path — the same :class:`ModelRunnerProcess` passes, pools and kernels
that the scheduler drives: a pass of single tokens of running requests is the decode step (captured graphs), anything
else is an extend batch.  Only the sampling is left out.  Logits go to ``DIR/<step>.f32`` (little-endian fp32,
[wanted, vocab], in the order of the entries); ``done <step>`` is printed after every step."""

from __future__ import annotations

import argparse
import json
import os
import sys
from typing import Any, Dict, List, Optional

import torch

MAX_LIVE = 4      # requests that may be live at a time


class TraceSession:
    """Feeds steps to a :class:`ModelRunnerProcess`."""

    def __init__(self, mrp) -> None:
        self.mrp = mrp
        self.live: Dict[str, Any] = {}

    def step(self, entries: List[dict], end: List[str]) -> Optional[torch.Tensor]:
        """Runs one batch; logits [wanted, vocab] or None when nothing is wanted."""
        from .engine.sampling_params import SamplingParams
        from .orchestrator.model_runner_process import Req

        vocab = self.mrp.runner.vocab_size
        items, rows, base, seen = [], [], 0, set()
        for e in entries:
            tokens, want = list(e["tokens"]), list(e.get("want") or [])
            if not tokens or min(tokens) < 0 or max(tokens) >= vocab:
                raise ValueError(f"request {e['id']!r}: token ids must lie in 0..{vocab - 1}, at least one a step")
            if e["id"] in seen or any(not 0 <= w < len(tokens) for w in want):
                raise ValueError(f"request {e['id']!r}: one entry a step, wanted places inside its tokens")
            seen.add(e["id"])
            req = self.live.get(e["id"])
            if req is None:
                req = Req(rid=e["id"], input_ids=tokens, sampling=SamplingParams())
                self.mrp.admit(req)
                self.live[e["id"]] = req
            else:
                req.input_ids.extend(tokens)
            items.append((req, len(tokens)))
            rows.extend(base + w for w in want)
            base += len(tokens)
        logits = None
        if items and all(n == 1 and req.num_computed > 0 for req, n in items):
            out = self.mrp.decode_logits([req for req, _ in items])
            if rows:
                logits = out.index_select(0, torch.tensor(rows, device=out.device))
        elif items:
            out = self.mrp.extend_logits(items, rows or None)
            logits = out if rows else None
        for rid in end:
            self.mrp.release(self.live.pop(rid), cache=False)
        return logits


def build_session(model: str, dtype: str, max_tokens: int, device: Optional[str] = None, **server) -> TraceSession:
    from .configs import ServerConfig
    from .executor import ModelRunner
    from .orchestrator.model_runner_process import ModelRunnerProcess

    # a pool of max_tokens, a request table (and state rows) for MAX_LIVE requests, and no prefix reuse: every token
    # that is fed is computed
    cfg = ServerConfig(model_path=model, dtype=dtype, max_total_tokens=max_tokens, context_length=max_tokens,
                       max_running_requests=MAX_LIVE, spare_request_slots=0, disable_radix_cache=True, **server)
    runner = ModelRunner(cfg, device=device)
    runner.initialize()
    return TraceSession(ModelRunnerProcess(runner, disable_radix_cache=True))


def main(argv: Optional[List[str]] = None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay token ids through a model and write logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and the weights")
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], required=True)
    ap.add_argument("--out", required=True, help="folder for <step>.f32 files")
    ap.add_argument("--max-tokens", type=int, required=True, help="tokens the cache pool holds")
    a = ap.parse_args(argv)
    if not torch.cuda.is_available():
        print("trace_run needs a GPU", file=sys.stderr)
        return 1
    from . import ops

    session = build_session(a.model, a.dtype, a.max_tokens)
    for line in sys.stdin:
        if not line.strip():
            continue
        s = json.loads(line)
        logits = session.step(s.get("entries", []), s.get("end", []))
        ops.check_status()
        if logits is not None:
            path = os.path.join(a.out, f"{int(s['step'])}.f32")
            logits.float().cpu().contiguous().numpy().astype("<f4", copy=False).tofile(path)
        print(f"done {int(s['step'])}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
