"""Schedules that feed sequences to a serving session in different ways; all must give the logits of one pass."""

from __future__ import annotations

from typing import Dict, List

import torch


def cut(n: int, sizes: List[int]) -> List[int]:
    out, k = [], 0
    while n > 0:
        out.append(min(n, sizes[k % len(sizes)]))
        n -= out[-1]
        k += 1
    return out


def run_alone(session, seq: List[int], portions: List[int]) -> torch.Tensor:
    """One request fed in the given portions; logits of every position."""
    rows, at = [], 0
    for n in portions:
        end = ["r"] if at + n == len(seq) else []
        rows.append(session.step([dict(id="r", tokens=seq[at:at + n], want=list(range(n)))], end))
        at += n
    return torch.cat([r.float().cpu() for r in rows])


def run_together(session, seqs: Dict[str, List[int]], portions: Dict[str, List[int]], start: Dict[str, int], live: int = 4
                 ) -> Dict[str, torch.Tensor]:
    """Requests join at step ``start[id]`` (later when ``live`` are running), each cut its own way; every step is one
    batch.  Logits of every position of every request."""
    at = {i: 0 for i in seqs}
    got: Dict[str, list] = {i: [] for i in seqs}
    left = {i: list(p) for i, p in portions.items()}
    running: List[str] = []
    step = 0
    while any(left.values()):
        for i in seqs:
            if i not in running and left[i] and start[i] <= step and len(running) < live:
                running.append(i)
        entries, end, order = [], [], []
        for i in running:
            n = left[i].pop(0)
            entries.append(dict(id=i, tokens=seqs[i][at[i]:at[i] + n], want=list(range(n))))
            order.append((i, n))
            at[i] += n
            if not left[i]:
                end.append(i)
        step += 1
        if not entries:
            continue
        out = session.step(entries, end).float().cpu()
        running = [i for i in running if i not in end]
        row = 0
        for i, n in order:
            got[i].append(out[row:row + n])
            row += n
    return {i: torch.cat(v) for i, v in got.items()}
