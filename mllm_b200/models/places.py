"""Helpers of the designs whose ``config.json`` lists its layers: checks of sizes, and loading by a table of places.

A place is a function that takes a checkpoint tensor and puts it where it belongs; a model gives a table from checkpoint
names to places, and every tensor must have a place and every place a tensor."""

from __future__ import annotations

from typing import Any, Callable, Dict, Iterable, Optional, Tuple

import torch

Places = Dict[str, Callable[[torch.Tensor], Any]]


def require_positive(where: str, sizes: Dict[str, Any], names: Iterable[str]) -> None:
    for n in names:
        if int(sizes.get(n) or 0) <= 0:
            raise ValueError(f"{where}: {n} must be given and positive")


def put(p: torch.Tensor) -> Callable[[torch.Tensor], None]:
    """The place of a whole parameter."""
    def copy(t):
        if t.shape != p.shape:
            raise ValueError(f"a tensor of shape {tuple(t.shape)} does not fit {tuple(p.shape)}")
        p.data.copy_(t)
    return copy


def mixture_places(at: str, block, shared: Optional[torch.nn.Module]) -> Places:
    """Places of a :class:`..layers.moe.SparseMoeBlock` and of a shared gated MLP beside it."""
    gate = block.gate
    out: Places = {at + "router": put(gate.weight[: gate.outputs])}
    if gate.correction is not None:
        out[at + "correction"] = put(gate.correction)
    for e in range(block.num_experts):
        for n in ("gate", "up") if block.gated else ("up",):
            out[f"{at}e{e}.{n}"] = lambda t, e=e, n=n: block.w13.weight_loader(block.w13, t, e, n)
        out[f"{at}e{e}.down"] = lambda t, e=e: block.w2.weight_loader(block.w2, t, e)
    if shared is not None:
        gu, down = shared.gate_up_proj.weight, shared.down_proj.weight
        for j, n in enumerate(("gate", "up")):
            out[f"{at}shared.{n}"] = lambda t, j=j: gu.weight_loader(gu, t, j)
        out[at + "shared.down"] = lambda t: down.weight_loader(down, t)
        if gate.extra:
            out[at + "shared.sg"] = put(gate.weight[gate.outputs:])
    return out


def load_places(places: Places, weights: Iterable[Tuple[str, torch.Tensor]], optional: Iterable[str] = ()) -> set:
    """``optional``: tensors that a checkpoint may lack."""
    loaded = set()
    for name, t in weights:
        place = places.get(name)
        if place is None:
            raise ValueError(f"unexpected tensor {name!r} in the checkpoint")
        place(t.materialize() if hasattr(t, "materialize") else t)
        loaded.add(name)
    missing = sorted(set(places) - loaded - set(optional))
    if missing:
        raise ValueError(f"the checkpoint lacks {len(missing)} tensors: {', '.join(missing[:8])}")
    return loaded
