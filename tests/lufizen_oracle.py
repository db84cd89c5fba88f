"""Plain, slow statement of the Lufizen decoder, one function per mechanism, in float64 on the CPU.

Everything here works on one sequence at a time, token by token or row by row, from a dict of named tensors in
the checkpoint's own layout.  It shares no code with the package: tests compare the package's kernels and
its serving path with it."""

from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

F64 = torch.float64


def f64(t) -> torch.Tensor:
    return t.detach().to("cpu", F64)


def unit_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return unit_rms(x, eps) * w


def sigmoid(z: torch.Tensor) -> torch.Tensor:
    return 1.0 / (1.0 + torch.exp(-z))


def frequencies(dims: int, base: float, scaling: Optional[dict] = None) -> List[float]:
    """One per rotated pair; with ``scaling`` long waves slow down by ``factor``, short ones stay, a ramp between."""
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if scaling is not None:
            wave = 2.0 * math.pi / f
            if wave > scaling["original"] / scaling["low"]:
                f = f / scaling["factor"]
            elif wave >= scaling["original"] / scaling["high"]:
                s = (scaling["original"] / wave - scaling["low"]) / (scaling["high"] - scaling["low"])
                f = (1.0 - s) * f / scaling["factor"] + s * f
        out.append(f)
    return out


def turn(x: torch.Tensor, pos: int, freqs: List[float], first, second) -> torch.Tensor:
    """x [heads, D]: feature ``first(i)`` and feature ``second(i)`` turn by ``pos * freqs[i]``."""
    y = x.clone()
    for i, f in enumerate(freqs):
        c, s, a, b = math.cos(pos * f), math.sin(pos * f), first(i), second(i)
        y[:, a] = x[:, a] * c - x[:, b] * s
        y[:, b] = x[:, b] * c + x[:, a] * s
    return y


def turn_halves(x: torch.Tensor, pos: int, freqs: List[float]) -> torch.Tensor:
    n = len(freqs)
    return turn(x, pos, freqs, lambda i: i, lambda i: i + n)


def turn_neighbours(x: torch.Tensor, pos: int, freqs: List[float]) -> torch.Tensor:
    return turn(x, pos, freqs, lambda i: 2 * i, lambda i: 2 * i + 1)


def softmax_with_sink(s: torch.Tensor, sink: Optional[float]) -> torch.Tensor:
    top = float(s.max()) if sink is None else max(float(s.max()), sink)
    e = torch.exp(s - top)
    return e / (e.sum() + (0.0 if sink is None else math.exp(sink - top)))


def causal_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, sink: Optional[torch.Tensor] = None) -> torch.Tensor:
    """q [T, H, D], k [T, G, D], v [T, G, Dv]; neighbouring query heads share a key / value head."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for i in range(T):
        for a in range(H):
            g = a // (H // G)
            w = softmax_with_sink((k[: i + 1, g] @ q[i, a]) * scale, None if sink is None else float(sink[a]))
            out[i, a] = w @ v[: i + 1, g]
    return out


def tied_qkv(h: torch.Tensor, w: Dict[str, torch.Tensor], pre: str, m: dict, eps: float):
    """(q, k, v): keys and queries turned, then of unit root mean square per head; values are the keys as projected."""
    H, G, D, T = m["heads"], m["kv_heads"], m["dim"], h.shape[0]
    fr = frequencies(m["rot"]["dims"], m["rot"]["base"], m["rot"].get("scaling"))
    q, v = (h @ w[pre + "q"].T).view(T, H, D), (h @ w[pre + "k"].T).view(T, G, D)
    q = unit_rms(torch.stack([turn_halves(q[t], t, fr) for t in range(T)]), eps)
    k = unit_rms(torch.stack([turn_halves(v[t], t, fr) for t in range(T)]), eps)
    return q, k, v


def attention_mixer(h: torch.Tensor, w: Dict[str, torch.Tensor], pre: str, m: dict, eps: float) -> torch.Tensor:
    o = causal_attention(*tied_qkv(h, w, pre, m, eps), m["scale"], w[pre + "sink"])
    return o.reshape(h.shape[0], -1) @ w[pre + "o"].T


def latent_mixer(h: torch.Tensor, w: Dict[str, torch.Tensor], pre: str, m: dict, eps: float) -> torch.Tensor:
    H, D, R, Dv, rank, T = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], h.shape[0]
    fr = frequencies(m["rot"]["dims"], m["rot"]["base"], m["rot"].get("scaling"))
    q = (rms_norm(h @ w[pre + "dq"].T, w[pre + "dq.norm"], eps) @ w[pre + "uq"].T).view(T, H, D + R)
    down = h @ w[pre + "dkv"].T
    c, kr = rms_norm(down[:, :rank], w[pre + "dkv.norm"], eps), down[:, rank:].view(T, 1, R)
    qr = torch.stack([turn_neighbours(q[t, :, D:], t, fr) for t in range(T)])
    kr = torch.stack([turn_neighbours(kr[t], t, fr) for t in range(T)])
    k = torch.cat([(c @ w[pre + "uk"].T).view(T, H, D), kr.expand(T, H, R)], -1)
    v = (c @ w[pre + "uv"].T).view(T, H, Dv)
    o = causal_attention(torch.cat([q[..., :D], qr], -1), k, v, m["scale"])
    o = o * sigmoid(h @ w[pre + "g"].T).unsqueeze(-1)
    return o.reshape(T, H * Dv) @ w[pre + "o"].T


def gated_ff(h: torch.Tensor, w: Dict[str, torch.Tensor], pre: str) -> torch.Tensor:
    g = h @ w[pre + "gate"].T
    return (g * sigmoid(g) * (h @ w[pre + "up"].T)) @ w[pre + "down"].T


def route(logits: torch.Tensor, correction: torch.Tensor, top: int, groups: int, keep: int, scale: float):
    """One token's (chosen experts, their weights)."""
    s = sigmoid(logits)
    choice = [float(v) for v in s + correction]
    size = len(choice) // groups
    rank = [sum(sorted(choice[g * size:(g + 1) * size])[-2:]) for g in range(groups)]
    open_groups = sorted(range(groups), key=lambda g: -rank[g])[:keep]
    allowed = [e for e in range(len(choice)) if e // size in open_groups]
    chosen = sorted(allowed, key=lambda e: -choice[e])[:top]
    return chosen, [float(s[e]) * scale for e in chosen]


def mixture_ff(h: torch.Tensor, w: Dict[str, torch.Tensor], pre: str, mlp: dict) -> torch.Tensor:
    r = mlp["router"]
    groups = r.get("groups") or dict(count=1, keep=1)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, g in zip(*route(w[pre + "router"] @ h[t], w[pre + "correction"], r["top"], groups["count"], groups["keep"], r["scale"])):
            out[t] += g * gated_ff(h[t], w, f"{pre}e{e}.")
    if mlp.get("shared") is not None:
        out = out + sigmoid(h @ w[pre + "shared.sg"].T) * gated_ff(h, w, pre + "shared.")
    return out


def forward(cfg: dict, weights: Dict[str, torch.Tensor], tokens: List[int], layer_out: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence; ``layer_out`` collects the residual stream after every layer."""
    w = {n: f64(t) for n, t in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"]
    for i, layer in enumerate(cfg["layers"]):
        pre = f"l{i}."
        mixer = latent_mixer if layer["type"] == "latent_attention" else attention_mixer
        x = x + rms_norm(mixer(x, w, pre + "mix.", layer["mixer"], eps), w[pre + "norm1"], eps)
        if layer.get("mlp") is not None:
            x = x + rms_norm(mixture_ff(x, w, pre + "mlp.", layer["mlp"]), w[pre + "norm2"], eps)
        if layer_out is not None:
            layer_out.append(x.clone())
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T * cfg["logit_scale"]
