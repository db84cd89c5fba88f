"""Plain, slow statement of the Kesovik decoder, one function per mechanism, in float64 on the CPU.

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


def rms_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def sigmoid(z: torch.Tensor) -> torch.Tensor:
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * sigmoid(z)


def relu_squared(z: torch.Tensor) -> torch.Tensor:
    return torch.clamp(z, min=0.0) ** 2


def rotate_pairs(x: torch.Tensor, pos: int, dims: int, base: float) -> torch.Tensor:
    """x [heads, D] of the token at ``pos``: neighbours (2i, 2i + 1) below ``dims`` turn by pos * base^(-2i / dims)."""
    y = x.clone()
    for i in range(dims // 2):
        a = pos * base ** (-2.0 * i / dims)
        u, v = x[:, 2 * i], x[:, 2 * i + 1]
        y[:, 2 * i] = u * math.cos(a) - v * math.sin(a)
        y[:, 2 * i + 1] = v * math.cos(a) + u * math.sin(a)
    return y


def window_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, window: int) -> torch.Tensor:
    """q [T, H, D], k [T, G, D], v [T, G, Dv]: token i sees itself and the ``window - 1`` tokens before it."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for i in range(T):
        lo = max(0, i - window + 1)
        for a in range(H):
            g = a // (H // G)
            s = (k[lo: i + 1, g] @ q[i, a]) * scale
            e = torch.exp(s - s.max())
            out[i, a] = (e / e.sum()) @ v[lo: i + 1, g]
    return out


def attention_mixer(h: torch.Tensor, w: Dict[str, torch.Tensor], pre: str, m: dict, eps: float) -> torch.Tensor:
    H, G, D, Dv, T = m["heads"], m["kv_heads"], m["dim"], m["vdim"], h.shape[0]
    q, k, v = (h @ w[pre + n].T + w[pre + n + ".b"] for n in ("q", "k", "v"))
    q = rms_norm(q, w[pre + "q.norm"], eps).view(T, H, D)       # over all heads at once
    k = rms_norm(k, w[pre + "k.norm"], eps).view(T, G, D)
    dims, base = m["rot"]["dims"], m["rot"]["base"]
    q = torch.stack([rotate_pairs(q[t], t, dims, base) for t in range(T)])
    k = torch.stack([rotate_pairs(k[t], t, dims, base) for t in range(T)])
    o = window_attention(q, k, v.view(T, G, Dv), m["scale"], m["mask"]["size"])
    return o.reshape(T, H * Dv) @ w[pre + "o"].T


def decayed_sums(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, decay, state: Optional[torch.Tensor] = None):
    """q, k [T, H, D], v [T, H, Dv]: per head S <- decay S + k v^T, o = S^T q; (o, S after the last token)."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[2], dtype=F64) if state is None else state.clone()
    o = torch.zeros(T, H, v.shape[2], dtype=F64)
    for t in range(T):
        for a in range(H):
            S[a] = float(decay[a]) * S[a] + torch.outer(k[t, a], v[t, a])
            o[t, a] = S[a].T @ q[t, a]
    return o, S


def lightning_mixer(h: torch.Tensor, w: Dict[str, torch.Tensor], pre: str, m: dict, eps: float) -> torch.Tensor:
    H, D, Dv, T = m["heads"], m["dim"], m["vdim"], h.shape[0]
    q, k, v = (silu(h @ w[pre + n].T) for n in ("q", "k", "v"))
    o, _ = decayed_sums(q.view(T, H, D), k.view(T, H, D), v.view(T, H, Dv), m["decay"])
    o = rms_norm(o.reshape(T, H * Dv), w[pre + "norm"], eps) * sigmoid(h @ w[pre + "g"].T)
    return o @ w[pre + "o"].T


def parallel_mixer(h: torch.Tensor, w: Dict[str, torch.Tensor], pre: str, m: dict, eps: float) -> torch.Tensor:
    return (m["left_scale"] * attention_mixer(h, w, pre + "left.", m["left"], eps)
            + m["right_scale"] * lightning_mixer(h, w, pre + "right.", m["right"], eps))


def dense_ff(h: torch.Tensor, w: Dict[str, torch.Tensor], pre: str) -> torch.Tensor:
    return relu_squared(h @ w[pre + "up"].T) @ w[pre + "down"].T


def gated_ff(h: torch.Tensor, w: Dict[str, torch.Tensor], pre: str) -> torch.Tensor:
    return (silu(h @ w[pre + "gate"].T) * (h @ w[pre + "up"].T)) @ w[pre + "down"].T


def route(logits: torch.Tensor, correction: torch.Tensor, top: int):
    """One token's (chosen outputs, their weights): chosen by softmax + correction, weighted by the softmax alone."""
    e = torch.exp(logits - logits.max())
    s = e / e.sum()
    chosen = sorted(range(len(s)), key=lambda j: -float(s[j] + correction[j]))[:top]
    total = sum(float(s[j]) for j in chosen) + 1e-20
    return chosen, [float(s[j]) / total for j in chosen]


def mixture_ff(h: torch.Tensor, w: Dict[str, torch.Tensor], pre: str, mlp: dict) -> torch.Tensor:
    r = mlp["router"]
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for j, g in zip(*route(w[pre + "router"] @ h[t], w[pre + "correction"], r["top"])):
            out[t] += g * (gated_ff(h[t], w, f"{pre}e{j}.") if j < r["experts"] else h[t])
    if mlp.get("shared") is not None:
        out = out + gated_ff(h, w, pre + "shared.")
    return out


def capped(z: torch.Tensor, cap: float) -> torch.Tensor:
    return cap * torch.tanh(z / cap)


def forward(cfg: dict, weights: Dict[str, torch.Tensor], tokens: List[int], layer_out: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence; ``layer_out`` collects the residual stream after every layer."""
    w = {n: f64(t) for n, t in weights.items()}
    eps, alpha = cfg["norm"]["eps"], cfg["postln_alpha"]
    x = w["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"]
    for i, layer in enumerate(cfg["layers"]):
        pre = f"l{i}."
        mixer = parallel_mixer if layer["type"] == "parallel" else lightning_mixer
        y = mixer(x, w, pre + "mix.", layer["mixer"], eps)
        x = rms_norm(alpha * x + w[pre + "ls1"] * y, w[pre + "norm1"], eps)
        mlp = layer.get("mlp")
        if mlp is not None:
            y = dense_ff(x, w, pre + "mlp.") if mlp["kind"] == "dense" else mixture_ff(x, w, pre + "mlp.", mlp)
            x = rms_norm(alpha * x + w[pre + "ls2"] * y, w[pre + "norm2"], eps)
        if layer_out is not None:
            layer_out.append(x.clone())
    return capped(rms_norm(x, w["final.norm"], eps) @ w["head"].T, cfg["logit_softcap"])
