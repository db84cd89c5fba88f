"""Plain, slow statement of the Pebulix decoder, one function per mechanism, in float64 on the CPU.

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


def dyt(x: torch.Tensor, alpha: torch.Tensor, w: torch.Tensor, b: torch.Tensor) -> torch.Tensor:
    """Dynamic Tanh: no statistic of the row is taken."""
    return torch.tanh(alpha * x) * w + b


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z: torch.Tensor) -> torch.Tensor:
    return z / (1.0 + torch.exp(-z))


def softplus(z: torch.Tensor) -> torch.Tensor:
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def sink_softmax(scores: torch.Tensor, sink: float) -> torch.Tensor:
    """Weights of a row of scores when one more term, exp(sink), stands in the denominator."""
    top = max(float(scores.max()), float(sink))
    e = torch.exp(scores - top)
    return e / (e.sum() + math.exp(float(sink) - top))


def geglu(h: torch.Tensor, w: Dict[str, torch.Tensor], pre: str) -> torch.Tensor:
    return (gelu_tanh(h @ w[pre + "gate"].T) * (h @ w[pre + "up"].T)) @ w[pre + "down"].T


def latent_rows(h: torch.Tensor, w: Dict[str, torch.Tensor], pre: str, eps: float) -> torch.Tensor:
    return rms_norm(h @ w[pre + "dkv"].T, w[pre + "dkv.norm"], eps)


def latent_attention(h: torch.Tensor, c: torch.Tensor, w: Dict[str, torch.Tensor], pre: str, m: dict, eps: float) -> torch.Tensor:
    """h [T, width] the mixer's input of the whole sequence, c [T, rank] the latents it attends to."""
    H, D, Dv = m["heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q = (rms_norm(h @ w[pre + "dq"].T, w[pre + "dq.norm"], eps) @ w[pre + "uq"].T).view(T, H, D)
    k = (c @ w[pre + "uk"].T).view(T, H, D)
    v = (c @ w[pre + "uv"].T).view(T, H, Dv)
    out = torch.zeros(T, H, Dv, dtype=F64)
    for i in range(T):
        for a in range(H):
            p = sink_softmax((k[: i + 1, a] @ q[i, a]) * m["scale"], float(w[pre + "sink"][a]))
            out[i, a] = p @ v[: i + 1, a]
    return out.reshape(T, H * Dv) @ w[pre + "o"].T


def short_conv(x: torch.Tensor, taps: torch.Tensor) -> torch.Tensor:
    """Causal depth-wise convolution: the last column of ``taps`` meets the current token."""
    T, K = x.shape[0], taps.shape[1]
    y = torch.zeros_like(x)
    for t in range(T):
        for j in range(K):
            s = t - (K - 1) + j
            if s >= 0:
                y[t] += taps[:, j] * x[s]
    return y


def delta_states(q, k, v, g, beta):
    """q, k [T, H, D] (unit keys, scaled unit queries), v [T, H, Dv], g decay factors and beta [T, H] -> (o, S)."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[2], dtype=F64)
    o = torch.zeros(T, H, v.shape[2], dtype=F64)
    for t in range(T):
        for h in range(H):
            S[h] = g[t, h] * S[h]
            u = beta[t, h] * (v[t, h] - S[h].T @ k[t, h])
            S[h] = S[h] + torch.outer(k[t, h], u)
            o[t, h] = S[h].T @ q[t, h]
    return o, S


def delta_mixer(h: torch.Tensor, w: Dict[str, torch.Tensor], pre: str, m: dict, eps: float) -> torch.Tensor:
    H, Hk, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    q, k, v = (silu(short_conv(h @ w[pre + n].T, w[pre + n + ".conv"])) for n in ("q", "k", "v"))
    q, k, v = q.view(T, Hk, D), k.view(T, Hk, D), v.view(T, H, Dv)
    q = q / torch.sqrt((q * q).sum(-1, keepdim=True) + 1e-6) * D ** -0.5
    k = k / torch.sqrt((k * k).sum(-1, keepdim=True) + 1e-6)
    own = [a // (H // Hk) for a in range(H)]
    beta = 1.0 / (1.0 + torch.exp(-(h @ w[pre + "b"].T)))
    g = torch.exp(-torch.exp(w[pre + "A_log"]) * softplus(h @ w[pre + "a"].T + w[pre + "dt_bias"]))
    o, _ = delta_states(q[:, own], k[:, own], v, g, beta)
    o = rms_norm(o, w[pre + "norm"], eps) * silu(h @ w[pre + "g"].T).view(T, H, Dv)
    return o.reshape(T, H * Dv) @ w[pre + "o"].T


def forward(cfg: dict, weights: Dict[str, torch.Tensor], tokens: List[int], layer_out: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence; ``layer_out`` collects the residual stream after every layer."""
    w = {n: f64(t) for n, t in weights.items()}
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]

    def norm(x, name):
        return dyt(x, w[name + ".alpha"], w[name], w[name + ".b"])

    x = w["embed"][torch.tensor(tokens)]
    latents: Dict[int, torch.Tensor] = {}
    for i, layer in enumerate(cfg["layers"]):
        pre, m = f"l{i}.", layer["mixer"]
        h = norm(x, pre + "norm1")
        if layer["type"] == "latent_attention":
            if m.get("kv_from") is None:
                latents[i] = latent_rows(h, w, pre + "mix.", eps)
            y = latent_attention(h, latents[i if m.get("kv_from") is None else m["kv_from"]], w, pre + "mix.", m, eps)
        else:
            y = delta_mixer(h, w, pre + "mix.", m, eps)
        x = x + mult * y
        if layer["mlp"] is not None:
            x = x + mult * geglu(norm(x, pre + "norm2"), w, pre + "mlp.")
        if layer_out is not None:
            layer_out.append(x.clone())
    return norm(x, "final.norm") @ w["embed"].T
