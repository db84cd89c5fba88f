"""Plain, slow statement of the Nikedra decoder, one function per mechanism, in float64 on the CPU.

Everything here works on one sequence at a time, token by token or row by row, from a dict of named tensors in
the checkpoint's own layout.  It shares no code with the package: tests compare the package's kernels and
its serving path with it."""

from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

F64 = torch.float64
Tensors = Dict[str, torch.Tensor]


def f64(t) -> torch.Tensor:
    return t.detach().to("cpu", F64)


def unit_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def sigmoid(z: torch.Tensor) -> torch.Tensor:
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * sigmoid(z)


def softplus(z: torch.Tensor) -> torch.Tensor:
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


# ---------------------------------------------------------------------------------------------- time
def causal_conv(x: torch.Tensor, w: torch.Tensor, bias: Optional[torch.Tensor] = None) -> torch.Tensor:
    """x [T, C], w [C, K]: column K - 1 meets the current token, column 0 the one K - 1 before it."""
    T, C = x.shape
    K = w.shape[1]
    out = torch.zeros(T, C, dtype=F64)
    for t in range(T):
        for back in range(min(K, t + 1)):
            out[t] += w[:, K - 1 - back] * x[t - back]
        if bias is not None:
            out[t] += bias
    return out


# ---------------------------------------------------------------------------------------------- rotation
def frequencies(dims: int, base: float, scaling: Optional[dict] = None) -> List[float]:
    """One per rotated pair; with ``scaling`` slow pairs are divided by ``factor``, fast ones stay, a ramp between."""
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if scaling is not None:
            def pair_of(turns):                 # the pair that turns this often over the original length
                return dims * math.log(scaling["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

            lo = max(math.floor(pair_of(scaling["fast"])), 0)
            hi = min(math.ceil(pair_of(scaling["slow"])), dims - 1)
            ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
            f = f / scaling["factor"] * ramp + f * (1.0 - ramp)
        out.append(f)
    return out


def turn_halves(x: torch.Tensor, freqs: List[float], magnitude: float = 1.0) -> torch.Tensor:
    """x [T, heads, D]: features i and i + len(freqs) of the token at position t turn by t * freqs[i]."""
    y, n = x.clone(), len(freqs)
    for t in range(x.shape[0]):
        for i, f in enumerate(freqs):
            c, s = math.cos(t * f) * magnitude, math.sin(t * f) * magnitude
            y[t, :, i] = x[t, :, i] * c - x[t, :, i + n] * s
            y[t, :, i + n] = x[t, :, i + n] * c + x[t, :, i] * s
    return y


# ---------------------------------------------------------------------------------------------- attention
def attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, first) -> torch.Tensor:
    """q [T, H, D], k [T, G, D], v [T, G, Dv]; token i sees first(i) .. i; neighbouring query heads share a key head."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for i in range(T):
        a = first(i)
        for h in range(H):
            g = h // (H // G)
            out[i, h] = torch.softmax((k[a: i + 1, g] @ q[i, h]) * scale, 0) @ v[a: i + 1, g]
    return out


def chunk_attention(h: torch.Tensor, w: Tensors, pre: str, m: dict) -> torch.Tensor:
    """Rotated grouped-query attention inside chunks of positions, a gate per head, the output projection."""
    T, H, G, D, Dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    rot = m["rot"]
    scaling = rot.get("scaling")
    fr = frequencies(rot["dims"], rot["base"], scaling)
    mag = 1.0 if scaling is None else 0.1 * math.log(scaling["factor"]) + 1.0
    q = turn_halves((h @ w[pre + "q"].T).view(T, H, D), fr, mag)
    k = turn_halves((h @ w[pre + "k"].T).view(T, G, D), fr, mag)
    v = (h @ w[pre + "v"].T).view(T, G, Dv)
    size = m["mask"]["size"]
    o = attention(q, k, v, m["scale"], lambda i: i // size * size)
    o = o * sigmoid(h @ w[pre + "g"].T).unsqueeze(-1)
    return o.reshape(T, H * Dv) @ w[pre + "o"].T


def latent_mixer(h: torch.Tensor, w: Tensors, pre: str, m: dict, eps: float) -> torch.Tensor:
    """Latent attention over the last positions, a gate per feature."""
    T, H, D, R, Dv, rank = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    fr = frequencies(m["rot"]["dims"], m["rot"]["base"], m["rot"].get("scaling"))
    q = (h @ w[pre + "q"].T).view(T, H, D + R)
    down = h @ w[pre + "dkv"].T
    c = unit_rms(down[:, :rank], eps) * w[pre + "dkv.norm"]
    q = torch.cat([q[..., :D], turn_halves(q[..., D:], fr)], -1)
    shared = turn_halves(down[:, rank:].view(T, 1, R), fr)
    k = torch.cat([(c @ w[pre + "uk"].T).view(T, H, D), shared.expand(T, H, R)], -1)
    v = (c @ w[pre + "uv"].T).view(T, H, Dv)
    size = m["mask"]["size"]
    o = attention(q, k, v, m["scale"], lambda i: max(0, i - size + 1)).reshape(T, H * Dv)
    return (o * sigmoid(h @ w[pre + "g"].T)) @ w[pre + "o"].T


# ---------------------------------------------------------------------------------------------- recurrences
def channel_delta_rule(q, k, v, g, beta) -> torch.Tensor:
    """One head: q, k [T, D] as projected, v [T, Dv], g [T, D] log decays of the key channels, beta [T]."""
    T, D = q.shape
    S = torch.zeros(D, v.shape[1], dtype=F64)
    out = torch.zeros(T, v.shape[1], dtype=F64)
    for t in range(T):
        qt = q[t] / torch.sqrt((q[t] * q[t]).sum() + 1e-6) * D ** -0.5
        kt = k[t] / torch.sqrt((k[t] * k[t]).sum() + 1e-6)
        S = torch.exp(g[t]).unsqueeze(1) * S
        u = beta[t] * (v[t] - S.T @ kt)
        S = S + torch.outer(kt, u)
        out[t] = S.T @ qt
    return out


def channel_delta_mixer(h: torch.Tensor, w: Tensors, pre: str, m: dict, eps: float) -> torch.Tensor:
    T, H, G, D, Dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]

    def projected(n, heads, dim):
        return silu(causal_conv(h @ w[pre + n].T, w[f"{pre}{n}.conv"])).view(T, heads, dim)

    q, k, v = projected("q", G, D), projected("k", G, D), projected("v", H, Dv)
    beta = sigmoid(h @ w[pre + "b"].T)
    a = ((h @ w[pre + "a1"].T) @ w[pre + "a2"].T + w[pre + "dt_bias"]).view(T, H, D)
    g = -torch.exp(w[pre + "A_log"]).view(1, H, 1) * softplus(a)
    gate = sigmoid((h @ w[pre + "g1"].T) @ w[pre + "g2"].T).view(T, H, Dv)
    o = torch.zeros(T, H, Dv, dtype=F64)
    for a_ in range(H):
        b_ = a_ // (H // G)
        o[:, a_] = channel_delta_rule(q[:, b_], k[:, b_], v[:, a_], g[:, a_], beta[:, a_])
    o = unit_rms(o, eps) * w[pre + "norm"] * gate
    return o.reshape(T, H * Dv) @ w[pre + "o"].T


def state_space_rule(x, B, C, dt, a_log: float, D: float) -> torch.Tensor:
    """One head: x [T, P], B and C [T, N], dt [T] positive step sizes."""
    S = torch.zeros(B.shape[1], x.shape[1], dtype=F64)
    out = torch.zeros_like(x)
    for t in range(x.shape[0]):
        S = math.exp(-math.exp(a_log) * float(dt[t])) * S + dt[t] * torch.outer(B[t], x[t])
        out[t] = S.T @ C[t] + D * x[t]
    return out


def state_space_mixer(h: torch.Tensor, w: Tensors, pre: str, m: dict, eps: float) -> torch.Tensor:
    T, H, P, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    row = h @ w[pre + "in"].T
    z, xbc, dt = row[:, :inner], row[:, inner: 2 * inner + 2 * G * N], row[:, 2 * inner + 2 * G * N:]
    xbc = silu(causal_conv(xbc, w[pre + "conv"], w[pre + "conv.b"]))
    x, B, C = xbc[:, :inner].view(T, H, P), xbc[:, inner: inner + G * N].view(T, G, N), xbc[:, inner + G * N:].view(T, G, N)
    dt = softplus(dt + w[pre + "dt_bias"])
    y = torch.zeros(T, H, P, dtype=F64)
    for a in range(H):
        g = a // (H // G)
        y[:, a] = state_space_rule(x[:, a], B[:, g], C[:, g], dt[:, a], float(w[pre + "A_log"][a]), float(w[pre + "D"][a]))
    y = (y.reshape(T, inner) * silu(z)).view(T, m["norm_groups"], -1)
    return (unit_rms(y, eps).reshape(T, inner) * w[pre + "norm"]) @ w[pre + "o"].T


def parallel_mixer(h: torch.Tensor, w: Tensors, pre: str, m: dict, eps: float) -> torch.Tensor:
    left = unit_rms(chunk_attention(h, w, pre + "left.", m["left"]), eps) * w[pre + "left.out"]
    right = unit_rms(state_space_mixer(h, w, pre + "right.", m["right"], eps), eps) * w[pre + "right.out"]
    return 0.5 * (left + right)


# ---------------------------------------------------------------------------------------------- feed-forward
def clamped_ff(h: torch.Tensor, w: Tensors, pre: str, limit: float) -> torch.Tensor:
    g = torch.clamp(h @ w[pre + "gate"].T + w[pre + "gate.b"], max=limit)
    u = torch.clamp(h @ w[pre + "up"].T + w[pre + "up.b"], min=-limit, max=limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ w[pre + "down"].T + w[pre + "down.b"]


def gelu(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def mixture_ff(h: torch.Tensor, w: Tensors, pre: str, router: dict) -> torch.Tensor:
    """The weight of a chosen expert scales what it reads."""
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        s = sigmoid(w[pre + "router"] @ h[t])
        for e in sorted(range(router["experts"]), key=lambda e: -float(s[e]))[: router["top"]]:
            out[t] += w[f"{pre}e{e}.down"] @ gelu(w[f"{pre}e{e}.up"] @ (s[e] * h[t]))
    return out


# ---------------------------------------------------------------------------------------------- the model
def depth_average(w: torch.Tensor, results: List[torch.Tensor]) -> torch.Tensor:
    return sum(w[j] * r for j, r in enumerate(results))


def forward(cfg: dict, weights: Tensors, tokens: List[int], layer_out: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence; ``layer_out`` collects what every layer hands on."""
    w = {n: f64(t) for n, t in weights.items()}
    eps = cfg["norm"]["eps"]
    x = unit_rms(w["embed"][torch.tensor(tokens)], eps) * w["embed.norm"]
    results = [x]
    for i, layer in enumerate(cfg["layers"]):
        pre, m = f"l{i}.", layer["mixer"]
        h = unit_rms(x, eps) * w[pre + "norm1"]
        h = h + causal_conv(h, w[pre + "canon1"])
        mixer = dict(latent_attention=latent_mixer, channel_delta=channel_delta_mixer, parallel=parallel_mixer)[layer["type"]]
        y = mixer(h, w, pre + "mix.", m, eps)
        mlp = layer.get("mlp")
        if mlp is not None:
            h2 = unit_rms(x, eps) * w[pre + "norm2"]
            y = y + (clamped_ff(h2, w, pre + "mlp.", mlp["limit"]) if mlp["kind"] == "dense" else
                     mixture_ff(h2, w, pre + "mlp.", mlp["router"]))
        results.append(x + y)
        x = depth_average(w[pre + "dwa"], results)
        if layer_out is not None:
            layer_out.append(x.clone())
    return (unit_rms(x, eps) * w["final.norm"]) @ w["head"].T * cfg["logit_scale"]
