"""Small Nikedra configurations with seeded random weights, in the checkpoint's layout, for the tests."""

from __future__ import annotations

import json
from typing import Dict, List, Optional, Tuple

import torch


def delta(heads, kv_heads, dim, vdim, conv=4, mlp=None) -> dict:
    return dict(type="channel_delta", mixer=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv), mlp=mlp)


def latent(heads, dim, rot_dim, vdim, kv_rank, window, base=1e4, scale=None, mlp=None) -> dict:
    m = dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, rot=dict(base=base, dims=rot_dim), mask=dict(size=window),
             scale=(dim + rot_dim) ** -0.5 if scale is None else scale)
    return dict(type="latent_attention", mixer=m, mlp=mlp)


def left(heads, kv_heads, dim, vdim, chunk, rot_dims, base=1e4, scale=None, scaling=None) -> dict:
    rot = dict(base=base, dims=rot_dims)
    if scaling is not None:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, mask=dict(size=chunk), rot=rot, scale=dim ** -0.5 if scale is None else scale)


def right(heads, vdim, state, groups=1, conv=4, norm_groups=1) -> dict:
    return dict(heads=heads, vdim=vdim, state=state, groups=groups, conv=conv, norm_groups=norm_groups)


def parallel(a, r, mlp=None) -> dict:
    return dict(type="parallel", mixer=dict(left=a, right=r), mlp=mlp)


def dense(ff, limit=1.5) -> dict:
    return dict(kind="dense", ff=ff, limit=limit)


def moe(experts, top, ff) -> dict:
    return dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top))


def config(layers: List[dict], width: int, vocab: int, eps: float = 1e-6, taps: int = 4, logit_scale: float = 0.7) -> dict:
    return dict(architecture="Nikedra", layers=layers, norm=dict(eps=eps), canon=dict(taps=taps), logit_scale=logit_scale, vocab=vocab,
                width=width)


CONFIGS: Dict[str, dict] = {
    # every mixer and feed-forward, shared key heads, groups, frequencies scaled on part of the heads, small windows and chunks
    "mixed": config([delta(6, 3, 24, 40, conv=3, mlp=dense(104)),
                     parallel(left(6, 2, 48, 40, 24, 32, scaling=(4.0, 64, 6.0, 0.5)), right(6, 16, 24, groups=2, conv=3, norm_groups=3), mlp=moe(6, 2, 72)),
                     latent(3, 24, 16, 40, 56, 20, base=300.0),
                     latent(2, 16, 8, 24, 24, 1, mlp=moe(5, 3, 40)),
                     delta(2, 2, 40, 24, conv=2, mlp=moe(4, 1, 48)),
                     parallel(left(4, 4, 32, 32, 7, 32, base=5e5, scale=0.31), right(3, 24, 16, groups=3, conv=5), mlp=dense(72, 0.7))],
                    160, 401, taps=3),
    # sizes the vectorised paths do not take, no history, one expert, no feed-forward
    "odd": config([parallel(left(3, 1, 10, 7, 5, 6, scaling=(2.0, 40, 8.0, 1.0)), right(3, 5, 9, conv=1, norm_groups=5), mlp=moe(3, 3, 21)),
                   delta(3, 1, 9, 7, conv=1, mlp=dense(33, 0.4)),
                   latent(3, 7, 6, 9, 13, 11),
                   delta(2, 1, 5, 11, conv=4)], 90, 203, eps=3e-4, taps=1, logit_scale=1.0),
    # heads of the kernels' own sizes, the fused products, ranks that fill the kernels' tiles
    "large": config([delta(4, 2, 128, 128, mlp=dense(256)),
                     parallel(left(8, 2, 128, 128, 64, 64, scaling=(8.0, 512, 32.0, 1.0)), right(8, 64, 128, groups=2, norm_groups=2), mlp=moe(8, 2, 128)),
                     latent(16, 64, 64, 128, 256, 100, mlp=dense(384, 3.0)),
                     delta(4, 4, 64, 64, mlp=moe(8, 3, 256))], 256, 512),
    # no choices between experts: 16-bit rounding cannot switch anything
    "no_experts": config([latent(4, 32, 16, 64, 128, 33, mlp=dense(96)), parallel(left(4, 1, 64, 48, 50, 48), right(4, 32, 64), mlp=moe(3, 3, 64)),
                          delta(4, 4, 32, 64, mlp=dense(128, 2.0)), parallel(left(6, 3, 200, 40, 31, 40), right(2, 64, 32, norm_groups=2))], 128, 300),
    "only_delta": config([delta(2, 1, 32, 32, mlp=dense(64)), delta(3, 3, 16, 24)], 64, 130, taps=2),
    "only_latent": config([latent(2, 32, 16, 32, 32, 9, mlp=dense(64)), latent(3, 8, 8, 16, 16, 40)], 64, 130),
    "only_parallel": config([parallel(left(2, 1, 32, 32, 16, 16), right(4, 16, 16)), parallel(left(2, 2, 64, 64, 3, 64), right(2, 32, 32, groups=2),
                                                                                             mlp=dense(64))], 64, 130, taps=5),
}
RANKS: Tuple[int, int] = (10, 14)         # inner sizes of the decays' and the gates' projections: only the tensors have them


def weights(cfg: dict, seed: int = 0, steady: bool = False, ranks: Tuple[int, int] = RANKS) -> Dict[str, torch.Tensor]:
    """Values that bf16 holds exactly, scaled so that every mechanism shows in the logits.  ``steady``: a few features of
    every token's embedding are alike and decide between the experts, so that no rounding can turn a choice."""
    g = torch.Generator().manual_seed(seed)
    out: Dict[str, torch.Tensor] = {}
    W, taps = cfg["width"], cfg["canon"]["taps"]

    def n(name, *shape, std=1.0, mean=0.0):
        out[name] = (torch.randn(shape, generator=g) * std + mean).to(torch.bfloat16)

    def mat(name, rows, cols, gain=1.0):
        n(name, rows, cols, std=gain * cols ** -0.5)

    n("embed", cfg["vocab"], W)
    if steady:
        out["embed"][:, :8] = 3.0
    n("embed.norm", std=0.1, mean=1.3)
    for i, layer in enumerate(cfg["layers"]):
        p, m, mlp, kind = f"l{i}.", layer["mixer"], layer["mlp"], layer["type"]
        n(p + "norm1", std=0.1, mean=0.9)
        if mlp is not None:
            n(p + "norm2", std=0.1, mean=1.1)
        n(p + "canon1", W, taps, std=0.4)
        n(p + "dwa", i + 2, std=0.25)
        out[p + "dwa"][-1] += 0.8
        p += "mix."
        if kind == "channel_delta":
            H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            for t, rows in (("q", G * D), ("k", G * D), ("v", H * Dv)):
                mat(p + t, rows, W, 1.5)
                n(f"{p}{t}.conv", rows, m["conv"], std=0.7)
            mat(p + "b", H, W, 1.5)
            n(p + "A_log", H, std=0.7, mean=-1.0)
            mat(p + "a1", ranks[0], W, 1.5)
            mat(p + "a2", H * D, ranks[0], 1.5)
            n(p + "dt_bias", H * D, std=1.5, mean=-1.0)         # decays from hardly any to e^-10 a token
            mat(p + "g1", ranks[1], W, 1.5)
            mat(p + "g2", H * Dv, ranks[1], 1.5)
            n(p + "norm", Dv, std=0.2, mean=1.0)
            mat(p + "o", W, H * Dv, 1.5)
        elif kind == "latent_attention":
            H, D, R, Dv, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
            mat(p + "q", H * (D + R), W, 1.7)
            mat(p + "dkv", rank + R, W, 1.3)
            n(p + "dkv.norm", rank, std=0.2, mean=1.0)
            mat(p + "uk", H * D, rank, 1.3)
            mat(p + "uv", H * Dv, rank)
            mat(p + "g", H * Dv, W, 1.5)
            mat(p + "o", W, H * Dv, 2.0)
        else:
            a, r = m["left"], m["right"]
            H, G = a["heads"], a["kv_heads"]
            mat(p + "left.q", H * a["dim"], W, 1.5)
            mat(p + "left.k", G * a["dim"], W, 1.5)
            mat(p + "left.v", G * a["vdim"], W)
            mat(p + "left.g", H, W, 1.5)
            mat(p + "left.o", W, H * a["vdim"])
            inner, gn = r["heads"] * r["vdim"], r["groups"] * r["state"]
            mat(p + "right.in", 2 * inner + 2 * gn + r["heads"], W, 1.3)
            n(p + "right.conv", inner + 2 * gn, r["conv"], std=0.6)
            n(p + "right.conv.b", inner + 2 * gn, std=0.3)
            n(p + "right.dt_bias", r["heads"], mean=-1.0)
            n(p + "right.A_log", r["heads"], std=0.7)
            n(p + "right.D", r["heads"], std=0.5, mean=0.5)
            n(p + "right.norm", inner, std=0.2, mean=1.0)
            mat(p + "right.o", W, inner)
            n(p + "left.out", W, std=0.2, mean=1.0)
            n(p + "right.out", W, std=0.2, mean=1.0)
        p = f"l{i}.mlp."
        if mlp is None:
            continue
        if mlp["kind"] == "dense":
            for t in ("gate", "up"):
                mat(p + t, mlp["ff"], W, 1.3)
                n(f"{p}{t}.b", mlp["ff"], std=0.5)
            mat(p + "down", W, mlp["ff"])
            n(p + "down.b", W, std=0.3)
        else:
            r = mlp["router"]
            mat(p + "router", r["experts"], W, 0.3 if steady else 2.5)
            if steady:
                at = (torch.randperm(r["experts"], generator=g).float() - 0.5 * r["experts"]) * (0.7 / max(1, r["experts"] - 1))
                out[p + "router"][:, :8] = at.unsqueeze(1).to(torch.bfloat16)
            for e in range(r["experts"]):
                mat(f"{p}e{e}.up", mlp["expert"]["ff"], W, 2.0)
                mat(f"{p}e{e}.down", W, mlp["expert"]["ff"], 2.0)
    n("final.norm", std=0.1, mean=1.0)
    mat("head", cfg["vocab"], W, 3.0)
    return out


def pointed_weights(cfg: dict, gain: float, seed: int = 0) -> Dict[str, torch.Tensor]:
    """Weights under which every attention layer looks for single keys: scores spread so widely that one key takes most of a
    row's weight, wherever it lies."""
    w = weights(cfg, seed)
    for i, layer in enumerate(cfg["layers"]):
        name = {"latent_attention": f"l{i}.mix.q", "parallel": f"l{i}.mix.left.q"}.get(layer["type"])
        if name:
            w[name] = (w[name].float() * gain).to(torch.bfloat16)
    return w


def write_checkpoint(path, cfg: dict, w: Optional[Dict[str, torch.Tensor]] = None, seed: int = 0) -> Dict[str, torch.Tensor]:
    from safetensors.torch import save_file

    w = weights(cfg, seed) if w is None else w
    path.mkdir(parents=True, exist_ok=True)
    (path / "config.json").write_text(json.dumps(cfg))
    save_file({k: v.contiguous() for k, v in w.items()}, str(path / "model.safetensors"))
    return w


def tokens(cfg: dict, n: int, seed: int = 1) -> List[int]:
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def logit_error(got: torch.Tensor, want: torch.Tensor) -> torch.Tensor:
    """Per row: root mean square of the difference (means taken off) over that of the expected logits."""
    d = got.detach().double().cpu() - want
    d = d - d.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / (want - want.mean(-1, keepdim=True)).pow(2).mean().sqrt()
