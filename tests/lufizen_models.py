"""Small Lufizen configurations with seeded random weights, in the checkpoint's layout, for the tests."""

from __future__ import annotations

import json
from typing import Dict, List, Optional

import torch


def attn(heads, kv_heads, dim, rot_dims, base=1e4, scale=None, scaling=None, mlp=None) -> dict:
    rot = dict(base=base, dims=rot_dims)
    if scaling is not None:
        rot["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    # queries and keys have unit root mean square: scores of standard deviation 1 need 1 / sqrt(dim)
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, rot=rot, scale=dim ** -0.5 if scale is None else scale)
    return dict(type="attention", mixer=m, mlp=mlp)


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, base=1e4, scale=None, mlp=None) -> dict:
    m = dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank, rot=dict(base=base, dims=rot_dim),
             scale=(dim + rot_dim) ** -0.5 if scale is None else scale)
    return dict(type="latent_attention", mixer=m, mlp=mlp)


def moe(experts, top, ff, shared=None, groups=None, scale=1.0) -> dict:
    out = dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top, scale=scale))
    if groups is not None:
        out["router"]["groups"] = dict(count=groups[0], keep=groups[1])
    if shared is not None:
        out["shared"] = dict(ff=shared)
    return out


def config(layers: List[dict], width: int, vocab: int, eps: float = 1e-6, embed: float = 7.5, logit_scale: float = 0.7) -> dict:
    return dict(architecture="Lufizen", layers=layers, norm=dict(eps=eps), embedding=dict(scale=embed), logit_scale=logit_scale,
                vocab=vocab, width=width)


CONFIGS: Dict[str, dict] = {
    # both kinds of layer in turn, heads partly rotated, frequencies scaled, groups of experts, a layer without feed-forward
    "mixed": config([latent(3, 24, 8, 40, 56, 48, mlp=moe(12, 3, 72, shared=104, groups=(4, 2), scale=1.6)),
                     attn(6, 2, 48, 32, scaling=(6.0, 0.9, 3.5, 64), mlp=moe(8, 2, 40, shared=40, groups=(2, 1), scale=0.8)),
                     attn(4, 4, 32, 32, base=5e5, scale=0.31),
                     latent(5, 16, 24, 16, 40, 72, base=300.0, mlp=moe(6, 4, 48, groups=(3, 2), scale=2.5))], 160, 401),
    # sizes the vectorised paths do not take, one expert to choose, groups of one expert, no groups, no shared expert
    "odd": config([attn(3, 1, 10, 6, scaling=(2.0, 1.0, 8.0, 40), mlp=moe(5, 1, 33, groups=(5, 2))),
                   latent(3, 7, 6, 9, 21, 13, mlp=moe(3, 3, 21, shared=35, scale=0.4)),
                   attn(2, 2, 9, 8, base=50.0, mlp=moe(6, 2, 17, shared=1, groups=(2, 2))),
                   latent(1, 12, 2, 5, 10, 30)], 90, 203, eps=3e-4, embed=1.0, logit_scale=1.0),
    # heads of the kernels' own sizes, the fused expert products, ranks that fill the kernels' tiles
    "large": config([attn(16, 2, 128, 64, mlp=moe(16, 4, 128, shared=256, groups=(4, 2), scale=2.5)),
                     latent(20, 64, 64, 128, 256, 256, mlp=moe(8, 2, 256, shared=128, groups=(2, 1))),
                     latent(16, 128, 32, 128, 192, 512, mlp=moe(8, 4, 128))], 256, 512),
    # no choices between experts: 16-bit rounding cannot switch anything
    "no_experts": config([latent(4, 32, 16, 64, 72, 128), attn(8, 1, 64, 48, scaling=(8.0, 1.0, 4.0, 128)), attn(6, 3, 200, 40),
                          latent(2, 48, 32, 24, 64, 64, base=2e3)], 128, 300),
    "only_attention": config([attn(4, 2, 64, 64, mlp=moe(4, 2, 64, shared=64)), attn(2, 1, 32, 16, mlp=moe(4, 1, 64, groups=(2, 1)))], 64, 130),
    "only_latent": config([latent(2, 32, 16, 32, 24, 32, mlp=moe(4, 2, 64, groups=(2, 1), scale=1.2)), latent(3, 8, 8, 16, 16, 16)], 64, 130),
}


def weights(cfg: dict, seed: int = 0, steady: bool = False) -> Dict[str, torch.Tensor]:
    """Values that bf16 holds exactly, scaled so that every mechanism shows in the logits.  ``steady``: corrections
    (and sums of two of them) further apart than any scores, so that no rounding can turn a choice between experts or
    groups."""
    g = torch.Generator().manual_seed(seed)
    out: Dict[str, torch.Tensor] = {}

    def n(name, *shape, std=1.0, mean=0.0):
        out[name] = (torch.randn(*shape, generator=g) * std + mean).to(torch.bfloat16)

    W, x_std = cfg["width"], max(1.0, cfg["embedding"]["scale"])     # the sublayers read the stream as it is

    def mat(name, rows, cols, gain=1.0):
        n(name, rows, cols, std=gain * cols ** -0.5)

    def from_stream(name, rows, gain=1.0):
        mat(name, rows, W, gain / x_std)

    n("embed", cfg["vocab"], W)
    for i, layer in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}.", layer["mixer"], layer["mlp"]
        H = m["heads"]
        n(p + "norm1", W, std=0.1 * x_std, mean=x_std)
        p += "mix."
        if layer["type"] == "attention":
            from_stream(p + "q", H * m["dim"])
            from_stream(p + "k", m["kv_heads"] * m["dim"], 1.5)
            n(p + "sink", H, mean=1.0)
            mat(p + "o", W, H * m["dim"])
        else:
            from_stream(p + "dq", m["q_rank"])
            n(p + "dq.norm", m["q_rank"], std=0.2, mean=1.0)
            mat(p + "uq", H * (m["dim"] + m["rot_dim"]), m["q_rank"], 1.7)
            from_stream(p + "dkv", m["kv_rank"] + m["rot_dim"], 1.5)
            n(p + "dkv.norm", m["kv_rank"], std=0.2, mean=1.0)
            mat(p + "uk", H * m["dim"], m["kv_rank"], 1.3)
            mat(p + "uv", H * m["vdim"], m["kv_rank"])
            from_stream(p + "g", H, 2.0)
            mat(p + "o", W, H * m["vdim"])
        if mlp is None:
            continue
        p, r = f"l{i}.", mlp["router"]
        n(p + "norm2", W, std=0.1 * x_std, mean=x_std)
        p += "mlp."
        # spread scores: few close calls between experts or groups, which 16-bit rounding could turn
        from_stream(p + "router", r["experts"], 2.5)
        n(p + "correction", r["experts"], std=0.3)
        if steady:
            out[p + "correction"] = (2.5 * 2.0 ** torch.randperm(r["experts"], generator=g)).to(torch.bfloat16)
        names = [f"e{e}" for e in range(r["experts"])] + (["shared"] if mlp.get("shared") else [])
        for name in names:
            ff = mlp["shared"]["ff"] if name == "shared" else mlp["expert"]["ff"]
            from_stream(f"{p}{name}.gate", ff, 1.5)
            from_stream(f"{p}{name}.up", ff, 1.5)
            mat(f"{p}{name}.down", W, ff, 1.5)
        if mlp.get("shared"):
            from_stream(p + "shared.sg", 1, 2.0)
    n("final.norm", W, std=0.1, mean=1.0)
    mat("head", cfg["vocab"], W, 3.0)
    return out


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


def pointed_weights(cfg: dict, gain: float, seed: int = 0) -> Dict[str, torch.Tensor]:
    """Weights under which every attention layer looks for single far keys: scores spread so widely that one key takes most
    of a row's weight, wherever it lies."""
    w = weights(cfg, seed)
    for i, layer in enumerate(cfg["layers"]):
        if layer["type"] == "latent_attention":
            w[f"l{i}.mix.uq"] = (w[f"l{i}.mix.uq"].float() * gain).to(torch.bfloat16)
    return w
