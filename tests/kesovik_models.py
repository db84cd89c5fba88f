"""Small Kesovik configurations with seeded random weights, in the checkpoint's layout, for the tests."""

from __future__ import annotations

import json
from typing import Dict, List, Optional

import torch


def attention(heads, kv_heads, dim, vdim, window, rot_dims, base=1e4, scale=None) -> dict:
    return dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, mask=dict(size=window), rot=dict(base=base, dims=rot_dims),
                scale=dim ** -0.5 if scale is None else scale)


def lightning(heads, dim, vdim, decay) -> dict:
    assert len(decay) == heads
    return dict(heads=heads, dim=dim, vdim=vdim, decay=list(decay))


def dense(ff) -> dict:
    return dict(kind="dense", ff=ff)


def moe(experts, identity, top, ff, shared=None) -> dict:
    out = dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, identity=identity, top=top))
    if shared is not None:
        out["shared"] = dict(ff=shared)
    return out


def par(left, right, ls, rs, mlp=None) -> dict:
    return dict(type="parallel", mixer=dict(left=left, right=right, left_scale=ls, right_scale=rs), mlp=mlp)


def lin(m, mlp=None) -> dict:
    return dict(type="lightning", mixer=m, mlp=mlp)


def config(layers: List[dict], width: int, vocab: int, eps: float = 1e-6, alpha: float = 1.7, embed: float = 2.5, cap: float = 9.0) -> dict:
    return dict(architecture="Kesovik", layers=layers, norm=dict(eps=eps), postln_alpha=alpha, embedding=dict(scale=embed),
                logit_softcap=cap, vocab=vocab, width=width)


CONFIGS: Dict[str, dict] = {
    # both kinds of layer in turn, values narrower than keys, heads partly rotated, a layer without feed-forward
    "mixed": config([lin(lightning(3, 24, 40, [0.3, 0.9, 0.999]), moe(6, 2, 3, 72, shared=104)),
                     par(attention(6, 2, 48, 24, 13, 32), lightning(2, 40, 16, [0.97, 0.8]), 0.7, 1.3, dense(136)),
                     lin(lightning(2, 16, 56, [0.999, 0.5])),
                     par(attention(4, 4, 32, 72, 29, 32, base=5e5, scale=0.31), lightning(4, 16, 32, [0.9, 0.99, 0.6, 1.0]), 1.2, -0.4,
                         moe(5, 1, 2, 40, shared=40))], 160, 401),
    # sizes the vectorised paths do not take, a window of one token, no shared expert, no identity experts, top 1
    "odd": config([par(attention(3, 1, 10, 7, 1, 4), lightning(1, 5, 6, [0.85]), 1.0, 0.5, moe(5, 0, 1, 33)),
                   lin(lightning(3, 18, 10, [0.99, 0.7, 0.2]), moe(3, 2, 4, 21, shared=35)),
                   par(attention(2, 2, 9, 13, 5, 8), lightning(2, 11, 3, [0.9, 0.4]), 0.3, 2.0, dense(50))], 90, 203, eps=3e-5, alpha=1.0,
                  embed=1.0, cap=30.0),
    # heads of the kernels' own sizes, long windows, the fused expert products
    "large": config([par(attention(16, 2, 128, 128, 70, 128), lightning(4, 128, 192, [0.95, 0.999, 0.8, 0.5]), 0.8, 0.9, dense(512)),
                     lin(lightning(4, 64, 128, [0.999, 0.99, 0.9, 0.3]), moe(8, 4, 4, 128, shared=256)),
                     par(attention(8, 8, 64, 40, 33, 64), lightning(2, 96, 64, [0.98, 0.7]), 0.5, 1.0, moe(4, 1, 2, 256))], 256, 512),
    # no choices between experts: 16-bit rounding cannot switch anything
    "no_experts": config([par(attention(4, 2, 64, 64, 21, 48), lightning(3, 32, 72, [0.9, 0.999, 0.6]), 0.6, 1.4, dense(200)),
                          lin(lightning(5, 48, 64, [0.5, 0.99, 0.8, 0.9, 0.999])),
                          par(attention(6, 1, 40, 200, 64, 40), lightning(2, 128, 128, [0.97, 0.7]), 1.1, 0.7, dense(96))], 128, 300),
    "only_lightning": config([lin(lightning(2, 32, 64, [0.9, 0.99]), dense(64)), lin(lightning(4, 32, 32, [0.5, 0.8, 0.9, 1.0]),
                                                                                     moe(4, 0, 2, 64, shared=64))], 64, 130, cap=5.0),
}


def weights(cfg: dict, seed: int = 0) -> Dict[str, torch.Tensor]:
    """Values that bf16 holds exactly, scaled so that every mechanism shows in the logits."""
    g = torch.Generator().manual_seed(seed)
    out: Dict[str, torch.Tensor] = {}

    def n(name, *shape, std=1.0, mean=0.0):
        out[name] = (torch.randn(*shape, generator=g) * std + mean).to(torch.bfloat16)

    def mat(name, rows, cols, gain=1.0):
        n(name, rows, cols, std=gain * cols ** -0.5)

    def norm(name, width):
        n(name, width, std=0.1, mean=1.0)

    W = cfg["width"]

    def lightning_part(p, m):
        H = m["heads"]
        for name, rows in (("q", H * m["dim"]), ("k", H * m["dim"]), ("v", H * m["vdim"])):
            mat(p + name, rows, W, 1.3)
        mat(p + "g", H * m["vdim"], W)
        norm(p + "norm", H * m["vdim"])
        mat(p + "o", W, H * m["vdim"], 2.5)

    def attention_part(p, m):
        for name, rows in (("q", m["heads"] * m["dim"]), ("k", m["kv_heads"] * m["dim"]), ("v", m["kv_heads"] * m["vdim"])):
            mat(p + name, rows, W)
            n(f"{p}{name}.b", rows, std=0.3)
        n(p + "q.norm", m["heads"] * m["dim"], std=0.3, mean=1.5)
        n(p + "k.norm", m["kv_heads"] * m["dim"], std=0.3, mean=1.5)
        mat(p + "o", W, m["heads"] * m["vdim"], 2.0)

    n("embed", cfg["vocab"], W)
    for i, layer in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}.", layer["mixer"], layer["mlp"]
        norm(p + "norm1", W)
        n(p + "ls1", W, std=0.2, mean=0.8)
        if layer["type"] == "parallel":
            attention_part(p + "mix.left.", m["left"])
            lightning_part(p + "mix.right.", m["right"])
        else:
            lightning_part(p + "mix.", m)
        if mlp is None:
            continue
        norm(p + "norm2", W)
        n(p + "ls2", W, std=0.2, mean=0.8)
        p += "mlp."
        if mlp["kind"] == "dense":
            mat(p + "up", mlp["ff"], W, 1.2)
            mat(p + "down", W, mlp["ff"])
            continue
        r = mlp["router"]
        # peaked scores: few close calls between outputs, which 16-bit rounding could turn
        mat(p + "router", r["experts"] + r["identity"], W, 4.0)
        n(p + "correction", r["experts"] + r["identity"], std=0.4)
        names = [f"e{e}" for e in range(r["experts"])] + (["shared"] if mlp.get("shared") else [])
        for name in names:
            ff = mlp["shared"]["ff"] if name == "shared" else mlp["expert"]["ff"]
            mat(f"{p}{name}.gate", ff, W, 1.5)
            mat(f"{p}{name}.up", ff, W, 1.5)
            mat(f"{p}{name}.down", W, ff, 1.5)
    norm("final.norm", W)
    mat("head", cfg["vocab"], W, 4.0)
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
