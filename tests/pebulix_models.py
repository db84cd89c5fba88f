"""Small Pebulix configurations with seeded random weights, in the checkpoint's layout, for the tests."""

from __future__ import annotations

import json
from typing import Dict, List, Optional

import torch


def latent(heads, dim, vdim, q_rank, kv_rank, scale=None, ff=None, kv_from=None) -> dict:
    m = dict(heads=heads, dim=dim, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank, scale=dim ** -0.5 if scale is None else scale)
    if kv_from is not None:
        m["kv_from"] = kv_from
    return dict(type="latent_attention", mixer=m, mlp=None if ff is None else dict(kind="dense", ff=ff))


def delta(heads, kv_heads, dim, vdim, conv, ff=None) -> dict:
    return dict(type="delta", mixer=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv),
                mlp=None if ff is None else dict(kind="dense", ff=ff))


def config(layers: List[dict], width: int, vocab: int, eps: float = 1e-6, mult: float = 0.6) -> dict:
    return dict(architecture="Pebulix", layers=layers, norm=dict(eps=eps), residual_mult=mult, vocab=vocab, width=width)


CONFIGS: Dict[str, dict] = {
    # delta first, a feed-forward on a delta layer and none on a latent one, a shared latent two layers up
    "mixed": config([delta(6, 3, 40, 24, 4, ff=136), latent(5, 48, 32, 56, 72), delta(2, 2, 24, 56, 2),
                     latent(3, 24, 40, 40, 40, ff=96), latent(4, 32, 32, 48, 72, kv_from=1, scale=0.31)], 160, 401),
    # sizes the vectorised paths do not take: odd widths and ranks, one tap, one head
    "odd": config([latent(3, 20, 12, 30, 36, ff=50), delta(3, 1, 18, 10, 1), latent(1, 9, 7, 11, 13), delta(1, 1, 5, 6, 5, ff=33),
                   latent(2, 20, 12, 14, 36, kv_from=0)], 90, 203, eps=3e-5, mult=1.0),
    # heads of the kernels' own sizes, ranks above 128, more than 16 heads
    "large": config([latent(20, 64, 64, 136, 264, ff=256), delta(4, 2, 128, 128, 4, ff=128), delta(4, 4, 64, 96, 3),
                     latent(8, 128, 128, 96, 512, ff=128), latent(6, 96, 128, 64, 264, kv_from=0)], 256, 512, mult=0.8),
    "only_latent": config([latent(4, 64, 64, 64, 64, ff=64), latent(4, 64, 64, 64, 64, kv_from=0, ff=64)], 64, 130),
    "only_delta": config([delta(4, 2, 32, 64, 4, ff=64), delta(4, 4, 32, 32, 3)], 64, 130),
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
        n(name + ".b", width, std=0.1)
        out[name + ".alpha"] = torch.tensor(0.75, dtype=torch.bfloat16)

    W = cfg["width"]
    n("embed", cfg["vocab"], W)
    norm("final.norm", W)
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}.mix."
        norm(f"l{i}.norm1", W)
        if layer["type"] == "latent_attention":
            mat(p + "dq", m["q_rank"], W)
            n(p + "dq.norm", m["q_rank"], std=0.1, mean=1.0)
            mat(p + "uq", m["heads"] * m["dim"], m["q_rank"], 1.6)
            if m.get("kv_from") is None:
                mat(p + "dkv", m["kv_rank"], W)
                n(p + "dkv.norm", m["kv_rank"], std=0.1, mean=1.0)
            mat(p + "uk", m["heads"] * m["dim"], m["kv_rank"], 1.6)
            mat(p + "uv", m["heads"] * m["vdim"], m["kv_rank"], 1.5)
            n(p + "sink", m["heads"], std=1.0, mean=1.0)
            mat(p + "o", W, m["heads"] * m["vdim"], 1.5)
        else:
            H, Hk = m["heads"], m["kv_heads"]
            for name, rows in (("q", Hk * m["dim"]), ("k", Hk * m["dim"]), ("v", H * m["vdim"])):
                mat(p + name, rows, W, 2.0)
                n(p + name + ".conv", rows, m["conv"], std=0.7)
            mat(p + "g", H * m["vdim"], W)
            mat(p + "b", H, W)
            mat(p + "a", H, W)
            n(p + "A_log", H, std=0.7, mean=-1.0)
            n(p + "dt_bias", H, std=0.7, mean=-1.0)
            n(p + "norm", m["vdim"], std=0.1, mean=1.0)
            mat(p + "o", W, H * m["vdim"], 1.5)
        if layer["mlp"] is not None:
            norm(f"l{i}.norm2", W)
            ff = layer["mlp"]["ff"]
            mat(f"l{i}.mlp.gate", ff, W, 1.5)
            mat(f"l{i}.mlp.up", ff, W, 1.5)
            mat(f"l{i}.mlp.down", W, ff)
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
