"""Lufizen: a decoder whose layers mix tokens by grouped-query attention that uses its keys as values, or by latent attention
with a rotated key part and output gates, in any order, each layer with its own sizes; norms stand on the sublayers' outputs.

    x = scale * embed[token]                                residual stream in fp32
    x += norm1(mixer(x));  x += norm2(ff(x))                a layer may have no feed-forward
    logits = logit_scale * head final_norm(x)

Norms are RMS norms (:class:`..layers.OutputRMSNorm`), whose kernel also weighs and sums the experts and adds to the
stream; mixers are :class:`..layers.HeadNormAttention` between its projections (:class:`..layers.ParallelMixer` with one
branch) and :class:`..layers.LatentAttention`; the feed-forward is a mixture of gated experts chosen within groups by
logistic scores, beside a shared expert with a gate per token.

``config.json`` lists the layers (``layers``: type, mixer sizes, feed-forward or null) beside ``vocab``, ``width``,
``norm.eps``, ``embedding.scale`` and ``logit_scale``; :func:`adapt_config` adds the field names the runner reads."""

from __future__ import annotations

import time
from types import SimpleNamespace
from typing import Any, Dict, Iterable, List, Optional, Tuple

import torch
from torch import nn

from .. import ops
from ..engine.forward_batch import ForwardBatch
from ..layers import MLP, HeadNormAttention, LatentAttention, OutputRMSNorm, ParallelMixer, PostRMSNorm, VocabParallelEmbedding
from ..layers.moe import SparseMoeBlock
from ..mem_cache import MixedPool
from ..parallel import state as pstate
from .places import Places, load_places, mixture_places, put, require_positive
from .qwen3 import LogitsProcessorOutput

ATTENTION, LATENT = "attention", "latent_attention"


def _check_rotation(where: str, rot: Optional[Dict[str, Any]], most: int) -> None:
    if rot is None:
        return
    dims = int(rot.get("dims", 0))
    if dims % 2 or not 0 <= dims <= most:
        raise ValueError(f"{where}: {dims} of {most} features rotated")
    if "base" not in rot:
        raise ValueError(f"{where}: rot.base must be given")
    if rot.get("scaling") is not None:
        s = rot["scaling"]
        require_positive(f"{where}: rot.scaling", s, ("factor", "original"))
        if not float(s["low"]) < float(s["high"]):
            raise ValueError(f"{where}: rot.scaling needs low < high")


def _check_mixer(where: str, kind: str, m: Dict[str, Any]) -> None:
    if "scale" not in m:
        raise ValueError(f"{where}: scale must be given")
    if kind == ATTENTION:
        require_positive(where, m, ("heads", "kv_heads", "dim"))
        if m["heads"] % m["kv_heads"]:
            raise ValueError(f"{where}: {m['heads']} query heads over {m['kv_heads']} key/value heads")
        if m.get("vdim", m["dim"]) != m["dim"]:
            raise ValueError(f"{where}: the values are the keys, so vdim {m['vdim']} must be dim {m['dim']}")
        _check_rotation(where, m.get("rot"), m["dim"])
    elif kind == LATENT:
        require_positive(where, m, ("heads", "dim", "vdim", "q_rank", "kv_rank", "rot_dim"))
        if m["kv_rank"] > 1024 or m["kv_rank"] + m["rot_dim"] > 1536:
            raise ValueError(f"{where}: cached rows of {m['kv_rank']} + {m['rot_dim']} features (at most 1024 and 1536 in all)")
        _check_rotation(where, m["rot"], m["rot_dim"])
        if m["rot"]["dims"] != m["rot_dim"]:
            raise ValueError(f"{where}: rot.dims {m['rot']['dims']} must be rot_dim {m['rot_dim']}")
    else:
        raise ValueError(f"{where}: unknown mixer {kind!r}")


def _groups(router: Dict[str, Any]) -> Tuple[int, int]:
    g = router.get("groups") or {}
    return int(g.get("count", 1)), int(g.get("keep", g.get("count", 1)))


def _check_mlp(where: str, mlp: Optional[Dict[str, Any]]) -> None:
    if mlp is None:
        return
    if mlp.get("kind") != "moe":
        raise ValueError(f"{where}: unknown feed-forward {mlp.get('kind')!r}")
    r = mlp["router"]
    require_positive(where, r, ("experts", "top"))
    require_positive(f"{where}: expert", mlp["expert"], ("ff",))
    if mlp.get("shared") is not None:
        require_positive(f"{where}: shared", mlp["shared"], ("ff",))
    E, top, (count, keep) = int(r["experts"]), int(r["top"]), _groups(r)
    if E > 256 or top > 32:
        raise ValueError(f"{where}: {top} of {E} experts (at most 32 of 256)")
    if count < 1 or not 1 <= keep <= count or E % count or (keep < count and count > 32):
        raise ValueError(f"{where}: {E} experts in {count} groups, {keep} of them kept (at most 32 equal groups)")
    if top > keep * (E // count):
        raise ValueError(f"{where}: {top} experts chosen from {keep} groups of {E // count}")


def adapt_config(raw: Dict[str, Any]) -> SimpleNamespace:
    """The config as an attribute bag: every key of ``config.json``, checked, plus the runner's field names."""
    layers = raw["layers"]
    for i, layer in enumerate(layers):
        _check_mixer(f"layer {i}", layer["type"], layer["mixer"])
        _check_mlp(f"layer {i}", layer.get("mlp"))
    ns = SimpleNamespace(**raw)
    ns.architectures, ns.model_type = ["LufizenForCausalLM"], "lufizen"
    ns.vocab_size, ns.hidden_size, ns.num_hidden_layers = int(raw["vocab"]), int(raw["width"]), len(layers)
    ns.rms_norm_eps = float(raw["norm"]["eps"])
    ns.tie_word_embeddings = False
    full = [layer["mixer"] for layer in layers if layer["type"] == ATTENTION]
    ns.num_attention_heads = max((layer["mixer"]["heads"] for layer in layers), default=1)
    ns.num_key_value_heads = max((m["kv_heads"] for m in full), default=1)
    ns.head_dim = max((m["dim"] for m in full), default=0) or ns.hidden_size
    return ns


class LufizenMoE(nn.Module):
    """Routed experts and the gated shared expert; the norm behind the block weighs and sums them."""

    def __init__(self, width: int, mlp: Dict[str, Any], params_dtype: torch.dtype, prefix: str) -> None:
        super().__init__()
        r, shared = mlp["router"], mlp.get("shared")
        self.block = SparseMoeBlock(width, mlp["expert"]["ff"], r["experts"], r["top"], False, params_dtype, prefix, choice_bias=True,
                                    sigmoid=True, groups=_groups(r), scale=float(r.get("scale", 1.0)), shared_gate=shared is not None)
        self.shared = None
        if shared is not None:
            self.shared = MLP(width, shared["ff"], None, f"{prefix}.shared", params_dtype, reduce_results=True)

    def forward(self, h: torch.Tensor):
        return self.block.expert_rows(h), None if self.shared is None else self.shared(h)


class LufizenLayer(nn.Module):
    def __init__(self, config, index: int, kv_index: int, latent_index: int, params_dtype: torch.dtype) -> None:
        super().__init__()
        spec = config.layers[index]
        m, mlp, W, eps = spec["mixer"], spec.get("mlp"), config.hidden_size, config.rms_norm_eps
        rot = m.get("rot") or {}
        if spec["type"] == ATTENTION:
            core = HeadNormAttention(m["heads"], m["kv_heads"], m["dim"], m["dim"], m["scale"], eps, kv_index, int(rot.get("dims", 0)),
                                     float(rot.get("base", 1.0)), rot.get("scaling"), halves=True, tied=True, sinks=True, dtype=params_dtype)
            self.mixer = ParallelMixer(W, [core], [1.0], params_dtype)
        else:
            self.mixer = LatentAttention(W, m["heads"], m["dim"], m["vdim"], m["q_rank"], m["kv_rank"], m["scale"], eps, latent_index,
                                         True, params_dtype, m["rot_dim"], float(rot["base"]), rot.get("scaling"), sinks=False, gated=True)
        self.norm1 = OutputRMSNorm(W, eps, params_dtype)
        self.mlp = None
        if mlp is not None:
            self.norm2 = OutputRMSNorm(W, eps, params_dtype)
            self.mlp = LufizenMoE(W, mlp, params_dtype, f"layers.{index}.mlp")

    def forward(self, x: torch.Tensor, h: torch.Tensor, fb) -> torch.Tensor:
        """``x`` the fp32 stream (updated in place), ``h`` the same in the activations' type; returns the new ``h``."""
        h = self.norm1(x, self.mixer(h, fb))
        if self.mlp is not None:
            experts, shared = self.mlp(h)
            h = self.norm2(x, shared, experts)
        return h


class LufizenForCausalLM(nn.Module):
    def __init__(self, config, quant_config=None, params_dtype: Optional[torch.dtype] = None) -> None:
        super().__init__()
        if pstate.get_tensor_model_parallel_world_size() > 1 or pstate.get_pipeline_parallel_world_size() > 1:
            raise NotImplementedError("Lufizen runs on one GPU per replica (tp_size and pp_size 1)")
        if quant_config is not None:
            raise NotImplementedError("Lufizen has no quantised form")
        dt = params_dtype or torch.get_default_dtype()
        self.config, self.quant_config = config, quant_config
        self.embed_scale = float((getattr(config, "embedding", None) or {}).get("scale", 1.0))
        self.embed = VocabParallelEmbedding(config.vocab_size, config.hidden_size, dt, shard=False)
        self.head = nn.Module()
        self.head.weight = nn.Parameter(torch.zeros(config.vocab_size, config.hidden_size, dtype=dt), requires_grad=False)
        layers: List[LufizenLayer] = []
        # buffers of the cache: K / V rows and latent rows are counted apart
        self.kv_shapes: List[Tuple[int, int, int]] = []
        self.latent_widths: List[int] = []
        for i, s in enumerate(config.layers):
            layer = LufizenLayer(config, i, len(self.kv_shapes), len(self.latent_widths), dt)
            if s["type"] == ATTENTION:
                self.kv_shapes.append(layer.mixer.branches[0].kv_shape)
            else:
                self.latent_widths.append(layer.mixer.cache_width)
            layers.append(layer)
        self.layers = nn.ModuleList(layers)
        self.final_norm = PostRMSNorm(config.hidden_size, config.rms_norm_eps, 1.0, dt)
        self.kv_layers = len(layers)

    # ------------------------------------------------------------------ cache
    def kv_cell_bytes(self, dtype: torch.dtype) -> int:
        return MixedPool.cell_bytes(self.kv_shapes, self.latent_widths, dtype)

    def make_kv_pool(self, tokens: int, dtype: torch.dtype, device, page_size: int) -> MixedPool:
        return MixedPool(tokens, self.kv_shapes, self.latent_widths, dtype, device, page_size)

    # ------------------------------------------------------------------ forward
    @property
    def lm_head_weight(self) -> torch.Tensor:
        return self.head.weight

    def forward(self, input_ids, positions, forward_batch: ForwardBatch, input_embeds=None) -> LogitsProcessorOutput:
        fb = forward_batch
        t0 = time.perf_counter()
        if input_embeds is None:
            x, h = ops.embedding_f32(input_ids, self.embed.weight, self.embed_scale, rounded=True)
        else:
            x = input_embeds.float()
            h = x.to(self.embed.weight.dtype)
        tap = fb.extra.get("layer_outputs")
        for layer in self.layers:
            h = layer(x, h, fb)
            if tap is not None:
                tap.append(x.clone())        # the stream after the layer
        rows = fb.logit_row_index()
        if rows is not None:
            x = x.index_select(0, rows)
        logits = ops.linear(self.final_norm.read(x), self.head.weight)
        ms = (time.perf_counter() - t0) * 1e3
        if fb.forward_mode.is_decode():
            fb.llm_decode_ms = ms
        else:
            fb.llm_prefill_ms = ms
        return LogitsProcessorOutput(next_token_logits=logits)

    # ------------------------------------------------------------------ loading
    def load_weights(self, weights: Iterable[Tuple[str, torch.Tensor]]) -> set:
        """Checkpoint names: ``embed``, ``head``, ``final.norm``, ``l<i>.norm1|norm2``, ``l<i>.mix.<tensor>``,
        ``l<i>.mlp.<tensor>``.  Every tensor must have a place and every place a tensor."""
        return load_places(self._places(), weights)

    def _places(self) -> Places:
        out: Places = {"embed": put(self.embed.weight), "head": put(self.head.weight), "final.norm": put(self.final_norm.weight)}
        for i, layer in enumerate(self.layers):
            at, m = f"l{i}.mix.", layer.mixer
            out[f"l{i}.norm1"] = put(layer.norm1.weight)
            if isinstance(m, LatentAttention):
                for n, part in (("dq", "q"), ("dkv", "kv"), ("g", "g")):
                    out[at + n] = lambda t, m=m, part=part: m.load_down(part, t)
                for n, p in (("dq.norm", m.q_latent_norm.weight), ("dkv.norm", m.kv_latent_norm.weight), ("uq", m.q_up.weight),
                             ("uk", m.k_up.weight), ("uv", m.v_up.weight), ("o", m.o_proj.weight)):
                    out[at + n] = put(p)
            else:
                core = m.branches[0]
                for n in core.shards:
                    out[at + n] = lambda t, m=m, n=n: m.load_in(0, n, t)
                out[at + "sink"] = put(core.sink)
                out[at + "o"] = lambda t, m=m: m.load_out(0, t)
            if layer.mlp is not None:
                out[f"l{i}.norm2"] = put(layer.norm2.weight)
                out.update(mixture_places(f"l{i}.mlp.", layer.mlp.block, layer.mlp.shared))
        return out

    def post_load(self) -> None:
        # the head's input carries the scale of the logits
        self.final_norm.weight.data.mul_(float(getattr(self.config, "logit_scale", 1.0)))
        for layer in self.layers:
            if isinstance(layer.mixer, LatentAttention):
                layer.mixer.post_load()
            if layer.mlp is not None:
                layer.mlp.block.process_weights_after_loading()


EntryClass = LufizenForCausalLM
