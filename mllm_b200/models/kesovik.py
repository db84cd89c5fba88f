"""Kesovik: a decoder whose layers mix tokens by lightning attention, alone or side by side with sliding-window attention,
in any order, each layer with its own sizes; norms stand behind the residual sums.

    x = scale * embed[token]                                   residual stream in fp32
    x = norm1(alpha * x + ls1 * mixer(x));  x = norm2(alpha * x + ls2 * ff(x))
    logits = cap * tanh(head final_norm(x) / cap)

Norms are RMS norms (:class:`..layers.PostRMSNorm`), whose kernel also forms the sum in front of them; mixers are
:class:`..layers.ParallelMixer` over :class:`..layers.LightningAttention` and :class:`..layers.RowNormAttention`; the
feed-forward is a squared-ReLU MLP or a mixture of gated experts, some of which may be the identity, with a shared
expert.  A layer may have no feed-forward.

``config.json`` lists the layers (``layers``: type, mixer sizes, feed-forward or null) beside ``vocab``, ``width``,
``norm.eps``, ``embedding.scale``, ``postln_alpha`` and ``logit_softcap``; :func:`adapt_config` adds the field names the
runner reads."""

from __future__ import annotations

import time
from types import SimpleNamespace
from typing import Any, Dict, Iterable, List, Optional, Tuple

import torch
from torch import nn

from .. import ops
from ..engine.forward_batch import ForwardBatch
from ..layers import MLP, LightningAttention, ParallelMixer, PostRMSNorm, RowNormAttention, SquaredReluMLP, VocabParallelEmbedding
from ..layers.moe import SparseMoeBlock
from ..mem_cache import LayeredGDNPool, LayeredKVPool
from ..parallel import state as pstate
from .places import load_places, mixture_places, put, require_positive
from .qwen3 import LogitsProcessorOutput

PARALLEL, LIGHTNING = "parallel", "lightning"
RENORM_EPS = 1e-20        # joins the sum that the chosen experts' scores are divided by


def _check_attention(where: str, m: Dict[str, Any]) -> None:
    require_positive(where, m, ("heads", "kv_heads", "dim", "vdim"))
    if m["heads"] % m["kv_heads"]:
        raise ValueError(f"{where}: {m['heads']} query heads over {m['kv_heads']} key/value heads")
    if "scale" not in m:
        raise ValueError(f"{where}: scale must be given")
    dims = int((m.get("rot") or {}).get("dims", 0))
    if dims % 2 or not 0 <= dims <= m["dim"]:
        raise ValueError(f"{where}: {dims} of {m['dim']} features rotated")
    if m.get("mask") is not None:
        require_positive(f"{where}: mask", m["mask"], ("size",))


def _check_lightning(where: str, m: Dict[str, Any]) -> None:
    require_positive(where, m, ("heads", "dim", "vdim"))
    d = m.get("decay")
    if not isinstance(d, (int, float)) and (d is None or len(d) != m["heads"]):
        raise ValueError(f"{where}: decay must hold one factor for each of {m['heads']} heads")


def _check_mlp(where: str, mlp: Optional[Dict[str, Any]]) -> None:
    if mlp is None:
        return
    if mlp.get("kind") == "dense":
        require_positive(where, mlp, ("ff",))
    elif mlp.get("kind") == "moe":
        r = mlp["router"]
        require_positive(where, r, ("experts", "top"))
        require_positive(f"{where}: expert", mlp["expert"], ("ff",))
        outputs = int(r["experts"]) + int(r.get("identity") or 0)
        if r["top"] > min(outputs, 32) or outputs > 256:
            raise ValueError(f"{where}: {r['top']} of {outputs} router outputs (at most 32 of 256)")
        if mlp.get("shared") is not None:
            require_positive(f"{where}: shared", mlp["shared"], ("ff",))
    else:
        raise ValueError(f"{where}: unknown feed-forward {mlp.get('kind')!r}")


def adapt_config(raw: Dict[str, Any]) -> SimpleNamespace:
    """The config as an attribute bag: every key of ``config.json``, checked, plus the runner's field names."""
    layers = raw["layers"]
    attention: List[Dict[str, Any]] = []
    for i, layer in enumerate(layers):
        kind, m, where = layer["type"], layer["mixer"], f"layer {i}"
        if kind == PARALLEL:
            _check_attention(f"{where} left", m["left"])
            _check_lightning(f"{where} right", m["right"])
            attention.append(m["left"])
        elif kind == LIGHTNING:
            _check_lightning(where, m)
        else:
            raise ValueError(f"{where}: unknown mixer {kind!r}")
        _check_mlp(where, layer.get("mlp"))
    ns = SimpleNamespace(**raw)
    ns.architectures, ns.model_type = ["KesovikForCausalLM"], "kesovik"
    ns.vocab_size, ns.hidden_size, ns.num_hidden_layers = int(raw["vocab"]), int(raw["width"]), len(layers)
    ns.rms_norm_eps = float(raw["norm"]["eps"])
    ns.tie_word_embeddings = False
    ns.num_attention_heads = max((m["heads"] for m in attention), default=1)
    ns.num_key_value_heads = max((m["kv_heads"] for m in attention), default=1)
    ns.head_dim = max((max(m["dim"], m["vdim"]) for m in attention), default=0) or ns.hidden_size
    return ns


class KesovikMoE(nn.Module):
    """Routed experts (weighted and summed by the norm behind the block) and the shared expert."""

    def __init__(self, width: int, mlp: Dict[str, Any], params_dtype: torch.dtype, prefix: str) -> None:
        super().__init__()
        r = mlp["router"]
        self.block = SparseMoeBlock(width, mlp["expert"]["ff"], r["experts"], r["top"], True, params_dtype, prefix,
                                    identity_experts=int(r.get("identity") or 0), choice_bias=True, renorm_eps=RENORM_EPS, fp32_logits=True)
        self.shared = None
        if mlp.get("shared") is not None:
            self.shared = MLP(width, mlp["shared"]["ff"], None, f"{prefix}.shared", params_dtype, reduce_results=True)

    def forward(self, h: torch.Tensor):
        return self.block.expert_rows(h), None if self.shared is None else self.shared(h)


class KesovikLayer(nn.Module):
    def __init__(self, config, index: int, kv_index: int, state_index: int, params_dtype: torch.dtype) -> None:
        super().__init__()
        spec = config.layers[index]
        m, mlp = spec["mixer"], spec.get("mlp")
        W, eps, alpha = config.hidden_size, config.rms_norm_eps, float(config.postln_alpha)

        def lightning(s):
            return LightningAttention(s["heads"], s["dim"], s["vdim"], s["decay"], eps, state_index)

        if spec["type"] == PARALLEL:
            a = m["left"]
            rot, mask = a.get("rot") or {}, a.get("mask")
            left = RowNormAttention(a["heads"], a["kv_heads"], a["dim"], a["vdim"], a["scale"], eps, kv_index, int(rot.get("dims", 0)),
                                    float(rot.get("base", 1.0)), None if mask is None else int(mask["size"]), params_dtype)
            self.mixer = ParallelMixer(W, [left, lightning(m["right"])], [m["left_scale"], m["right_scale"]], params_dtype)
        else:
            self.mixer = ParallelMixer(W, [lightning(m)], [1.0], params_dtype)

        def scale():
            return nn.Parameter(torch.ones(W, dtype=torch.float32), requires_grad=False)

        self.norm1, self.ls1 = PostRMSNorm(W, eps, alpha, params_dtype), scale()
        self.mlp = None
        if mlp is not None:
            self.norm2, self.ls2 = PostRMSNorm(W, eps, alpha, params_dtype), scale()
            self.mlp = KesovikMoE(W, mlp, params_dtype, f"layers.{index}.mlp") if mlp["kind"] == "moe" else \
                SquaredReluMLP(W, mlp["ff"], params_dtype)

    def forward(self, x: torch.Tensor, h: torch.Tensor, fb) -> torch.Tensor:
        """``x`` the fp32 stream (updated in place), ``h`` the same in the activations' type; returns the new ``h``."""
        h = self.norm1(x, self.mixer(h, fb), self.ls1)
        if isinstance(self.mlp, KesovikMoE):
            experts, shared = self.mlp(h)
            h = self.norm2(x, shared, self.ls2, experts=experts)
        elif self.mlp is not None:
            h = self.norm2(x, self.mlp(h), self.ls2)
        return h


class KesovikForCausalLM(nn.Module):
    def __init__(self, config, quant_config=None, params_dtype: Optional[torch.dtype] = None) -> None:
        super().__init__()
        if pstate.get_tensor_model_parallel_world_size() > 1 or pstate.get_pipeline_parallel_world_size() > 1:
            raise NotImplementedError("Kesovik runs on one GPU per replica (tp_size and pp_size 1)")
        if quant_config is not None:
            raise NotImplementedError("Kesovik has no quantised form")
        dt = params_dtype or torch.get_default_dtype()
        self.config, self.quant_config = config, quant_config
        self.embed_scale = float((getattr(config, "embedding", None) or {}).get("scale", 1.0))
        self.softcap = float(getattr(config, "logit_softcap", None) or 0.0)
        self.embed = VocabParallelEmbedding(config.vocab_size, config.hidden_size, dt, shard=False)
        self.head = nn.Module()
        self.head.weight = nn.Parameter(torch.zeros(config.vocab_size, config.hidden_size, dtype=dt), requires_grad=False)
        layers, kv = [], 0
        for i, s in enumerate(config.layers):
            layers.append(KesovikLayer(config, i, kv, i, dt))       # every layer has a lightning state
            kv += s["type"] == PARALLEL
        self.layers = nn.ModuleList(layers)
        self.final_norm = PostRMSNorm(config.hidden_size, config.rms_norm_eps, 1.0, dt)
        self.kv_shapes = [b.kv_shape for b in self._branches() if isinstance(b, RowNormAttention)]
        self.kv_layers = len(self.kv_shapes)
        self._state_pool: Optional[LayeredGDNPool] = None

    def _branches(self) -> Iterable[nn.Module]:
        for layer in self.layers:
            yield from layer.mixer.branches

    # ------------------------------------------------------------------ cache and state
    def kv_cell_bytes(self, dtype: torch.dtype) -> int:
        return LayeredKVPool.cell_bytes(self.kv_shapes, dtype)

    def make_kv_pool(self, tokens: int, dtype: torch.dtype, device, page_size: int) -> LayeredKVPool:
        return LayeredKVPool(tokens, self.kv_shapes, dtype, device, page_size)

    def make_gdn_pool(self, slots: int, track_slots: int = 0) -> LayeredGDNPool:
        """One state row per request-table row plus snapshot rows for the prefix cache."""
        shapes = [b.state_shape for b in self._branches() if isinstance(b, LightningAttention)]
        w = self.embed.weight
        self._state_pool = LayeredGDNPool(shapes, slots, w.device, w.dtype, track_slots)
        return self._state_pool

    # ------------------------------------------------------------------ forward
    @property
    def lm_head_weight(self) -> torch.Tensor:
        return self.head.weight

    def forward(self, input_ids, positions, forward_batch: ForwardBatch, input_embeds=None) -> LogitsProcessorOutput:
        fb = forward_batch
        fb.extra["gdn_pool"] = self._state_pool
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
        if self.softcap > 0:
            logits = ops.soft_cap(logits, self.softcap)
        ms = (time.perf_counter() - t0) * 1e3
        if fb.forward_mode.is_decode():
            fb.llm_decode_ms = ms
        else:
            fb.llm_prefill_ms = ms
        return LogitsProcessorOutput(next_token_logits=logits)

    # ------------------------------------------------------------------ loading
    def load_weights(self, weights: Iterable[Tuple[str, torch.Tensor]]) -> set:
        """Checkpoint names: ``embed``, ``head``, ``final.norm``, ``l<i>.norm1|norm2|ls1|ls2``, ``l<i>.mix.[left.|right.]<tensor>``,
        ``l<i>.mlp.<tensor>``.  Every tensor must have a place and every place a tensor."""
        return load_places(self._places(), weights)

    def _places(self) -> Dict[str, Any]:
        out: Dict[str, Any] = {}

        out["embed"], out["head"], out["final.norm"] = put(self.embed.weight), put(self.head.weight), put(self.final_norm.weight)
        for i, layer in enumerate(self.layers):
            pre, mixer = f"l{i}.", layer.mixer
            out[pre + "norm1"], out[pre + "ls1"] = put(layer.norm1.weight), put(layer.ls1)
            for j, b in enumerate(mixer.branches):
                at = pre + "mix." + (("left.", "right.")[j] if len(mixer.branches) > 1 else "")
                for n in b.shards:
                    out[at + n] = lambda t, m=mixer, j=j, n=n: m.load_in(j, n, t)
                for n in b.biased:
                    out[f"{at}{n}.b"] = lambda t, m=mixer, j=j, n=n: m.load_bias(j, n, t)
                out[at + "o"] = lambda t, m=mixer, j=j: m.load_out(j, t)
                if isinstance(b, RowNormAttention):
                    out[at + "q.norm"], out[at + "k.norm"] = put(b.q_norm.weight), put(b.k_norm.weight)
                else:
                    out[at + "norm"] = put(b.norm.weight)
            if layer.mlp is None:
                continue
            out[pre + "norm2"], out[pre + "ls2"] = put(layer.norm2.weight), put(layer.ls2)
            at = pre + "mlp."
            if isinstance(layer.mlp, SquaredReluMLP):
                out[at + "up"], out[at + "down"] = put(layer.mlp.up_proj.weight), put(layer.mlp.down_proj.weight)
                continue
            out.update(mixture_places(at, layer.mlp.block, layer.mlp.shared))
        return out

    def post_load(self) -> None:
        for layer in self.layers:
            layer.mixer.fold_scales()
            layer.ls1.data.mul_(layer.mixer.result_scale)
            if isinstance(layer.mlp, KesovikMoE):
                layer.mlp.block.process_weights_after_loading()


EntryClass = KesovikForCausalLM
