"""Pebulix: a decoder whose layers mix tokens either by latent attention without positions or by a gated delta rule,
in any order, each layer with its own sizes.

    x = embed[token]                                       residual stream in fp32
    x += m * mixer(norm1(x));  x += m * mlp(norm2(x))      m = residual_mult; a layer may have no feed-forward
    logits = embed norm(x)                                 tied output projection

Norms are Dynamic Tanh (:class:`..layers.DynamicTanh`), whose kernel also adds the previous sublayer's output to the
stream; mixers are :class:`..layers.LatentAttention` (some layers read an earlier layer's cached latents) and
:class:`..layers.gdn.FusedGatedDeltaNet`; the feed-forward is the gated MLP with the tanh form of the GELU.

``config.json`` lists the layers (``layers``: type, mixer sizes, feed-forward or null) beside ``vocab``, ``width``,
``norm.eps`` and ``residual_mult``; :func:`adapt_config` adds the field names the runner reads."""

from __future__ import annotations

import time
from types import SimpleNamespace
from typing import Any, Dict, Iterable, List, Optional, Tuple

import torch
from torch import nn

from .. import ops
from ..engine.forward_batch import ForwardBatch
from ..layers import MLP, DynamicTanh, LatentAttention, VocabParallelEmbedding
from ..layers.gdn import FusedGatedDeltaNet
from ..mem_cache import LatentPool, LayeredGDNPool
from ..parallel import state as pstate
from .places import load_places, require_positive
from .qwen3 import LogitsProcessorOutput

LATENT, DELTA = "latent_attention", "delta"


def adapt_config(raw: Dict[str, Any]) -> SimpleNamespace:
    """The config as an attribute bag: every key of ``config.json``, checked, plus the runner's field names."""
    layers = raw["layers"]
    for i, layer in enumerate(layers):
        kind, m, mlp, where = layer["type"], layer["mixer"], layer.get("mlp"), f"layer {i}"
        if kind == LATENT:
            require_positive(where, m, ("heads", "dim", "vdim", "q_rank", "kv_rank"))
            j = m.get("kv_from")
            if j is not None:
                src = layers[j] if 0 <= j < i else None
                if src is None or src["type"] != LATENT or src["mixer"].get("kv_from") is not None \
                        or src["mixer"]["kv_rank"] != m["kv_rank"]:
                    raise ValueError(f"{where}: kv_from {j} must name an earlier latent-attention layer with latents of its "
                                     "own and the same kv_rank")
        elif kind == DELTA:
            require_positive(where, m, ("heads", "kv_heads", "dim", "vdim", "conv"))
            if m["heads"] % m["kv_heads"]:
                raise ValueError(f"{where}: {m['heads']} value heads over {m['kv_heads']} key heads")
        else:
            raise ValueError(f"{where}: unknown mixer {kind!r}")
        if mlp is not None and mlp.get("kind") != "dense":
            raise ValueError(f"{where}: unknown feed-forward {mlp.get('kind')!r}")
    ns = SimpleNamespace(**raw)
    ns.architectures, ns.model_type = ["PebulixForCausalLM"], "pebulix"
    ns.vocab_size, ns.hidden_size, ns.num_hidden_layers = int(raw["vocab"]), int(raw["width"]), len(layers)
    ns.rms_norm_eps = float(raw["norm"]["eps"])
    ns.tie_word_embeddings = True
    latent = [layer["mixer"] for layer in layers if layer["type"] == LATENT]
    ns.num_attention_heads = max((m["heads"] for m in latent), default=1)
    ns.num_key_value_heads, ns.head_dim = 1, max((m["kv_rank"] for m in latent), default=0) or ns.hidden_size
    return ns


class PebulixLayer(nn.Module):
    def __init__(self, config, index: int, latent_of: Dict[int, int], gdn_index: int, quant_config, params_dtype) -> None:
        super().__init__()
        spec = config.layers[index]
        m, mlp = spec["mixer"], spec.get("mlp")
        W, eps = config.hidden_size, config.rms_norm_eps
        self.norm1 = DynamicTanh(W, params_dtype)
        if spec["type"] == LATENT:
            src = index if m.get("kv_from") is None else m["kv_from"]
            self.mixer = LatentAttention(W, m["heads"], m["dim"], m["vdim"], m["q_rank"], m["kv_rank"], m["scale"], eps,
                                         latent_of[src], src == index, params_dtype)
        else:
            self.mixer = FusedGatedDeltaNet(W, m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"], eps, gdn_index,
                                            params_dtype)
        self.mlp = None
        if mlp is not None:
            self.norm2 = DynamicTanh(W, params_dtype)
            self.mlp = MLP(W, mlp["ff"], quant_config, f"layers.{index}.mlp", params_dtype, reduce_results=True,
                           activation="gelu_tanh")

    def forward(self, x: torch.Tensor, y: Optional[torch.Tensor], mult: float, fb) -> torch.Tensor:
        """``x`` the fp32 stream without the previous sublayer's output ``y``; returns this layer's last output, which
        the next norm adds."""
        y = self.mixer(self.norm1(x, y, mult), fb)
        if self.mlp is not None:
            y = self.mlp(self.norm2(x, y, mult))
        return y


class PebulixForCausalLM(nn.Module):
    def __init__(self, config, quant_config=None, params_dtype: Optional[torch.dtype] = None) -> None:
        super().__init__()
        if pstate.get_tensor_model_parallel_world_size() > 1 or pstate.get_pipeline_parallel_world_size() > 1:
            raise NotImplementedError("Pebulix runs on one GPU per replica (tp_size and pp_size 1)")
        dt = params_dtype or torch.get_default_dtype()
        self.config, self.quant_config, self.mult = config, quant_config, float(config.residual_mult)
        self.embed = VocabParallelEmbedding(config.vocab_size, config.hidden_size, dt, shard=False)
        # buffers of the latent pool, one per layer that writes latents
        writers = [i for i, s in enumerate(config.layers) if s["type"] == LATENT and s["mixer"].get("kv_from") is None]
        self.latent_widths: List[int] = [config.layers[i]["mixer"]["kv_rank"] for i in writers]
        latent_of = {i: n for n, i in enumerate(writers)}
        layers, g = [], 0
        for i, s in enumerate(config.layers):
            layers.append(PebulixLayer(config, i, latent_of, g, quant_config, dt))
            g += s["type"] == DELTA
        self.layers = nn.ModuleList(layers)
        self.final_norm = DynamicTanh(config.hidden_size, dt)
        self.kv_layers = len(writers)
        self._gdn_pool: Optional[LayeredGDNPool] = None

    # ------------------------------------------------------------------ cache and state
    def kv_cell_bytes(self, dtype: torch.dtype) -> int:
        return LatentPool.cell_bytes(self.latent_widths, dtype)

    def make_kv_pool(self, tokens: int, dtype: torch.dtype, device, page_size: int) -> LatentPool:
        return LatentPool(tokens, self.latent_widths, dtype, device, page_size)

    def make_gdn_pool(self, slots: int, track_slots: int = 0) -> Optional[LayeredGDNPool]:
        """One state row per request-table row plus snapshot rows for the prefix cache (None: no delta-net layers)."""
        shapes = [layer.mixer.state_shape for layer in self.layers if isinstance(layer.mixer, FusedGatedDeltaNet)]
        w = self.embed.weight
        self._gdn_pool = LayeredGDNPool(shapes, slots, w.device, w.dtype, track_slots) if shapes else None
        return self._gdn_pool

    # ------------------------------------------------------------------ forward
    @property
    def lm_head_weight(self) -> torch.Tensor:
        return self.embed.weight

    def forward(self, input_ids, positions, forward_batch: ForwardBatch, input_embeds=None) -> LogitsProcessorOutput:
        fb = forward_batch
        fb.extra["gdn_pool"] = self._gdn_pool
        t0 = time.perf_counter()
        x = ops.embedding_f32(input_ids, self.embed.weight) if input_embeds is None else input_embeds.float()
        y, tap = None, fb.extra.get("layer_outputs")
        for layer in self.layers:
            y = layer(x, y, self.mult, fb)
            if tap is not None:
                tap.append(x + self.mult * y.float())     # the stream after the layer
        rows = fb.logit_row_index()
        if rows is not None:
            x, y = x.index_select(0, rows), y.index_select(0, rows)
        logits = ops.linear(self.final_norm(x, y, self.mult), self.embed.weight)
        ms = (time.perf_counter() - t0) * 1e3
        if fb.forward_mode.is_decode():
            fb.llm_decode_ms = ms
        else:
            fb.llm_prefill_ms = ms
        return LogitsProcessorOutput(next_token_logits=logits)

    # ------------------------------------------------------------------ loading
    def load_weights(self, weights: Iterable[Tuple[str, torch.Tensor]]) -> set:
        """Checkpoint names: ``embed``, ``l<i>.norm1|norm2`` and ``final.norm`` (each with ``.alpha`` and ``.b``),
        ``l<i>.mix.<tensor>``, ``l<i>.mlp.gate|up|down``.  Every tensor must have a place and every place a tensor."""
        return load_places(self._places(), weights)

    def _places(self) -> Dict[str, Any]:
        out: Dict[str, Any] = {}

        def put(p):
            return lambda t: p.data.copy_(t.reshape(p.shape) if t.numel() == p.numel() else t)

        def add_norm(name, norm):
            out[name], out[name + ".b"], out[name + ".alpha"] = put(norm.weight), put(norm.bias), put(norm.alpha)

        out["embed"] = put(self.embed.weight)
        add_norm("final.norm", self.final_norm)
        for i, layer in enumerate(self.layers):
            pre, m = f"l{i}.mix.", layer.mixer
            add_norm(f"l{i}.norm1", layer.norm1)
            if isinstance(m, LatentAttention):
                out[pre + "dq"] = lambda t, m=m: m.load_down("q", t)
                out[pre + "dq.norm"] = put(m.q_latent_norm.weight)
                if m.writes_latent:
                    out[pre + "dkv"] = lambda t, m=m: m.load_down("kv", t)
                    out[pre + "dkv.norm"] = put(m.kv_latent_norm.weight)
                for name, p in (("uq", m.q_up.weight), ("uk", m.k_up.weight), ("uv", m.v_up.weight), ("sink", m.sink), ("o", m.o_proj.weight)):
                    out[pre + name] = put(p)
            else:
                for name in m.shards:
                    out[pre + name] = lambda t, m=m, n=name: m.load_projection(n, t)
                for name in ("q", "k", "v"):
                    out[f"{pre}{name}.conv"] = lambda t, m=m, n=name: m.load_conv(n, t)
                for name, p in (("A_log", m.A_log), ("dt_bias", m.dt_bias), ("norm", m.norm.weight), ("o", m.out_proj.weight)):
                    out[pre + name] = put(p)
            if layer.mlp is not None:
                add_norm(f"l{i}.norm2", layer.norm2)
                gu = layer.mlp.gate_up_proj
                for j, name in enumerate(("gate", "up")):
                    out[f"l{i}.mlp.{name}"] = lambda t, p=gu.weight, j=j: p.weight_loader(p, t, j)
                out[f"l{i}.mlp.down"] = lambda t, p=layer.mlp.down_proj.weight: p.weight_loader(p, t)
        return out

    def post_load(self) -> None:
        for layer in self.layers:
            if isinstance(layer.mixer, LatentAttention):
                layer.mixer.post_load()


EntryClass = PebulixForCausalLM
