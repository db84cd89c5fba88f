"""Nikedra: a decoder whose layers mix tokens by latent attention over a sliding window, by a gated delta rule with a decay per
key channel, or by attention inside chunks of positions side by side with a state-space recurrence, in any order, each layer
with its own sizes.  Mixer and feed-forward read the same stream; every layer hands on an average of all results so far.

    x = norm(embed[token])                                   results = [x], in fp32
    h = norm1(x);  h += conv(h)                              a short causal convolution in front of the mixer
    z = x + mixer(h) + ff(norm2(x))                          a layer may have no feed-forward;  results += [z]
    x = sum_j dwa[j] * results[j]
    logits = logit_scale * head final_norm(x)

Norms divide by the root mean square and multiply by one number.  Everything between two layers, the norms of a parallel
mixer's two outputs and the sum of a mixture's experts included, is one kernel (:func:`..ops.depth_step`), which in decode steps
also applies the convolution.  Mixers are :class:`..layers.LatentAttention`, :class:`..layers.gdn.ChannelDeltaNet` and
:class:`..layers.NormedParallelMixer` over :class:`..layers.RotaryAttention` and :class:`..layers.StateSpace`; the feed-forward is a
bounded gated MLP with biases, or a mixture of experts without gates whose weights scale their inputs.

``config.json`` lists the layers (``layers``: type, mixer sizes, feed-forward or null) beside ``vocab``, ``width``,
``norm.eps``, ``canon.taps`` and ``logit_scale``; :func:`adapt_config` adds the field names the runner reads."""

from __future__ import annotations

import time
from types import SimpleNamespace
from typing import Any, Dict, Iterable, List, Optional, Tuple

import torch
from torch import nn

from .. import ops
from ..engine.forward_batch import ForwardBatch
from ..layers import MLP, LatentAttention, NormedParallelMixer, RotaryAttention, StateSpace, VocabParallelEmbedding
from ..layers.gdn import CausalConvolution, ChannelDeltaNet
from ..layers.moe import SparseMoeBlock
from ..mem_cache import LayeredGDNPool, MixedPool
from ..parallel import state as pstate
from .places import Places, load_places, mixture_places, put, require_positive
from .qwen3 import LogitsProcessorOutput

LATENT, DELTA, PARALLEL = "latent_attention", "channel_delta", "parallel"


def _window(m: Dict[str, Any]) -> Optional[int]:
    mask = m.get("mask")
    return None if mask is None else int(mask["size"])


def _rotation(m: Dict[str, Any]) -> Tuple[int, float, Optional[dict]]:
    rot = m.get("rot") or {}
    return int(rot.get("dims", 0)), float(rot.get("base", 1.0)), rot.get("scaling")


def _check_attention(where: str, m: Dict[str, Any], most: int) -> None:
    if "scale" not in m:
        raise ValueError(f"{where}: scale must be given")
    if m.get("mask") is not None:
        require_positive(f"{where}: mask", m["mask"], ("size",))
    dims, _, scaling = _rotation(m)
    if dims % 2 or not 0 <= dims <= most:
        raise ValueError(f"{where}: {dims} of {most} features rotated")
    if scaling is not None:
        require_positive(f"{where}: rot.scaling", scaling, ("original",))
        if not all(float(scaling.get(n) or 0.0) > 0.0 for n in ("factor", "fast", "slow")):
            raise ValueError(f"{where}: rot.scaling needs factor, fast and slow, all positive")


def _check_mixer(where: str, kind: str, m: Dict[str, Any]) -> None:
    if kind == LATENT:
        require_positive(where, m, ("heads", "dim", "vdim", "kv_rank", "rot_dim"))
        if m["kv_rank"] > 1024 or m["kv_rank"] + m["rot_dim"] > 1536:
            raise ValueError(f"{where}: cached rows of {m['kv_rank']} + {m['rot_dim']} features (at most 1024 and 1536 in all)")
        _check_attention(where, m, m["rot_dim"])
        if _rotation(m)[0] != m["rot_dim"]:
            raise ValueError(f"{where}: rot.dims {_rotation(m)[0]} must be rot_dim {m['rot_dim']}")
        if _rotation(m)[2] is not None:
            raise ValueError(f"{where}: the rotated key part has no scaled frequencies")
    elif kind == DELTA:
        require_positive(where, m, ("heads", "kv_heads", "dim", "vdim", "conv"))
        if m["heads"] % m["kv_heads"]:
            raise ValueError(f"{where}: {m['heads']} value heads over {m['kv_heads']} key heads")
    elif kind == PARALLEL:
        a, r = m["left"], m["right"]
        require_positive(f"{where} left", a, ("heads", "kv_heads", "dim", "vdim"))
        if a["heads"] % a["kv_heads"]:
            raise ValueError(f"{where} left: {a['heads']} query heads over {a['kv_heads']} key/value heads")
        _check_attention(f"{where} left", a, a["dim"])
        require_positive(f"{where} right", r, ("heads", "vdim", "state", "groups", "conv", "norm_groups"))
        if r["heads"] % r["groups"] or (r["heads"] * r["vdim"]) % r["norm_groups"]:
            raise ValueError(f"{where} right: {r['heads']} heads of {r['vdim']} in {r['groups']} groups, norm over {r['norm_groups']} parts")
    else:
        raise ValueError(f"{where}: unknown mixer {kind!r}")


def _check_mlp(where: str, mlp: Optional[Dict[str, Any]]) -> None:
    if mlp is None:
        return
    if mlp.get("kind") == "dense":
        require_positive(where, mlp, ("ff",))
        if "limit" not in mlp:
            raise ValueError(f"{where}: limit must be given")
    elif mlp.get("kind") == "moe":
        r = mlp["router"]
        require_positive(where, r, ("experts", "top"))
        require_positive(f"{where}: expert", mlp["expert"], ("ff",))
        if r["top"] > min(int(r["experts"]), 32) or r["experts"] > 256:
            raise ValueError(f"{where}: {r['top']} of {r['experts']} experts (at most 32 of 256)")
    else:
        raise ValueError(f"{where}: unknown feed-forward {mlp.get('kind')!r}")


def adapt_config(raw: Dict[str, Any]) -> SimpleNamespace:
    """The config as an attribute bag: every key of ``config.json``, checked, plus the runner's field names."""
    layers = raw["layers"]
    for i, layer in enumerate(layers):
        _check_mixer(f"layer {i}", layer["type"], layer["mixer"])
        _check_mlp(f"layer {i}", layer.get("mlp"))
    require_positive("canon", raw["canon"], ("taps",))
    if raw["canon"]["taps"] > 16:
        raise ValueError(f"canon: {raw['canon']['taps']} taps (at most 16)")
    ns = SimpleNamespace(**raw)
    ns.architectures, ns.model_type = ["NikedraForCausalLM"], "nikedra"
    ns.vocab_size, ns.hidden_size, ns.num_hidden_layers = int(raw["vocab"]), int(raw["width"]), len(layers)
    ns.rms_norm_eps = float(raw["norm"]["eps"])
    ns.tie_word_embeddings = False
    left = [layer["mixer"]["left"] for layer in layers if layer["type"] == PARALLEL]
    ns.num_attention_heads = max((m["heads"] for m in left), default=1)
    ns.num_key_value_heads = max((m["kv_heads"] for m in left), default=1)
    ns.head_dim = max((max(m["dim"], m["vdim"]) for m in left), default=0) or ns.hidden_size
    return ns


def _number() -> nn.Parameter:
    return nn.Parameter(torch.ones((), dtype=torch.float32), requires_grad=False)


class NikedraLayer(nn.Module):
    def __init__(self, config, index: int, kv_index: int, latent_index: int, state_index: int, params_dtype: torch.dtype) -> None:
        super().__init__()
        spec = config.layers[index]
        m, mlp, W, eps, kind = spec["mixer"], spec.get("mlp"), config.hidden_size, config.rms_norm_eps, spec["type"]
        self.norm1, self.norm2 = _number(), _number()
        self.conv = CausalConvolution(W, int(config.canon["taps"]), state_index, params_dtype)
        if kind == LATENT:
            dims, base, _ = _rotation(m)
            self.mixer = LatentAttention(W, m["heads"], m["dim"], m["vdim"], None, m["kv_rank"], m["scale"], eps, latent_index, True, params_dtype,
                                         dims, base, sinks=False, gated="features", halves=True, window=_window(m))
        elif kind == DELTA:
            rank = int(m.get("rank") or m["vdim"])      # of the decays and gates; a checkpoint's tensors overrule it
            self.mixer = ChannelDeltaNet(W, m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"], rank, rank, eps, state_index + 1,
                                         params_dtype)
        else:
            a, r = m["left"], m["right"]
            left = RotaryAttention(a["heads"], a["kv_heads"], a["dim"], a["vdim"], a["scale"], kv_index, *_rotation(a), chunk=_window(a),
                                   gated=True, dtype=params_dtype)
            right = StateSpace(r["heads"], r["vdim"], r["state"], r["groups"], r["conv"], r["norm_groups"], eps, state_index + 1, params_dtype)
            self.mixer = NormedParallelMixer(W, [left, right], params_dtype)
        self.mlp: Optional[nn.Module] = None
        if mlp is not None and mlp["kind"] == "dense":
            self.mlp = MLP(W, mlp["ff"], None, f"layers.{index}.mlp", params_dtype, reduce_results=True, activation="clamped", bias=True,
                           limit=float(mlp["limit"]))
        elif mlp is not None:
            router = mlp["router"]
            self.mlp = SparseMoeBlock(W, mlp["expert"]["ff"], router["experts"], router["top"], False, params_dtype, f"layers.{index}.mlp",
                                      sigmoid=True, gated=False, weigh_input=True)
        self.dwa = nn.Parameter(torch.zeros(index + 2, dtype=torch.float32), requires_grad=False)

    @property
    def norms(self) -> List[torch.Tensor]:
        return [self.norm1] if self.mlp is None else [self.norm1, self.norm2]

    @property
    def state_shapes(self) -> List[Tuple[int, int, int, int, int]]:
        """Shapes of the layer's states: its convolution's, then its mixer's where that has one."""
        out = [self.conv.state_shape]
        if isinstance(self.mixer, ChannelDeltaNet):
            out.append(self.mixer.state_shape)
        elif isinstance(self.mixer, NormedParallelMixer):
            out.append(self.mixer.branches[1].state_shape)
        return out

    def forward(self, h: List[torch.Tensor], fb):
        """``h``: the normed inputs of mixer (in decode steps behind the convolution) and feed-forward.  Returns the mixer's
        outputs, and the feed-forward's output or its expert rows."""
        x = h[0] if fb.forward_mode.is_decode() else self.conv(h[0], fb)
        mix = self.mixer(x, fb)
        mix = mix if isinstance(mix, tuple) else (mix,)
        if self.mlp is None:
            return mix, None, None
        if isinstance(self.mlp, SparseMoeBlock):
            return mix, None, self.mlp.expert_rows(h[1])
        return mix, self.mlp(h[1]), None


class NikedraForCausalLM(nn.Module):
    def __init__(self, config, quant_config=None, params_dtype: Optional[torch.dtype] = None) -> None:
        super().__init__()
        if pstate.get_tensor_model_parallel_world_size() > 1 or pstate.get_pipeline_parallel_world_size() > 1:
            raise NotImplementedError("Nikedra runs on one GPU per replica (tp_size and pp_size 1)")
        if quant_config is not None:
            raise NotImplementedError("Nikedra has no quantised form")
        dt = params_dtype or torch.get_default_dtype()
        self.config, self.quant_config, self.eps = config, quant_config, config.rms_norm_eps
        self.embed = VocabParallelEmbedding(config.vocab_size, config.hidden_size, dt, shard=False)
        self.embed_norm, self.final_norm = _number(), _number()
        self.head = nn.Module()
        self.head.weight = nn.Parameter(torch.zeros(config.vocab_size, config.hidden_size, dtype=dt), requires_grad=False)
        layers: List[NikedraLayer] = []
        # buffers of the cache and of the states: K / V rows, latent rows and states are counted apart
        self.kv_shapes: List[Tuple[int, int, int]] = []
        self.latent_widths: List[int] = []
        self.state_shapes: List[Tuple[int, int, int, int, int]] = []
        for i, s in enumerate(config.layers):
            layer = NikedraLayer(config, i, len(self.kv_shapes), len(self.latent_widths), len(self.state_shapes), dt)
            if s["type"] == PARALLEL:
                self.kv_shapes.append(layer.mixer.branches[0].kv_shape)
            elif s["type"] == LATENT:
                self.latent_widths.append(layer.mixer.cache_width)
            self.state_shapes.extend(layer.state_shapes)
            layers.append(layer)
        self.layers = nn.ModuleList(layers)
        self.kv_layers = len(self.kv_shapes) + len(self.latent_widths)
        self._state_pool: Optional[LayeredGDNPool] = None

    # ------------------------------------------------------------------ cache and state
    def kv_cell_bytes(self, dtype: torch.dtype) -> int:
        return MixedPool.cell_bytes(self.kv_shapes, self.latent_widths, dtype)

    def make_kv_pool(self, tokens: int, dtype: torch.dtype, device, page_size: int) -> MixedPool:
        return MixedPool(tokens, self.kv_shapes, self.latent_widths, dtype, device, page_size)

    def make_gdn_pool(self, slots: int, track_slots: int = 0) -> LayeredGDNPool:
        """One state row per request-table row plus snapshot rows for the prefix cache."""
        w = self.embed.weight
        self._state_pool = LayeredGDNPool(self.state_shapes, slots, w.device, w.dtype, track_slots)
        return self._state_pool

    # ------------------------------------------------------------------ forward
    @property
    def lm_head_weight(self) -> torch.Tensor:
        return self.head.weight

    def forward(self, input_ids, positions, forward_batch: ForwardBatch, input_embeds=None) -> LogitsProcessorOutput:
        fb = forward_batch
        fb.extra["gdn_pool"] = self._state_pool
        t0 = time.perf_counter()
        table, dt, L = self.embed.weight, self.embed.weight.dtype, len(self.layers)
        if input_embeds is not None:
            table = input_embeds.to(dt).contiguous()
            input_ids = torch.arange(table.shape[0], device=table.device)
        tap = fb.extra.get("layer_outputs")
        # the embedding output, then every layer's result that a later average reads
        results = torch.empty((L, input_ids.numel(), table.shape[1]), dtype=torch.float32, device=table.device)
        ends = [(layer.norms, layer.conv.step(fb)) for layer in self.layers] + [([self.final_norm], None)]
        h = ops.embed_norm(input_ids, table, self.embed_norm, results[0], self.eps, *ends[0])
        x, out = results[0], torch.empty_like(results[0])
        for i, layer in enumerate(self.layers):
            mix, f, experts = layer(h, fb)
            norms, conv = ends[i + 1]
            last = i + 1 == L
            h = ops.depth_step(x, mix, f, experts, results, i + 1, layer.dwa, norms, self.eps, dt, None if last and tap is None else out,
                               keep=not last, conv=conv)
            x = out
            if tap is not None:
                tap.append(x.clone())        # what the layer hands on
        rows = fb.logit_row_index()
        logits = ops.linear(h[0] if rows is None else h[0].index_select(0, rows), self.head.weight)
        ms = (time.perf_counter() - t0) * 1e3
        if fb.forward_mode.is_decode():
            fb.llm_decode_ms = ms
        else:
            fb.llm_prefill_ms = ms
        return LogitsProcessorOutput(next_token_logits=logits)

    # ------------------------------------------------------------------ loading
    def load_weights(self, weights: Iterable[Tuple[str, torch.Tensor]]) -> set:
        """Checkpoint names: ``embed``, ``embed.norm``, ``head``, ``final.norm``, ``l<i>.norm1|norm2|canon1|dwa``,
        ``l<i>.mix.[left.|right.]<tensor>``, ``l<i>.mlp.<tensor>``.  Every tensor must have a place and every place a tensor (layers
        without a feed-forward may or may not have a second norm)."""
        return load_places(self._places(), weights, [f"l{i}.norm2" for i, layer in enumerate(self.layers) if layer.mlp is None])

    def _places(self) -> Places:
        out: Places = {"embed": put(self.embed.weight), "embed.norm": put(self.embed_norm), "head": put(self.head.weight),
                       "final.norm": put(self.final_norm)}
        for i, layer in enumerate(self.layers):
            pre, at, m = f"l{i}.", f"l{i}.mix.", layer.mixer
            for n, p in (("norm1", layer.norm1), ("norm2", layer.norm2), ("canon1", layer.conv.weight), ("dwa", layer.dwa)):
                out[pre + n] = put(p)
            if isinstance(m, LatentAttention):
                for n, part in (("q", "q"), ("dkv", "kv"), ("g", "g")):
                    out[at + n] = lambda t, m=m, part=part: m.load_down(part, t)
                for n, p in (("dkv.norm", m.kv_latent_norm.weight), ("uk", m.k_up.weight), ("uv", m.v_up.weight), ("o", m.o_proj.weight)):
                    out[at + n] = put(p)
            elif isinstance(m, ChannelDeltaNet):
                for n in ("q", "k", "v", "b"):
                    out[at + n] = lambda t, m=m, n=n: m.load_projection(n, t)
                for n in ("q", "k", "v"):
                    out[f"{at}{n}.conv"] = lambda t, m=m, n=n: m.load_conv(n, t)
                for n in ("a1", "a2", "g1", "g2"):
                    out[at + n] = lambda t, m=m, n=n: m.load_low_rank(n, t)
                for n, p in (("A_log", m.A_log), ("dt_bias", m.dt_bias), ("norm", m.norm.weight), ("o", m.out_proj.weight)):
                    out[at + n] = put(p)
            else:
                right = m.branches[1]
                for j, (side, b) in enumerate(zip(("left.", "right."), m.branches)):
                    for n in b.shards:
                        out[at + side + n] = lambda t, m=m, j=j, n=n: m.load_in(j, n, t)
                    out[at + side + "o"] = lambda t, m=m, j=j: m.load_out(j, t)
                    out[at + side + "out"] = put(m.out_norms[j])
                for n, p in (("conv", right.conv1d.weight), ("conv.b", right.conv1d.bias), ("dt_bias", right.dt_bias), ("A_log", right.A_log),
                             ("D", right.D), ("norm", right.norm.weight)):
                    out[f"{at}right.{n}"] = put(p)
            at = pre + "mlp."
            if isinstance(layer.mlp, SparseMoeBlock):
                out.update(mixture_places(at, layer.mlp, None))
            elif layer.mlp is not None:
                gu, down = layer.mlp.gate_up_proj, layer.mlp.down_proj
                for j, n in enumerate(("gate", "up")):
                    out[at + n] = lambda t, p=gu.weight, j=j: p.weight_loader(p, t, j)
                    out[f"{at}{n}.b"] = lambda t, p=gu.bias, j=j: p.weight_loader(p, t, j)
                out[at + "down"] = lambda t, p=down.weight: p.weight_loader(p, t)
                out[at + "down.b"] = put(down.bias)
        return out

    def post_load(self) -> None:
        # the head's input carries the scale of the logits
        self.final_norm.data.mul_(float(getattr(self.config, "logit_scale", 1.0)))
        for layer in self.layers:
            if isinstance(layer.mixer, LatentAttention):
                layer.mixer.post_load()
            if isinstance(layer.mlp, SparseMoeBlock):
                layer.mlp.process_weights_after_loading()


EntryClass = NikedraForCausalLM
