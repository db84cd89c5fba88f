"""Built-in model shapes so benchmarks and tests can run without a checkpoint directory.

Each preset is a plain attribute bag with the HF ``config.json`` field names the
models read.  Shapes: Qwen3 dense (0.6B / 1.7B / 4B / 8B / 14B / 32B), Qwen3-30B-A3B
(MoE), Llama / Qwen2 decoders, the Qwen3.5 hybrids, Pebulix, Kesovik, Lufizen, Nikedra, and the vision+language pairs Qwen3-VL-2B,
Qwen2-VL-2B and Qwen2.5-VL-3B (each with a ``-tiny`` shape for tests).
"""

from __future__ import annotations

import copy
from types import SimpleNamespace
from typing import Any, Dict


def _dense(hidden, layers, heads, kv, inter, tie, vocab=151936, theta=1e6) -> Dict[str, Any]:
    return dict(
        architectures=["Qwen3ForCausalLM"], model_type="qwen3", hidden_size=hidden, num_hidden_layers=layers,
        num_attention_heads=heads, num_key_value_heads=kv, head_dim=128, intermediate_size=inter,
        vocab_size=vocab, rms_norm_eps=1e-6, rope_theta=theta, tie_word_embeddings=tie,
        max_position_embeddings=40960, attention_bias=False, hidden_act="silu", torch_dtype="bfloat16",
        eos_token_id=151645, bos_token_id=151643,
    )


PRESETS: Dict[str, Dict[str, Any]] = {
    "qwen3-0.6b": _dense(1024, 28, 16, 8, 3072, True),
    "qwen3-1.7b": _dense(2048, 28, 16, 8, 6144, True),
    "qwen3-4b": _dense(2560, 36, 32, 8, 9728, True),
    "qwen3-8b": _dense(4096, 36, 32, 8, 12288, False),
    "qwen3-14b": _dense(5120, 40, 40, 8, 17408, False),
    "qwen3-32b": _dense(5120, 64, 64, 8, 25600, False),
    "qwen3-tiny": _dense(256, 2, 4, 2, 512, True, vocab=1024),
}
PRESETS["qwen3-30b-a3b"] = dict(
    _dense(2048, 48, 32, 4, 6144, False),
    architectures=["Qwen3MoeForCausalLM"], model_type="qwen3_moe", num_experts=128, num_experts_per_tok=8,
    moe_intermediate_size=768, norm_topk_prob=True, decoder_sparse_step=1, mlp_only_layers=[],
)
PRESETS["qwen3-moe-tiny"] = dict(
    _dense(256, 2, 4, 2, 512, True, vocab=1024),
    architectures=["Qwen3MoeForCausalLM"], model_type="qwen3_moe", num_experts=8, num_experts_per_tok=2,
    moe_intermediate_size=256, norm_topk_prob=True, decoder_sparse_step=1, mlp_only_layers=[],
)
# Llama / Qwen2 families (same decoder stack without q/k norms; published shapes)
PRESETS["llama-3.1-8b"] = dict(
    _dense(4096, 32, 32, 8, 14336, False, vocab=128256, theta=5e5),
    architectures=["LlamaForCausalLM"], model_type="llama", rms_norm_eps=1e-5, max_position_embeddings=131072,
    rope_scaling=dict(rope_type="llama3", factor=8.0, low_freq_factor=1.0, high_freq_factor=4.0,
                      original_max_position_embeddings=8192), eos_token_id=128009, bos_token_id=128000,
)
PRESETS["qwen2.5-7b"] = dict(
    _dense(3584, 28, 28, 4, 18944, False, vocab=152064, theta=1e6),
    architectures=["Qwen2ForCausalLM"], model_type="qwen2", max_position_embeddings=32768,
)
PRESETS["llama-tiny"] = dict(_dense(256, 2, 4, 2, 512, True, vocab=1024, theta=1e4),
                             architectures=["LlamaForCausalLM"], model_type="llama")
PRESETS["qwen2-tiny"] = dict(_dense(256, 2, 4, 2, 512, True, vocab=1024), architectures=["Qwen2ForCausalLM"], model_type="qwen2")


def _hybrid(hidden, layers, heads, kv_heads, inter, head_dim, lin_k_heads, lin_v_heads, vocab=151936):
    return dict(
        architectures=["Qwen3_5ForCausalLM"], model_type="qwen3_5_text", vocab_size=vocab, hidden_size=hidden,
        intermediate_size=inter, num_hidden_layers=layers, num_attention_heads=heads, num_key_value_heads=kv_heads,
        head_dim=head_dim, rms_norm_eps=1e-6, tie_word_embeddings=False, max_position_embeddings=32768, attention_bias=False,
        hidden_act="silu", linear_conv_kernel_dim=4, linear_key_head_dim=128, linear_value_head_dim=128,
        linear_num_key_heads=lin_k_heads, linear_num_value_heads=lin_v_heads, full_attention_interval=4,
        layer_types=["full_attention" if (i + 1) % 4 == 0 else "linear_attention" for i in range(layers)],
        rope_parameters=dict(rope_theta=1e7, partial_rotary_factor=0.25, rope_type="default", mrope_section=[11, 11, 10]),
        torch_dtype="bfloat16", eos_token_id=151645,
    )


PRESETS["qwen3.5-2b"] = _hybrid(2048, 24, 8, 2, 6144, 256, 16, 16)
PRESETS["qwen3.5-moe-6b"] = dict(
    PRESETS["qwen3.5-2b"], architectures=["Qwen3_5MoeForCausalLM"], model_type="qwen3_5_moe_text", num_experts=64, num_experts_per_tok=8,
    moe_intermediate_size=512, shared_expert_intermediate_size=512, norm_topk_prob=True,
)
PRESETS["qwen3.5-tiny"] = dict(_hybrid(256, 4, 2, 1, 512, 128, 1, 2, vocab=1024),
                               rope_parameters=dict(rope_theta=1e4, partial_rotary_factor=0.25, rope_type="default",
                                                    mrope_section=[6, 5, 5]))


def _pebulix(layers, width, ff, vocab, heads, dim, q_rank, kv_rank, delta_heads, delta_dim, conv=4) -> Dict[str, Any]:
    """Three delta-net layers to one latent-attention layer; every second latent layer reads the latents of the one before."""
    out, last = [], None
    for i in range(layers):
        mlp = dict(kind="dense", ff=ff)
        if (i + 1) % 4:
            out.append(dict(type="delta", mlp=mlp, mixer=dict(heads=delta_heads, kv_heads=delta_heads, dim=delta_dim,
                                                              vdim=delta_dim, conv=conv)))
            continue
        m = dict(heads=heads, dim=dim, vdim=dim, q_rank=q_rank, kv_rank=kv_rank, scale=dim ** -0.5)
        if last is not None:
            m["kv_from"], last = last, None
        else:
            last = i
        out.append(dict(type="latent_attention", mlp=mlp, mixer=m))
    return dict(architecture="Pebulix", layers=out, norm=dict(eps=1e-6), residual_mult=1.0, vocab=vocab, width=width,
                torch_dtype="bfloat16")


# hidden size, depth, feed-forward, vocabulary and delta-net heads of qwen3.5-2b
PRESETS["pebulix-2b"] = _pebulix(24, 2048, 6144, 151936, heads=16, dim=128, q_rank=1024, kv_rank=512, delta_heads=16, delta_dim=128)
PRESETS["pebulix-tiny"] = _pebulix(4, 128, 256, 1024, heads=2, dim=64, q_rank=64, kv_rank=64, delta_heads=2, delta_dim=32)


def _kesovik(layers, width, ff, vocab, heads, kv_heads, dim, window, lin_heads, lin_dim, par_lin_heads, experts, identity, top, expert_ff,
             shared_ff) -> Dict[str, Any]:
    """Three lightning layers to one with sliding-window attention beside lightning attention; the first feed-forward is
    dense, the others are mixtures."""
    def lightning(n):
        # half-lives from a few tokens to a few hundred, as a geometric series over the heads
        return dict(heads=n, dim=lin_dim, vdim=lin_dim, decay=[1.0 - 2.0 ** (-2.0 - 7.0 * i / max(1, n - 1)) for i in range(n)])

    out = []
    for i in range(layers):
        mlp = dict(kind="dense", ff=ff) if i == 0 else dict(kind="moe", expert=dict(ff=expert_ff), shared=dict(ff=shared_ff),
                                                            router=dict(experts=experts, identity=identity, top=top))
        if (i + 1) % 4:
            out.append(dict(type="lightning", mlp=mlp, mixer=lightning(lin_heads)))
        else:
            left = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, mask=dict(size=window), rot=dict(base=1e6, dims=dim), scale=dim ** -0.5)
            out.append(dict(type="parallel", mlp=mlp, mixer=dict(left=left, right=lightning(par_lin_heads), left_scale=1.0, right_scale=1.0)))
    return dict(architecture="Kesovik", layers=out, norm=dict(eps=1e-6), postln_alpha=2.0, embedding=dict(scale=1.0), logit_softcap=30.0,
                vocab=vocab, width=width, torch_dtype="bfloat16")


# hidden size, depth, vocabulary, linear-attention heads and experts of qwen3.5-moe-6b
PRESETS["kesovik-6b"] = _kesovik(24, 2048, 6144, 151936, heads=16, kv_heads=4, dim=128, window=2048, lin_heads=16, lin_dim=128,
                                 par_lin_heads=8, experts=64, identity=8, top=8, expert_ff=512, shared_ff=512)
PRESETS["kesovik-tiny"] = _kesovik(4, 128, 256, 1024, heads=4, kv_heads=2, dim=32, window=48, lin_heads=2, lin_dim=32, par_lin_heads=2,
                                   experts=6, identity=2, top=2, expert_ff=64, shared_ff=64)


def _lufizen(layers, width, vocab, heads, kv_heads, dim, rot_dim, vdim, q_rank, kv_rank, experts, groups, keep, top, expert_ff,
             shared_ff) -> Dict[str, Any]:
    """Latent attention and key-valued attention in turn, a mixture behind each."""
    out = []
    for i in range(layers):
        mlp = dict(kind="moe", expert=dict(ff=expert_ff), shared=dict(ff=shared_ff),
                   router=dict(experts=experts, groups=dict(count=groups, keep=keep), scale=2.5, top=top))
        if i % 2 == 0:
            m = dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank, rot=dict(base=1e4, dims=rot_dim),
                     scale=(dim + rot_dim) ** -0.5)
            out.append(dict(type="latent_attention", mlp=mlp, mixer=m))
        else:
            rot = dict(base=5e5, dims=dim // 2, scaling=dict(factor=8.0, low=1.0, high=4.0, original=8192))
            m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, rot=rot, scale=dim ** -0.5)
            out.append(dict(type="attention", mlp=mlp, mixer=m))
    return dict(architecture="Lufizen", layers=out, norm=dict(eps=1e-6), embedding=dict(scale=1.0), logit_scale=1.0, vocab=vocab, width=width,
                torch_dtype="bfloat16")


# hidden size, depth, vocabulary, query and key heads and experts of qwen2-moe-6b
PRESETS["lufizen-6b"] = _lufizen(24, 2048, 151936, heads=16, kv_heads=4, dim=128, rot_dim=64, vdim=128, q_rank=1024, kv_rank=512, experts=64,
                                 groups=8, keep=4, top=8, expert_ff=512, shared_ff=512)
PRESETS["lufizen-tiny"] = _lufizen(4, 128, 1024, heads=4, kv_heads=2, dim=32, rot_dim=16, vdim=32, q_rank=64, kv_rank=64, experts=8, groups=4,
                                   keep=2, top=2, expert_ff=64, shared_ff=64)


def _nikedra(layers, width, ff, vocab, heads, kv_heads, dim, chunk, ssd_heads, ssd_vdim, state, groups, lin_heads, lin_dim, rank, lat_heads, lat_dim,
             rot_dim, lat_vdim, kv_rank, window, experts, top, expert_ff) -> Dict[str, Any]:
    """Three delta-net layers and one with attention in turn, the latter alternately parallel and latent; a mixture beside all but
    every eighth layer, which has a dense feed-forward."""
    out = []
    for i in range(layers):
        moe = dict(kind="moe", expert=dict(ff=expert_ff), router=dict(experts=experts, top=top))
        mlp = moe if i % 8 else dict(kind="dense", ff=ff, limit=7.0)
        if i % 8 == 3:
            left = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, mask=dict(size=chunk), scale=dim ** -0.5,
                        rot=dict(base=1e6, dims=dim, scaling=dict(factor=8.0, original=4096, fast=32.0, slow=1.0)))
            right = dict(heads=ssd_heads, vdim=ssd_vdim, state=state, groups=groups, conv=4, norm_groups=groups)
            out.append(dict(type="parallel", mlp=mlp, mixer=dict(left=left, right=right)))
        elif i % 8 == 7:
            m = dict(heads=lat_heads, dim=lat_dim, rot_dim=rot_dim, vdim=lat_vdim, kv_rank=kv_rank, rot=dict(base=1e4, dims=rot_dim),
                     mask=dict(size=window), scale=(lat_dim + rot_dim) ** -0.5)
            out.append(dict(type="latent_attention", mlp=mlp, mixer=m))
        else:
            out.append(dict(type="channel_delta", mlp=mlp, mixer=dict(heads=lin_heads, kv_heads=lin_heads, dim=lin_dim, vdim=lin_dim, conv=4,
                                                                      rank=rank)))
    return dict(architecture="Nikedra", layers=out, norm=dict(eps=1e-6), canon=dict(taps=4), logit_scale=1.0, vocab=vocab, width=width,
                torch_dtype="bfloat16")


# hidden size, depth, vocabulary, linear-attention heads and size of the experts of qwen3.5-moe-6b
PRESETS["nikedra-6b"] = _nikedra(24, 2048, 6144, 151936, heads=16, kv_heads=4, dim=128, chunk=4096, ssd_heads=32, ssd_vdim=64, state=128, groups=1,
                                 lin_heads=16, lin_dim=128, rank=128, lat_heads=16, lat_dim=128, rot_dim=64, lat_vdim=128, kv_rank=512, window=2048,
                                 experts=64, top=8, expert_ff=768)
PRESETS["nikedra-tiny"] = _nikedra(8, 128, 256, 1024, heads=4, kv_heads=2, dim=32, chunk=48, ssd_heads=4, ssd_vdim=16, state=32, groups=2, lin_heads=4,
                                   lin_dim=32, rank=16, lat_heads=4, lat_dim=32, rot_dim=16, lat_vdim=32, kv_rank=64, window=40, experts=6, top=2,
                                   expert_ff=64)
PRESETS["qwen2-moe-6b"] = dict(
    _dense(2048, 24, 16, 4, 6144, False), architectures=["Qwen2MoeForCausalLM"], model_type="qwen2_moe", num_experts=64, num_experts_per_tok=8,
    moe_intermediate_size=512, shared_expert_intermediate_size=512, norm_topk_prob=False, decoder_sparse_step=1, mlp_only_layers=[],
)
_VL_VISION = dict(
    depth=24, hidden_size=1024, num_heads=16, intermediate_size=4096, patch_size=16, temporal_patch_size=2,
    spatial_merge_size=2, in_channels=3, out_hidden_size=2048, num_position_embeddings=2304,
    deepstack_visual_indexes=[5, 11, 17], hidden_act="gelu_pytorch_tanh",
)
PRESETS["qwen3-vl-2b"] = dict(
    architectures=["Qwen3VLForConditionalGeneration"], model_type="qwen3_vl", tie_word_embeddings=True,
    image_token_id=151655, video_token_id=151656, vision_start_token_id=151652, vision_end_token_id=151653,
    text_config=dict(_dense(2048, 28, 16, 8, 6144, True, theta=5e6),
                     rope_scaling=dict(mrope_section=[24, 20, 20], mrope_interleaved=True, rope_type="default")),
    vision_config=_VL_VISION, torch_dtype="bfloat16", eos_token_id=151645,
)
PRESETS["qwen3-vl-tiny"] = dict(
    architectures=["Qwen3VLForConditionalGeneration"], model_type="qwen3_vl", tie_word_embeddings=True,
    image_token_id=1001, video_token_id=1002, vision_start_token_id=1003, vision_end_token_id=1004,
    text_config=dict(_dense(256, 3, 2, 1, 512, True, vocab=1024, theta=5e6),
                     rope_scaling=dict(mrope_section=[24, 20, 20], mrope_interleaved=True, rope_type="default")),
    vision_config=dict(depth=3, hidden_size=128, num_heads=2, intermediate_size=256, patch_size=16,
                       temporal_patch_size=2, spatial_merge_size=2, in_channels=3, out_hidden_size=256,
                       num_position_embeddings=64, deepstack_visual_indexes=[0, 1],
                       hidden_act="gelu_pytorch_tanh"),
    torch_dtype="bfloat16", eos_token_id=1,
)

# Qwen2-VL / Qwen2.5-VL: Qwen2 decoder (biased q / k / v, sectioned 3-D rope) behind their own vision towers
_Q2VL_IDS = dict(image_token_id=151655, video_token_id=151656, vision_start_token_id=151652, vision_end_token_id=151653)
_Q2VL_TINY_IDS = dict(image_token_id=1001, video_token_id=1002, vision_start_token_id=1003, vision_end_token_id=1004)


def _qwen2_text(hidden, layers, heads, kv, inter, tie, vocab=151936, sections=(16, 24, 24)) -> Dict[str, Any]:
    d = _dense(hidden, layers, heads, kv, inter, tie, vocab=vocab, theta=1e6)
    d.update(architectures=["Qwen2ForCausalLM"], model_type="qwen2", head_dim=hidden // heads, max_position_embeddings=32768,
             rope_scaling=dict(type="mrope", mrope_section=list(sections)))
    return d


PRESETS["qwen2-vl-2b"] = dict(
    architectures=["Qwen2VLForConditionalGeneration"], model_type="qwen2_vl", tie_word_embeddings=True, **_Q2VL_IDS,
    text_config=_qwen2_text(1536, 28, 12, 2, 8960, True),
    vision_config=dict(depth=32, embed_dim=1280, hidden_size=1536, num_heads=16, mlp_ratio=4, patch_size=14,
                       spatial_merge_size=2, temporal_patch_size=2, in_channels=3, hidden_act="quick_gelu"),
    torch_dtype="bfloat16", eos_token_id=151645,
)
PRESETS["qwen2-vl-tiny"] = dict(
    architectures=["Qwen2VLForConditionalGeneration"], model_type="qwen2_vl", tie_word_embeddings=True, **_Q2VL_TINY_IDS,
    text_config=_qwen2_text(256, 2, 4, 2, 512, True, vocab=1024, sections=(8, 12, 12)),
    vision_config=dict(depth=2, embed_dim=64, hidden_size=256, num_heads=2, mlp_ratio=2, patch_size=14,
                       spatial_merge_size=2, temporal_patch_size=2, in_channels=3, hidden_act="quick_gelu"),
    torch_dtype="bfloat16", eos_token_id=1,
)
PRESETS["qwen2.5-vl-3b"] = dict(
    architectures=["Qwen2_5_VLForConditionalGeneration"], model_type="qwen2_5_vl", tie_word_embeddings=True, **_Q2VL_IDS,
    text_config=_qwen2_text(2048, 36, 16, 2, 11008, True),
    vision_config=dict(depth=32, hidden_size=1280, hidden_act="silu", intermediate_size=3420, num_heads=16, in_channels=3,
                       patch_size=14, spatial_merge_size=2, temporal_patch_size=2, window_size=112, out_hidden_size=2048,
                       fullatt_block_indexes=[7, 15, 23, 31], tokens_per_second=2),
    torch_dtype="bfloat16", eos_token_id=151645,
)
PRESETS["qwen2.5-vl-tiny"] = dict(
    architectures=["Qwen2_5_VLForConditionalGeneration"], model_type="qwen2_5_vl", tie_word_embeddings=True, **_Q2VL_TINY_IDS,
    text_config=_qwen2_text(256, 2, 4, 2, 512, True, vocab=1024, sections=(8, 12, 12)),
    vision_config=dict(depth=3, hidden_size=64, hidden_act="silu", intermediate_size=96, num_heads=2, in_channels=3,
                       patch_size=14, spatial_merge_size=2, temporal_patch_size=2, window_size=56, out_hidden_size=256,
                       fullatt_block_indexes=[1], tokens_per_second=2),
    torch_dtype="bfloat16", eos_token_id=1,
)


def _to_ns(d: Dict[str, Any]) -> SimpleNamespace:
    ns = SimpleNamespace()
    for k, v in d.items():
        setattr(ns, k, _to_ns(v) if isinstance(v, dict) and k.endswith("_config") else copy.deepcopy(v))
    return ns


def get_preset(name: str, **overrides) -> SimpleNamespace:
    key = name.lower()
    if key not in PRESETS:
        raise KeyError(f"unknown preset {name!r}; have {sorted(PRESETS)}")
    d = copy.deepcopy(PRESETS[key])
    d.update(overrides)
    from . import get_config_adapter

    adapt = get_config_adapter(d)
    return adapt(d) if adapt is not None else _to_ns(d)


def preset_to_config_json(name: str) -> Dict[str, Any]:
    """The preset as a HF-style ``config.json`` dict (used to materialise random checkpoints)."""
    return copy.deepcopy(PRESETS[name.lower()])
