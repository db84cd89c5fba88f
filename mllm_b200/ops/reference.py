"""Plain-PyTorch statement of every op in :mod:`mllm_b200.ops`.

These functions are the numerical contract of the CUDA kernels: each kernel's
test compares against the function of the same name evaluated in fp32.  They
also run the whole engine on a machine without a GPU (CPU tests, the fp32
oracle of the Qwen3 model).  They are never used for tensors that live on a
GPU unless ``MLLM_B200_FORCE_TORCH=1`` is set for A/B comparisons.
"""

from __future__ import annotations

import math
from typing import Optional, Tuple

import torch
import torch.nn.functional as F


def _f32(x: torch.Tensor) -> torch.Tensor:
    return x.float()


# --------------------------------------------------------------------------
# normalisation / activation / embedding
# --------------------------------------------------------------------------
def rmsnorm(x: torch.Tensor, weight: torch.Tensor, eps: float, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    xf = _f32(x)
    y = xf * torch.rsqrt(xf.pow(2).mean(-1, keepdim=True) + eps) * _f32(weight)
    y = y.to(x.dtype)
    if out is not None:
        out.copy_(y)
        return out
    return y


def fused_add_rmsnorm(x: torch.Tensor, residual: torch.Tensor, weight: torch.Tensor, eps: float) -> None:
    """In place: ``residual += x`` (rounded to the storage dtype), ``x = rmsnorm(residual) * weight``."""
    s = (_f32(x) + _f32(residual)).to(residual.dtype)
    residual.copy_(s)
    x.copy_(rmsnorm(s, weight, eps))


def layernorm(x: torch.Tensor, weight: torch.Tensor, bias: Optional[torch.Tensor], eps: float) -> torch.Tensor:
    return F.layer_norm(_f32(x), (x.shape[-1],), _f32(weight), None if bias is None else _f32(bias), eps).to(x.dtype)


def silu_and_mul(x: torch.Tensor) -> torch.Tensor:
    d = x.shape[-1] // 2
    return (F.silu(_f32(x[..., :d])) * _f32(x[..., d:])).to(x.dtype)


def gelu_tanh_and_mul(x: torch.Tensor) -> torch.Tensor:
    d = x.shape[-1] // 2
    return (F.gelu(_f32(x[..., :d]), approximate="tanh") * _f32(x[..., d:])).to(x.dtype)


def gelu_tanh(x: torch.Tensor) -> torch.Tensor:
    return F.gelu(_f32(x), approximate="tanh").to(x.dtype)


def gelu_erf(x: torch.Tensor) -> torch.Tensor:
    return F.gelu(_f32(x)).to(x.dtype)


def vision_rope(x: torch.Tensor, cos: torch.Tensor, sin: torch.Tensor) -> torch.Tensor:
    """2-D rotary embedding of the vision tower: x [T, H, D], cos/sin [T, D/2] (first quarter of the
    frequencies from the row position, second from the column position); pairs (i, i + D/2)
    (pymllm/models/qwen3_vl.py:118-167)."""
    xf = _f32(x)
    half = x.shape[-1] // 2
    c, s = _f32(cos).unsqueeze(1), _f32(sin).unsqueeze(1)
    x1, x2 = xf[..., :half], xf[..., half:]
    return torch.cat([x1 * c - x2 * s, x2 * c + x1 * s], dim=-1).to(x.dtype)


def vision_pos_embed_add(x: torch.Tensor, table: torch.Tensor, idx: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """``x + sum_i w[i] * table[idx[i]]`` over the four bilinear corners (pymllm/models/qwen3_vl.py:456-491)."""
    pe = (_f32(table)[idx] * w.float().unsqueeze(-1)).sum(0)
    return (_f32(x) + pe).to(x.dtype)


def embedding(ids: torch.Tensor, table: torch.Tensor) -> torch.Tensor:
    return table[ids.long()]


# --------------------------------------------------------------------------
# GEMMs
# --------------------------------------------------------------------------
def linear(
    x: torch.Tensor,
    weight: torch.Tensor,
    bias: Optional[torch.Tensor] = None,
    residual: Optional[torch.Tensor] = None,
    out_dtype: Optional[torch.dtype] = None,
) -> torch.Tensor:
    """``x @ weight.T (+ bias) (+ residual)`` with fp32 accumulation, one rounding at the end."""
    y = _f32(x) @ _f32(weight).t()
    if bias is not None:
        y = y + _f32(bias)
    if residual is not None:
        y = y + _f32(residual)
    return y.to(out_dtype or x.dtype)


def deinterleave_gate_up(y: torch.Tensor, block: int) -> Tuple[torch.Tensor, torch.Tensor]:
    """Split the columns of a ``[.., 2I]`` tensor whose columns alternate
    ``block`` gate features, ``block`` up features, ... into (gate, up)."""
    lead = y.shape[:-1]
    v = y.reshape(*lead, -1, 2, block)
    return v[..., 0, :].reshape(*lead, -1), v[..., 1, :].reshape(*lead, -1)


def interleave_gate_up(w: torch.Tensor, block: int) -> torch.Tensor:
    """Rows ``[gate(I) ; up(I)]`` -> rows alternating ``block`` gate, ``block`` up."""
    i = w.shape[0] // 2
    g = w[:i].reshape(i // block, 1, block, *w.shape[1:])
    u = w[i:].reshape(i // block, 1, block, *w.shape[1:])
    return torch.cat([g, u], dim=1).reshape(w.shape)


def clamped_gate(gate: torch.Tensor, up: torch.Tensor, limit: float) -> torch.Tensor:
    """Gated unit with bounds: ``g = min(gate, limit)``, ``u = clamp(up, -limit, limit)``, ``g * sigmoid(1.702 g) * (u + 1)``."""
    g, u = _f32(gate).clamp(max=limit), _f32(up).clamp(-limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)).to(gate.dtype)


def linear_swiglu(x: torch.Tensor, weight: torch.Tensor, block: int = 0, act: str = "silu", bias: Optional[torch.Tensor] = None,
                  limit: float = 0.0) -> torch.Tensor:
    """``act(x Wg^T) * (x Wu^T)``; ``block`` = row interleave of ``weight`` (0: ``[gate ; up]``) and of ``bias``."""
    y = _f32(x) @ _f32(weight).t()
    if bias is not None:
        y = y + _f32(bias)
    if block:
        g, u = deinterleave_gate_up(y, block)
    else:
        d = y.shape[-1] // 2
        g, u = y[..., :d], y[..., d:]
    if act == "clamped":
        return clamped_gate(g, u, limit).to(x.dtype)
    return ((F.gelu(g, approximate="tanh") if act == "gelu_tanh" else F.silu(g)) * u).to(x.dtype)


def per_token_quant_int8(x: torch.Tensor) -> Tuple[torch.Tensor, torch.Tensor]:
    """Symmetric per-row int8: ``scale = absmax/127``, ``q = round(x/scale)``."""
    xf = _f32(x)
    absmax = xf.abs().amax(-1, keepdim=True).clamp_min(1e-10)
    scale = absmax / 127.0
    q = torch.round(xf / scale).clamp(-128, 127).to(torch.int8)
    return q, scale.float()


def int8_scaled_mm(
    a_q: torch.Tensor, w_q: torch.Tensor, a_scale: torch.Tensor, w_scale: torch.Tensor,
    out_dtype: torch.dtype, bias: Optional[torch.Tensor] = None,
) -> torch.Tensor:
    """``(a_q @ w_q.T) * a_scale[M,1] * w_scale[N]`` with exact int32 accumulation."""
    acc = (a_q.to(torch.int32).cpu() @ w_q.to(torch.int32).cpu().t()).to(a_q.device) if a_q.is_cuda else (
        a_q.to(torch.int32) @ w_q.to(torch.int32).t())
    y = acc.float() * a_scale.reshape(-1, 1).float() * w_scale.reshape(1, -1).float()
    if bias is not None:
        y = y + _f32(bias)
    return y.to(out_dtype)


def unpack_int4_rows(packed: torch.Tensor) -> torch.Tensor:
    """int32 ``[N, K/8]`` (nibble i of word j = element 8j+i) -> uint8-valued ``[N, K]`` in 0..15."""
    shifts = torch.arange(0, 32, 4, device=packed.device, dtype=torch.int32)
    return ((packed.unsqueeze(-1) >> shifts) & 0xF).reshape(packed.shape[0], -1)


def dequant_w4(qweight: torch.Tensor, scales: torch.Tensor, zeros: Optional[torch.Tensor], group: int) -> torch.Tensor:
    """``qweight`` int32 ``[N, K/8]``, ``scales`` ``[N, K/g]``, ``zeros`` uint8-valued ``[N, K/g]`` or
    None (symmetric, zero point 8) -> fp32 ``[N, K]``."""
    q = unpack_int4_rows(qweight).float()
    s = scales.float().repeat_interleave(group, dim=1)
    z = 8.0 if zeros is None else zeros.float().repeat_interleave(group, dim=1)
    return (q - z) * s


def w4a16_gemm(x, qweight, scales, zeros, group: int, bias=None) -> torch.Tensor:
    y = _f32(x) @ dequant_w4(qweight, scales, zeros, group).t()
    if bias is not None:
        y = y + _f32(bias)
    return y.to(x.dtype)


# --------------------------------------------------------------------------
# rotary embedding, QK-norm, cache write
# --------------------------------------------------------------------------
def rope_cos_sin(positions: torch.Tensor, head_dim: int, theta: float, rotary_dim: Optional[int] = None,
                 inv_freq: Optional[torch.Tensor] = None):
    rd = rotary_dim or head_dim
    inv = inv_freq.to(positions.device) if inv_freq is not None else \
        1.0 / (theta ** (torch.arange(0, rd, 2, device=positions.device, dtype=torch.float32) / rd))
    ang = positions.float().unsqueeze(-1) * inv  # [..., rd/2]
    return ang.cos(), ang.sin()


def apply_rope_neox(x: torch.Tensor, cos: torch.Tensor, sin: torch.Tensor) -> torch.Tensor:
    """x: [T, H, D] fp32; cos/sin: [T, rd/2]; rotates the first ``rd`` features (half-split pairing)."""
    half = cos.shape[-1]
    x1, x2, rest = x[..., :half], x[..., half : 2 * half], x[..., 2 * half :]
    c, s = cos.unsqueeze(1), sin.unsqueeze(1)
    return torch.cat([x1 * c - x2 * s, x2 * c + x1 * s, rest], dim=-1)


def mrope_cos_sin(positions3: torch.Tensor, head_dim: int, theta: float, sections, interleaved: bool):
    """positions3: [3, T] (t, h, w).  Returns cos/sin [T, D/2] whose frequency
    index i takes its position from axis ``a(i)``: consecutive sections
    ``[t]*s0 + [h]*s1 + [w]*s2`` or, when ``interleaved``, ``a(i) = i % 3`` for
    ``i < 3*s1`` / ``3*s2`` (h, w) and t elsewhere (pymllm/layers/rope.py:320-408)."""
    half = head_dim // 2
    inv = 1.0 / (theta ** (torch.arange(0, head_dim, 2, device=positions3.device, dtype=torch.float32) / head_dim))
    ang = positions3.float().unsqueeze(-1) * inv  # [3, T, half]
    axis = torch.zeros(half, dtype=torch.long, device=positions3.device)
    if interleaved:
        idx = torch.arange(half, device=positions3.device)
        axis[(idx % 3 == 1) & (idx < 3 * sections[1])] = 1
        axis[(idx % 3 == 2) & (idx < 3 * sections[2])] = 2
    else:
        axis[sections[0] : sections[0] + sections[1]] = 1
        axis[sections[0] + sections[1] : sections[0] + sections[1] + sections[2]] = 2
    sel = ang.permute(1, 2, 0).gather(-1, axis.view(1, half, 1).expand(ang.shape[1], half, 1)).squeeze(-1)
    return sel.cos(), sel.sin()


def qk_norm_rope_kv_write(
    qkv: torch.Tensor, q_weight: Optional[torch.Tensor], k_weight: Optional[torch.Tensor],
    positions: torch.Tensor, cache_loc: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor,
    num_q_heads: int, num_kv_heads: int, head_dim: int, theta: float, eps: float,
    mrope_sections=None, mrope_interleaved: bool = False, inv_freq: Optional[torch.Tensor] = None,
) -> None:
    """In place on ``qkv`` ``[T, (Hq+2Hkv)*D]``: per-head RMSNorm of q and k (if weights
    given), NeoX RoPE at ``positions`` (``[T]``, or ``[3,T]`` with ``mrope_sections``); then
    ``k_cache[cache_loc] = k`` (normed, rotated) and ``v_cache[cache_loc] = v``."""
    T = qkv.shape[0]
    qd, kd = num_q_heads * head_dim, num_kv_heads * head_dim
    q = _f32(qkv[:, :qd]).reshape(T, num_q_heads, head_dim)
    k = _f32(qkv[:, qd : qd + kd]).reshape(T, num_kv_heads, head_dim)
    v = qkv[:, qd + kd :].reshape(T, num_kv_heads, head_dim)
    if q_weight is not None:
        q = q * torch.rsqrt(q.pow(2).mean(-1, keepdim=True) + eps) * _f32(q_weight)
        q = q.to(qkv.dtype).float()
    if k_weight is not None:
        k = k * torch.rsqrt(k.pow(2).mean(-1, keepdim=True) + eps) * _f32(k_weight)
        k = k.to(qkv.dtype).float()
    if mrope_sections is not None:
        cos, sin = mrope_cos_sin(positions, head_dim, theta, mrope_sections, mrope_interleaved)
    else:
        cos, sin = rope_cos_sin(positions, head_dim, theta, inv_freq=inv_freq)
    q = apply_rope_neox(q, cos, sin).to(qkv.dtype)
    k = apply_rope_neox(k, cos, sin).to(qkv.dtype)
    qkv[:, :qd] = q.reshape(T, qd)
    qkv[:, qd : qd + kd] = k.reshape(T, kd)
    loc = cache_loc.long()
    k_cache[loc] = k.to(k_cache.dtype)
    v_cache[loc] = v.to(v_cache.dtype)


def kv_write(k, v, loc, k_cache, v_cache) -> None:
    """k, v: [T, Hkv * D] or [T, Hkv, D] rows written to the cache slots ``loc``."""
    k_cache[loc.long()] = k.reshape(k.shape[0], *k_cache.shape[1:]).to(k_cache.dtype)
    v_cache[loc.long()] = v.reshape(v.shape[0], *v_cache.shape[1:]).to(v_cache.dtype)


def create_kv_indices(req_to_token: torch.Tensor, req_pool_indices: torch.Tensor, seq_lens: torch.Tensor,
                      kv_start: Optional[torch.Tensor] = None, max_len: Optional[int] = None):
    """Flat KV index list of a batch, as paged-attention libraries want it (role of mllm-kernel's
    ``create_kv_indices``): ``kv_indices[kv_indptr[b] + j] = req_to_token[req_pool_indices[b], kv_start[b] + j]``
    for ``j < seq_lens[b]``.  Returns ``(kv_indptr int32 [B + 1], kv_indices int32 [sum(seq_lens)])``.  The
    attention kernels of this package read ``req_to_token`` directly and do not need it."""
    lens = seq_lens.to(torch.int64)
    B = lens.numel()
    indptr = torch.zeros(B + 1, dtype=torch.int32, device=lens.device)
    indptr[1:] = torch.cumsum(lens, 0).to(torch.int32)
    width = int(max_len if max_len is not None else (int(lens.max()) if B else 0))
    j = torch.arange(width, device=lens.device).unsqueeze(0)
    start = kv_start.to(torch.int64).view(-1, 1) if kv_start is not None else 0
    cols = (j + start).clamp_(max=req_to_token.shape[1] - 1)
    rows = req_to_token[req_pool_indices.long().view(-1, 1), cols]
    return indptr, rows[j < lens.view(-1, 1)].to(torch.int32)


# --------------------------------------------------------------------------
# attention over the slot-indexed KV pool
# --------------------------------------------------------------------------
def _attend(q, k, v, scale, causal_offset: Optional[int], window: Optional[int] = None, logit_cap: float = 0.0, sink=None,
            chunk: Optional[int] = None):
    """q [Tq,Hq,D] k,v [Tk,Hkv,D] fp32 -> [Tq,Hq,D]; key j visible to query i iff j <= i + causal_offset and,
    with a sliding ``window``, j > i + causal_offset - window (the last ``window`` keys, the query's own
    included); with ``chunk``, keys before the start of the query's chunk of positions are hidden too.  ``sink`` [Hq]: one more softmax term per head, without a value.  ``logit_cap`` > 0 soft-caps the scaled scores: ``cap * tanh(s / cap)``."""
    Hq, Hkv = q.shape[1], k.shape[1]
    g = Hq // Hkv
    kk = k.repeat_interleave(g, dim=1)
    vv = v.repeat_interleave(g, dim=1)
    s = torch.einsum("qhd,khd->hqk", q, kk) * scale
    if logit_cap and logit_cap > 0:
        s = logit_cap * torch.tanh(s / logit_cap)
    if causal_offset is not None or window or chunk:
        off = causal_offset if causal_offset is not None else k.shape[0] - q.shape[0]
        i = torch.arange(q.shape[0], device=q.device).unsqueeze(-1)
        j = torch.arange(k.shape[0], device=q.device).unsqueeze(0)
        hidden = j > i + off if causal_offset is not None else torch.zeros_like(j > i)
        if window:
            hidden = hidden | (j <= i + off - int(window))
        elif chunk:
            hidden = hidden | (j < (i + off) // int(chunk) * int(chunk))
        s = s.masked_fill(hidden, float("-inf"))
    p = sink_softmax(s, sink)
    return torch.einsum("hqk,khd->qhd", p, vv)


def _attend_sdpa(q, k, v, scale, causal_offset: Optional[int], window: Optional[int] = None):
    """:func:`_attend` through ``scaled_dot_product_attention`` in the tensors' own dtype (no fp32 score
    matrix): the fallback used on GPUs for head sizes without a kernel.  q [Tq,Hq,D], k / v [Tk,Hkv,D]."""
    import torch.nn.functional as F

    Tq, Tk = q.shape[0], k.shape[0]
    qh, kh, vh = q.transpose(0, 1).unsqueeze(0), k.transpose(0, 1).unsqueeze(0), v.transpose(0, 1).unsqueeze(0)
    mask, causal = None, False
    if causal_offset is not None:
        if causal_offset == 0 and Tq == Tk and not window:
            causal = True
        else:
            i = torch.arange(Tq, device=q.device).unsqueeze(-1)
            j = torch.arange(Tk, device=q.device).unsqueeze(0)
            mask = j <= i + causal_offset
            if window:
                mask = mask & (j > i + causal_offset - int(window))
    o = F.scaled_dot_product_attention(qh, kh, vh, attn_mask=mask, is_causal=causal, scale=scale,
                                       enable_gqa=q.shape[1] != k.shape[1])
    return o.squeeze(0).transpose(0, 1)


def attention_prefill(
    q: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, req_to_token: torch.Tensor,
    req_pool_indices: torch.Tensor, seq_lens: torch.Tensor, prefix_lens: torch.Tensor,
    q_start_loc: torch.Tensor, scale: float, out: Optional[torch.Tensor] = None, max_q_len: int = 0,
    window: Optional[int] = None, logit_cap: float = 0.0, sink: Optional[torch.Tensor] = None, chunk: Optional[int] = None,
) -> torch.Tensor:
    """Causal attention of each request's new tokens over its cached prefix plus itself.

    Request ``b`` owns query rows ``q_start_loc[b] .. +seq_lens[b]-prefix_lens[b]``; its keys
    are the slots ``req_to_token[req_pool_indices[b], :seq_lens[b]]``; query ``i`` sees keys
    ``0 .. prefix_lens[b]+i``."""
    out = torch.empty_like(q) if out is None else out
    for b in range(req_pool_indices.numel()):
        sl, pl, qs = int(seq_lens[b]), int(prefix_lens[b]), int(q_start_loc[b])
        n = sl - pl
        slots = req_to_token[int(req_pool_indices[b]), :sl].long()
        o = _attend(_f32(q[qs : qs + n]), _f32(k_cache[slots]), _f32(v_cache[slots]), scale, pl, window, logit_cap, sink, chunk)
        out[qs : qs + n] = o.to(out.dtype)
    return out


def attention_prefill_sdpa(q, k_cache, v_cache, req_to_token, req_pool_indices, seq_lens, prefix_lens, q_start_loc,
                           scale: float, seq_lens_cpu=None, prefix_lens_cpu=None, window: Optional[int] = None) -> torch.Tensor:
    """:func:`attention_prefill` with ``scaled_dot_product_attention`` per request in the activation dtype —
    not a numerical reference but the serving fallback on GPUs for head sizes without a kernel.  The host
    copies of the lengths avoid device read-backs."""
    out = torch.empty_like(q)
    sls = seq_lens_cpu if seq_lens_cpu is not None else seq_lens.tolist()
    pls = prefix_lens_cpu if prefix_lens_cpu is not None else prefix_lens.tolist()
    qs = 0
    pools = req_pool_indices.long()
    for b, (sl, pl) in enumerate(zip(sls, pls)):
        n = int(sl) - int(pl)
        slots = req_to_token[pools[b], : int(sl)].long()
        out[qs : qs + n] = _attend_sdpa(q[qs : qs + n], k_cache[slots].to(q.dtype), v_cache[slots].to(q.dtype), scale, int(pl), window)
        qs += n
    return out


def attention_decode(
    q: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, req_to_token: torch.Tensor,
    req_pool_indices: torch.Tensor, seq_lens: torch.Tensor, scale: float, out: Optional[torch.Tensor] = None,
    window: Optional[int] = None, logit_cap: float = 0.0, sink: Optional[torch.Tensor] = None, chunk: Optional[int] = None,
) -> torch.Tensor:
    """One query token per request over ``req_to_token[req, :seq_len]`` (the new token's K/V included)."""
    out = torch.empty_like(q) if out is None else out
    for b in range(req_pool_indices.numel()):
        sl = int(seq_lens[b])
        slots = req_to_token[int(req_pool_indices[b]), :sl].long()
        o = _attend(_f32(q[b : b + 1]), _f32(k_cache[slots]), _f32(v_cache[slots]), scale, None, window, logit_cap, sink, chunk)
        out[b] = o[0].to(out.dtype)
    return out


def attention_decode_batched(
    q: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, req_to_token: torch.Tensor,
    req_pool_indices: torch.Tensor, seq_lens: torch.Tensor, scale: float, max_seq_len: int,
    out: Optional[torch.Tensor] = None, window: Optional[int] = None, logit_cap: float = 0.0,
) -> torch.Tensor:
    """:func:`attention_decode` for the whole batch at once: keys are gathered up to ``max_seq_len`` (a host
    bound on ``seq_lens``) and the tail of every request is masked, so nothing is read back from the device.
    Used on GPUs for head sizes the decode kernel does not cover."""
    B, Hq, D = q.shape
    Hkv = k_cache.shape[1]
    S = int(max_seq_len)
    slots = req_to_token[req_pool_indices.long(), :S].long()                  # [B, S]
    k = _f32(k_cache[slots])                                                  # [B, S, Hkv, D]
    v = _f32(v_cache[slots])
    qg = _f32(q).view(B, Hkv, Hq // Hkv, D)
    s = torch.einsum("bhgd,bshd->bhgs", qg, k) * scale
    if logit_cap and logit_cap > 0:
        s = logit_cap * torch.tanh(s / logit_cap)
    pos = torch.arange(S, device=q.device).unsqueeze(0)
    valid = pos < seq_lens.view(-1, 1)
    if window:
        valid = valid & (pos >= seq_lens.view(-1, 1) - int(window))
    s = s.masked_fill(~valid.view(B, 1, 1, S), float("-inf"))
    o = torch.einsum("bhgs,bshd->bhgd", torch.softmax(s, dim=-1), v).reshape(B, Hq, D)
    if out is None:
        return o.to(q.dtype)
    out.copy_(o)
    return out


def attention_varlen_bidirectional(q, k, v, cu_seqlens, scale) -> torch.Tensor:
    """Full (non-causal) attention inside each segment ``cu_seqlens[i]..cu_seqlens[i+1]``; q,k,v [T,H,D]."""
    out = torch.empty_like(q)
    cu = cu_seqlens.tolist()
    for a, b in zip(cu[:-1], cu[1:]):
        out[a:b] = _attend(_f32(q[a:b]), _f32(k[a:b]), _f32(v[a:b]), scale, None).to(q.dtype)
    return out


# --------------------------------------------------------------------------
# sampling
# --------------------------------------------------------------------------
def argmax(logits: torch.Tensor) -> torch.Tensor:
    return torch.argmax(logits.float(), dim=-1)


def apply_penalties(logits, output_counts, prompt_mask, frequency_penalty, presence_penalty, repetition_penalty):
    """OpenAI-style frequency/presence penalties on generated-token counts and HF-style
    repetition penalty on tokens seen in prompt or output.  All per-request vectors are [B]."""
    lf = logits.float()
    seen_out = output_counts > 0
    lf = lf - frequency_penalty.view(-1, 1) * output_counts.float() - presence_penalty.view(-1, 1) * seen_out.float()
    seen = seen_out | prompt_mask
    rp = repetition_penalty.view(-1, 1)
    lf = torch.where(seen, torch.where(lf > 0, lf / rp, lf * rp), lf)
    return lf


def top_k_top_p_min_p_sample(
    logits: torch.Tensor, temperature: torch.Tensor, top_k: torch.Tensor, top_p: torch.Tensor,
    min_p: Optional[torch.Tensor], uniform: torch.Tensor,
) -> torch.Tensor:
    """Sample one id per row.  ``temperature <= 1e-6`` rows are greedy; ``top_k <= 0`` disables top-k.

    With ``e = exp((logits - max) / T)`` every filter is a cut-off on ``e`` (values equal to the cut-off
    are all kept): top-k keeps ``e >= k-th largest``; top-p keeps the values whose strictly-larger mass
    is below ``top_p * sum(e)``; min-p keeps ``e >= min_p`` (the largest ``e`` is 1).  ``uniform`` [B]
    in [0,1) drives inverse-CDF sampling over the kept set in token-id order: the first id whose running
    kept mass exceeds ``u * kept_mass``."""
    B, V = logits.shape
    out = torch.empty(B, dtype=torch.long, device=logits.device)
    for b in range(B):
        t = float(temperature[b])
        row = logits[b].float()
        if t <= 1e-6:
            out[b] = torch.argmax(row)
            continue
        e = torch.exp((row - row.max()) / t).double()
        tau = 0.0
        k = int(top_k[b])
        se = torch.sort(e, descending=True).values
        if 0 < k < V:
            tau = max(tau, float(se[k - 1]))
        tp = float(top_p[b])
        if tp < 1.0:
            before = torch.cumsum(se, 0) - se
            n = int((before < max(tp * float(se.sum()), 1e-30)).sum())
            tau = max(tau, float(se[max(n, 1) - 1]))
        if min_p is not None and float(min_p[b]) > 0:
            tau = max(tau, min(float(min_p[b]), 1.0))
        kept = torch.where(e >= tau, e, torch.zeros_like(e))
        cdf = torch.cumsum(kept, 0)
        target = float(uniform[b]) * float(cdf[-1])
        idx = int((cdf > target).nonzero()[0]) if bool((cdf > target).any()) else int((kept > 0).nonzero()[-1])
        out[b] = idx
    return out


# --------------------------------------------------------------------------
# mixture of experts
# --------------------------------------------------------------------------
def moe_router_topk(hidden: torch.Tensor, gate_weight: torch.Tensor, top_k: int, renormalize: bool = True,
                    correction: Optional[torch.Tensor] = None, renorm_eps: float = 0.0, sigmoid: bool = False, groups: int = 1,
                    keep: int = 1, scale: float = 1.0):
    """fp32 ``softmax(hidden @ gate_weight.T)`` over all experts -> top-k (sorted by weight) ->
    optional renormalisation of the k weights (mllm/models/qwen3_moe/modeling_qwen3_moe_fa2.hpp:121-138).
    With ``correction`` the choice goes by ``scores + correction``, the weights are the scores alone.  ``sigmoid``: the
    scores are logistic functions of the logits.  ``keep`` < ``groups``: only experts of the ``keep`` groups of neighbours
    with the largest sums of their two largest choice scores.  ``scale``: factor of the weights.
    Returns (weights fp32 [T, k], expert ids int32 [T, k])."""
    logits = _f32(hidden) @ _f32(gate_weight).t()
    scores = torch.sigmoid(logits) if sigmoid else torch.softmax(logits, dim=-1)
    choice = scores if correction is None else scores + _f32(correction)
    if keep < groups:
        by_group = choice.unflatten(-1, (groups, -1))
        best = by_group.topk(min(2, by_group.shape[-1]), dim=-1).values.sum(-1).topk(keep, dim=-1).indices
        closed = torch.ones_like(by_group[..., 0], dtype=torch.bool).scatter_(-1, best, False)
        choice = by_group.masked_fill(closed.unsqueeze(-1), float("-inf")).flatten(-2)
    idx = torch.topk(choice, top_k, dim=-1, sorted=True).indices
    w = scores.gather(-1, idx)
    if renormalize:
        w = w / (w.sum(-1, keepdim=True) + renorm_eps)
    return w * scale, idx.to(torch.int32)


def moe_experts(x: torch.Tensor, w13: torch.Tensor, w2: torch.Tensor, topk_w: torch.Tensor, topk_ids: torch.Tensor,
                expert_offset: int = 0, swiglu_block: int = 0) -> torch.Tensor:
    """Sum over the k routed experts of ``w * down_e(silu(gate_e(x)) * up_e(x))``.

    ``w13`` [E_local, 2I, H] (rows ``[gate ; up]``, or interleaved in ``swiglu_block`` rows), ``w2``
    [E_local, H, I]; expert ids outside ``[expert_offset, expert_offset + E_local)`` contribute
    nothing (they live on another expert-parallel rank)."""
    T, H = x.shape
    out = torch.zeros((T, H), dtype=torch.float32, device=x.device)
    E = w13.shape[0]
    for e in range(E):
        tok, slot = (topk_ids == (e + expert_offset)).nonzero(as_tuple=True)
        if tok.numel() == 0:
            continue
        h = linear_swiglu(x[tok], w13[e], swiglu_block)
        y = linear(h, w2[e], out_dtype=torch.float32)
        out.index_add_(0, tok, y * topk_w[tok, slot].unsqueeze(-1).float())
    return out.to(x.dtype)


def moe_expert_rows(x, w13, w2, topk_ids, swiglu_block: int = 0, gated: bool = True, input_w: Optional[torch.Tensor] = None):
    """Outputs of the chosen experts, a row per (token, choice), and the row of every pair (-1: no such expert)."""
    T, k = topk_ids.shape
    rows = torch.zeros((T * k, x.shape[1]), dtype=x.dtype, device=x.device)
    for e in range(w13.shape[0]):
        tok, slot = (topk_ids == e).nonzero(as_tuple=True)
        if tok.numel():
            xe = x[tok] if input_w is None else (_f32(x[tok]) * input_w[tok, slot].unsqueeze(-1)).to(x.dtype)
            h = linear_swiglu(xe, w13[e], swiglu_block) if gated else F.gelu(_f32(linear(xe, w13[e], out_dtype=torch.float32))).to(x.dtype)
            rows[tok * k + slot] = linear(h, w2[e])
    flat = topk_ids.reshape(-1)
    pos = torch.arange(T * k, dtype=torch.int32, device=x.device)
    return rows, torch.where((flat >= 0) & (flat < w13.shape[0]), pos, torch.full_like(pos, -1))


# --------------------------------------------------------------------------
# fp32 residual stream, norms after the sum, Dynamic Tanh, latent attention
# --------------------------------------------------------------------------
def post_norm(x, y, ls, alpha, weight, eps, dtype, update=True, experts=None, inner=False, y_logit=None):
    z = torch.zeros_like(x) if y is None else _f32(y)
    if y_logit is not None:
        z = z * torch.sigmoid(y_logit).unsqueeze(-1)
    if experts is not None:
        T, k = experts.topk_w.shape
        pos = experts.sorted_pos[: T * k].view(T, k).long()
        w = _f32(experts.topk_w)
        part = torch.where((pos >= 0).unsqueeze(-1), _f32(experts.rows)[pos.clamp(min=0)], torch.zeros((), device=x.device))
        z = z + (part * w.unsqueeze(-1)).sum(1)
        if experts.identity_from > 0:
            z = z + _f32(experts.token_in) * (w * (experts.ids >= experts.identity_from)).sum(1, keepdim=True)

    def norm(t):
        return t * torch.rsqrt(t.pow(2).mean(-1, keepdim=True) + eps) * _f32(weight)

    if inner:
        z = norm(z)
    z = float(alpha) * x + (z if ls is None else _f32(ls) * z)
    if not inner:
        z = norm(z)
    if update:
        x.copy_(z)
    return z.to(dtype)


def rmsnorm_sigmoid_gate(x, gate, weight, eps):
    xf = _f32(x)
    return (xf * torch.rsqrt(xf.pow(2).mean(-1, keepdim=True) + eps) * _f32(weight) * torch.sigmoid(_f32(gate))).to(x.dtype)


def rotate_pairs(x: torch.Tensor, positions: torch.Tensor, inv_freq: torch.Tensor) -> torch.Tensor:
    """x [T, H, D] fp32: neighbouring features (2i, 2i + 1) turn by ``positions * inv_freq[i]``, later ones stay."""
    n = inv_freq.numel()
    a = (positions.double().unsqueeze(-1) * inv_freq.double()).unsqueeze(1)
    c, s = torch.cos(a).float(), torch.sin(a).float()
    u, v = x[..., 0:2 * n:2], x[..., 1:2 * n:2]
    turned = torch.stack([u * c - v * s, v * c + u * s], -1).flatten(-2)
    return torch.cat([turned, x[..., 2 * n:]], -1)


def rownorm_rope_kv(row, q_w, k_w, inv_freq, positions, loc, q_out, k_cache, v_cache, heads, kv_heads, dim, vdim, eps):
    T, nq, nk = row.shape[0], heads * dim, kv_heads * dim

    def norm(t, w):
        t = _f32(t)
        return t * torch.rsqrt(t.pow(2).mean(-1, keepdim=True) + eps) * _f32(w)

    q = rotate_pairs(norm(row[:, :nq], q_w).view(T, heads, dim), positions, inv_freq)
    k = rotate_pairs(norm(row[:, nq:nq + nk], k_w).view(T, kv_heads, dim), positions, inv_freq)
    q_out.zero_()
    q_out[..., :dim] = q.to(q_out.dtype)
    k_cache[loc.long(), :, :dim] = k.to(k_cache.dtype)
    v_cache[loc.long(), :, :vdim] = row[:, nq + nk:nq + nk + kv_heads * vdim].reshape(T, kv_heads, vdim)


def rotate_halves(x: torch.Tensor, positions: torch.Tensor, inv_freq: torch.Tensor) -> torch.Tensor:
    """x [T, H, D] fp32: features i and i + n, n frequencies, turn by ``positions * inv_freq[i]``, later ones stay."""
    n = inv_freq.numel()
    a = (positions.double().unsqueeze(-1) * inv_freq.double()).unsqueeze(1)
    c, s = torch.cos(a).float(), torch.sin(a).float()
    u, v = x[..., :n], x[..., n:2 * n]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * n:]], -1)


def headnorm_rope_kv(row, inv_freq, positions, loc, q_out, k_cache, v_cache, heads, kv_heads, dim, vdim, v_at, halves, eps, norm=True,
                     magnitude=1.0):
    T, turn, R = row.shape[0], rotate_halves if halves else rotate_pairs, 2 * inv_freq.numel()

    def head(t, n):
        t = turn(_f32(t).reshape(T, n, dim), positions, inv_freq)
        t = torch.cat([t[..., :R] * magnitude, t[..., R:]], -1)
        return t * torch.rsqrt(t.pow(2).mean(-1, keepdim=True) + eps) if norm else t

    q_out.zero_()
    q_out[..., :dim] = head(row[:, : heads * dim], heads).to(q_out.dtype)
    k_cache[loc.long(), :, :dim] = head(row[:, heads * dim: (heads + kv_heads) * dim], kv_heads).to(k_cache.dtype)
    v_cache[loc.long(), :, :vdim] = row[:, v_at: v_at + kv_heads * vdim].reshape(T, kv_heads, vdim)


def gated_rmsnorm(x, gate, weight, groups, eps):
    z = (_f32(x) * F.silu(_f32(gate))).unflatten(-1, (groups, -1))
    z = (z * torch.rsqrt(z.pow(2).mean(-1, keepdim=True) + eps)).flatten(-2)
    return (z * _f32(weight)).to(x.dtype)


def _depth_inputs(x, norms, eps, dtype, conv):
    r = torch.rsqrt(x.pow(2).mean(-1, keepdim=True) + eps)
    h = [(x * r * _f32(g)).to(dtype) for g in norms]
    if conv is not None:        # every row is the next token of the request with state row slots[t]
        at = conv.slots.long()
        seq = torch.cat([conv.state[at], h[0].unsqueeze(-1)], -1)
        h[0] = (_f32(h[0]) + (_f32(seq) * _f32(conv.weight)).sum(-1)).to(dtype)
        conv.state[at] = seq[..., 1:]
    return h


def depth_step(x, mix, f, experts, results, n, dwa, norms, eps, dtype, x_out, keep=True, mix_scale=0.5, conv=None):
    def norm(t, w):
        t = _f32(t)
        return t * torch.rsqrt(t.pow(2).mean(-1, keepdim=True) + eps) * _f32(w)

    z = _f32(mix[0]) if len(mix) == 1 else mix_scale * (norm(mix[0], mix[2]) + norm(mix[1], mix[3]))
    if f is not None:
        z = z + _f32(f)
    if experts is not None:
        T, k = experts.ids.shape
        pos = experts.sorted_pos[: T * k].view(T, k).long()
        part = torch.where((pos >= 0).unsqueeze(-1), _f32(experts.rows)[pos.clamp(min=0)], torch.zeros((), device=x.device))
        z = z + (part if experts.topk_w is None else part * _f32(experts.topk_w).unsqueeze(-1)).sum(1)
    z = x + z
    out = z
    if dwa is not None:
        if keep:
            results[n] = z
        out = dwa[n] * z
        for j in range(n):
            out = out + dwa[j] * results[j]
    if x_out is not None:
        x_out.copy_(out)
    return _depth_inputs(out, norms, eps, dtype, conv)


def embed_norm(ids, table, weight, x, eps, norms, conv=None):
    e = _f32(embedding(ids, table)).view(x.shape)
    x.copy_(e * torch.rsqrt(e.pow(2).mean(-1, keepdim=True) + eps) * _f32(weight))
    return _depth_inputs(x, norms, eps, table.dtype, conv)


def soft_cap(x, cap):
    return torch.tanh(_f32(x) / cap) * cap


def relu_squared(x):
    return x.copy_(torch.relu(x) ** 2)


def attention_rows(q, k_cache, v_cache, req_to_token, row_req, row_pos, scale, out, window=0, logit_cap=0.0, sink=None, chunk=0):
    rep = q.shape[1] // k_cache.shape[1]
    for t in range(q.shape[0]):
        pos = int(row_pos[t])
        lo = max(0, pos - window + 1) if window else pos // chunk * chunk if chunk else 0
        slots = req_to_token[int(row_req[t]), lo: pos + 1].long()
        k = _f32(k_cache[slots]).repeat_interleave(rep, 1)                 # [n, H, D]
        v = _f32(v_cache[slots]).repeat_interleave(rep, 1)
        s = torch.einsum("hd,nhd->hn", _f32(q[t]), k) * scale
        if logit_cap:
            s = logit_cap * torch.tanh(s / logit_cap)
        out[t] = torch.einsum("hn,nhd->hd", sink_softmax(s, sink), v).to(q.dtype)
    return out


def lightning_attention(q, k, v, decay, state, state_indices, seq_lens, has_state):
    """q, k [T, H, D], v [T, H, Dv] before their SiLU; the state rows are read where ``has_state`` and written back."""
    q, k, v = (_f32(torch.nn.functional.silu(_f32(t)).to(t.dtype)) for t in (q, k, v))
    out = torch.empty(v.shape, dtype=torch.float32, device=v.device)
    g, at = _f32(decay).view(-1, 1, 1), 0
    for slot, n, has in zip(state_indices.tolist(), seq_lens, has_state):
        S = state[slot].clone() if has else torch.zeros_like(state[slot])
        for t in range(at, at + n):
            S = g * S + k[t].unsqueeze(-1) * v[t].unsqueeze(-2)
            out[t] = (S * q[t].unsqueeze(-1)).sum(-2)
        state[slot] = S
        at += n
    return out


def state_space(x, B, C, dt, dt_bias, a_log, skip, state, state_indices, seq_lens, has_state):
    """x [T, H, P], B and C [T, G, N] activated, dt [T, H] raw; the state rows [H, N, P] are read where ``has_state`` and written
    back."""
    H = x.shape[1]
    xf, B, C = _f32(x), _f32(B).repeat_interleave(H // B.shape[1], 1), _f32(C).repeat_interleave(H // C.shape[1], 1)
    step = F.softplus(_f32(dt) + _f32(dt_bias))                                  # [T, H]
    decay = torch.exp(-torch.exp(_f32(a_log)) * step)
    out, at = torch.empty(x.shape, dtype=torch.float32, device=x.device), 0
    for slot, n, has in zip(state_indices.tolist(), seq_lens, has_state):
        S = state[slot].clone() if has else torch.zeros_like(state[slot])
        for t in range(at, at + n):
            S = decay[t].view(-1, 1, 1) * S + B[t].unsqueeze(-1) * (step[t].unsqueeze(-1) * xf[t]).unsqueeze(-2)
            out[t] = (S * C[t].unsqueeze(-1)).sum(-2) + _f32(skip).unsqueeze(-1) * xf[t]
        state[slot] = S
        at += n
    return out


def channel_delta_rule(q, k, v, b, a, a_log, dt_bias, state, state_indices, seq_lens, has_state):
    """q, k [T, H, Dk], v [T, H, Dv], b [T, H], a [T, H * Dk] raw; the state rows [H, Dk, Dv] are read where ``has_state`` and
    written back."""
    T, H, Dk = q.shape
    qf, kf, vf = _f32(q), _f32(k), _f32(v)
    qf = qf * torch.rsqrt((qf * qf).sum(-1, keepdim=True) + 1e-6) * Dk ** -0.5
    kf = kf * torch.rsqrt((kf * kf).sum(-1, keepdim=True) + 1e-6)
    decay = torch.exp(-torch.exp(_f32(a_log)).view(1, H, 1) * F.softplus(_f32(a) + _f32(dt_bias)).view(T, H, Dk))
    beta = torch.sigmoid(_f32(b))
    out, at = torch.empty(v.shape, dtype=torch.float32, device=v.device), 0
    for slot, n, has in zip(state_indices.tolist(), seq_lens, has_state):
        S = state[slot].clone() if has else torch.zeros_like(state[slot])
        for t in range(at, at + int(n)):
            S = decay[t].unsqueeze(-1) * S
            u = beta[t].unsqueeze(-1) * (vf[t] - (S * kf[t].unsqueeze(-1)).sum(-2))
            S = S + kf[t].unsqueeze(-1) * u.unsqueeze(-2)
            out[t] = (S * qf[t].unsqueeze(-1)).sum(-2)
        state[slot] = S
        at += int(n)
    return out.to(v.dtype)


def residual_dyt(x, y, mult, alpha, weight, bias, dtype):
    if y is not None:
        x.add_(_f32(y), alpha=float(mult))
    return (torch.tanh(_f32(alpha) * x) * _f32(weight) + _f32(bias)).to(dtype)


def turns_of(positions, inv_freq):
    """[T, pairs, 2] fp32: cosine and sine of ``positions * inv_freq``."""
    a = positions.double().unsqueeze(-1) * inv_freq.double()
    return torch.stack([torch.cos(a), torch.sin(a)], -1).float()


def turn_heads(x, turns, halves=False):
    """x [T, H, rot]: neighbouring features (``halves``: feature i and i + rot / 2) turn by ``turns`` [T, rot / 2, 2]."""
    c, s = turns[:, None, :, 0], turns[:, None, :, 1]
    if halves:
        u, v = _f32(x).chunk(2, dim=-1)
        return torch.cat([u * c - v * s, v * c + u * s], -1).to(x.dtype)
    u, v = _f32(x[..., 0::2]), _f32(x[..., 1::2])
    return torch.stack([u * c - v * s, v * c + u * s], -1).flatten(-2).to(x.dtype)


def latent_prologue(y, q_weight, kv_weight, eps, loc=None, cache=None, positions=None, inv_freq=None, halves=False):
    def norm(t, w):
        t = _f32(t)
        return (t * torch.rsqrt(t.pow(2).mean(-1, keepdim=True) + eps) * _f32(w)).to(y.dtype)

    nq = 0 if q_weight is None else q_weight.numel()
    turns = None if inv_freq is None else turns_of(positions, inv_freq)
    if kv_weight is not None:
        rank = kv_weight.numel()
        cache[loc.long(), :rank] = norm(y[:, nq:nq + rank], kv_weight)
        if turns is not None:
            cache[loc.long(), rank:] = turn_heads(y[:, None, nq + rank: nq + rank + 2 * turns.shape[1]], turns, halves)[:, 0]
    return None if q_weight is None else norm(y[:, :nq], q_weight), turns


def latent_gather(cache, req_to_token, req, lens, first=None):
    at = [0] * len(req) if first is None else first.tolist()
    return torch.cat([cache[req_to_token[int(r), f: f + int(n)].long()] for r, n, f in zip(req, lens, at)]) if len(req) else cache[:0]


def latent_attention(q, cache, req_to_token, row_req, row_pos, scale, sink=None, rank=None, window=0):
    rank = q.shape[2] if rank is None else rank
    out = q.new_empty((*q.shape[:2], rank))
    for t in range(q.shape[0]):
        n = int(row_pos[t]) + 1
        c = _f32(cache[req_to_token[int(row_req[t]), max(0, n - window) if window else 0: n].long()])      # [n, rank]
        s = (_f32(q[t]) @ c.t()) * scale                                                  # [H, n]
        p = sink_softmax(s, sink)
        out[t] = (p @ c[:, :rank]).to(q.dtype)
    return out


def sink_softmax(scores: torch.Tensor, sink: Optional[torch.Tensor]) -> torch.Tensor:
    """Softmax over the last dimension of ``scores`` [H, ...]; a head's sink is one more term of the denominator."""
    if sink is None:
        return torch.softmax(scores, dim=-1)
    extra = _f32(sink).view(-1, *([1] * (scores.dim() - 1))).expand(*scores.shape[:-1], 1)
    return torch.softmax(torch.cat([scores, extra], dim=-1), dim=-1)[..., :-1]


# --------------------------------------------------------------------------
# gated delta net (linear attention of the Qwen3.5 hybrid models)
# --------------------------------------------------------------------------
def rmsnorm_gated(x: torch.Tensor, gate: torch.Tensor, weight: torch.Tensor, eps: float, round_norm: bool = True,
                  sigmoid: bool = False) -> torch.Tensor:
    """``weight * rmsnorm(x) * silu(gate)`` (``sigmoid``: that of the gate) over runs of ``weight.numel()`` features (norm before gate; the normed
    value is rounded to x's type first when ``round_norm``)."""
    xf = _f32(x).reshape(*x.shape[:-1], -1, weight.numel())
    n = xf * torch.rsqrt(xf.pow(2).mean(-1, keepdim=True) + eps)
    if round_norm:
        n = _f32(n.to(x.dtype))
    g = _f32(gate)
    return ((_f32(weight) * n).reshape(x.shape) * (torch.sigmoid(g) if sigmoid else F.silu(g))).to(x.dtype)


def gdn_gates(b, a, a_log, dt_bias):
    g = -torch.exp(_f32(a_log)) * F.softplus(_f32(a) + _f32(dt_bias))
    return g, torch.sigmoid(_f32(b))


def causal_conv1d_silu(x: torch.Tensor, weight: torch.Tensor, conv_state: torch.Tensor, state_indices: torch.Tensor,
                       seq_lens, has_state, bias: Optional[torch.Tensor] = None, add_input: bool = False) -> torch.Tensor:
    """Depth-wise causal convolution (kernel K) + SiLU over ragged sequences (``add_input``: plus its input instead of the SiLU).

    ``x`` [T, C] holds the new tokens of every request back to back (``seq_lens`` each); ``weight`` [C, K];
    ``conv_state`` [slots, C, K-1] keeps the last K-1 inputs of each request (row ``state_indices[b]``),
    read when ``has_state[b]`` (a continuation) and always written back."""
    K = weight.shape[1]
    out = torch.empty_like(x)
    off = 0
    for b, n in enumerate(list(seq_lens)):
        n = int(n)
        slot = int(state_indices[b])
        hist = _f32(conv_state[slot]) if bool(has_state[b]) else torch.zeros_like(conv_state[slot], dtype=torch.float32)
        seq = torch.cat([hist, _f32(x[off:off + n]).t()], dim=1)          # [C, K-1+n]
        y = F.conv1d(seq.unsqueeze(0), _f32(weight).unsqueeze(1), None if bias is None else _f32(bias), groups=weight.shape[0]).squeeze(0)  # [C, n]
        out[off:off + n] = (_f32(x[off:off + n]) + y.t() if add_input else F.silu(y).t()).to(x.dtype)
        conv_state[slot] = seq[:, seq.shape[1] - (K - 1):].to(conv_state.dtype)
        off += n
    return out


def gated_delta_rule(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, g: torch.Tensor, beta: torch.Tensor,
                     state: torch.Tensor, state_indices: torch.Tensor, seq_lens, has_state) -> torch.Tensor:
    """Recurrent gated delta rule, one token at a time (the definition the chunked forms must match).

    q, k [T, H, Dk] (l2-normalised here, q scaled by Dk^-0.5), v [T, H, Dv], g (log decay) and beta [T, H];
    ``state`` [slots, H, Dk, Dv] fp32 is read when ``has_state[b]`` and always written back:
    ``S *= exp(g); S += k (x) ((v - S^T k) * beta); o = S^T q``."""
    T, H, Dk = q.shape
    qf = _f32(q)
    kf = _f32(k)
    qf = qf * torch.rsqrt((qf * qf).sum(-1, keepdim=True) + 1e-6) * Dk ** -0.5
    kf = kf * torch.rsqrt((kf * kf).sum(-1, keepdim=True) + 1e-6)
    vf, gf, bf = _f32(v), _f32(g), _f32(beta)
    out = torch.empty(T, H, v.shape[-1], dtype=torch.float32, device=q.device)
    off = 0
    for b, n in enumerate(list(seq_lens)):
        n = int(n)
        slot = int(state_indices[b])
        S = state[slot].float().clone() if bool(has_state[b]) else torch.zeros_like(state[slot], dtype=torch.float32)
        for t in range(off, off + n):
            S = S * gf[t].exp().view(H, 1, 1)
            mem = (S * kf[t].unsqueeze(-1)).sum(-2)                        # [H, Dv]
            delta = (vf[t] - mem) * bf[t].unsqueeze(-1)
            S = S + kf[t].unsqueeze(-1) * delta.unsqueeze(-2)
            out[t] = (S * qf[t].unsqueeze(-1)).sum(-2)
        state[slot] = S.to(state.dtype)
        off += n
    return out.to(v.dtype)



def gated_delta_rule_chunked(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, g: torch.Tensor, beta: torch.Tensor,
                             state: torch.Tensor, state_indices: torch.Tensor, seq_lens, has_state,
                             chunk: int = 64) -> torch.Tensor:
    """The same rule as :func:`gated_delta_rule`, evaluated ``chunk`` tokens at a time with matrix
    products (the chunk-parallel form used for prefill; role of pymllm's ``gdn_chunkwise`` reference).

    Inside a chunk with cumulative log decay ``G_i = sum_{j<=i} g_j`` and incoming state ``S0``:

        A[i, j] = exp(G_i - G_j) (k_i . k_j)  for j < i          (strictly lower triangular)
        U       = (I + diag(beta) A)^-1 diag(beta) (V - exp(G) * (K S0))      # the per-token updates
        O       = exp(G) * (Q S0) + (M * (Q K^T)) U,   M[i, j] = exp(G_i - G_j) for j <= i
        S_end   = exp(G_C) S0 + (exp(G_C - G) * K)^T U

    All exponents are of non-positive numbers (``g <= 0``), so nothing overflows."""
    T, H, Dk = q.shape
    qf = _f32(q)
    kf = _f32(k)
    qf = qf * torch.rsqrt((qf * qf).sum(-1, keepdim=True) + 1e-6) * Dk ** -0.5
    kf = kf * torch.rsqrt((kf * kf).sum(-1, keepdim=True) + 1e-6)
    vf, gf, bf = _f32(v), _f32(g), _f32(beta)
    out = torch.empty(T, H, v.shape[-1], dtype=torch.float32, device=q.device)
    off = 0
    for b, n in enumerate(list(seq_lens)):
        n = int(n)
        slot = int(state_indices[b])
        S = state[slot].float().clone() if bool(has_state[b]) else torch.zeros_like(state[slot], dtype=torch.float32)
        for c0 in range(off, off + n, chunk):
            c1 = min(off + n, c0 + chunk)
            C = c1 - c0
            Q, K, V = (t[c0:c1].transpose(0, 1) for t in (qf, kf, vf))          # [H, C, D]
            G = gf[c0:c1].transpose(0, 1).cumsum(-1)                            # [H, C]
            B = bf[c0:c1].transpose(0, 1)                                       # [H, C]
            diff = G.unsqueeze(-1) - G.unsqueeze(-2)                            # G_i - G_j
            lower = torch.ones(C, C, dtype=torch.bool, device=q.device).tril()
            M = torch.where(lower, diff, torch.full_like(diff, float("-inf"))).exp()   # j <= i
            A = (M * (K @ K.transpose(-1, -2))).tril(-1)
            eG = G.exp().unsqueeze(-1)
            rhs = B.unsqueeze(-1) * (V - eG * (K @ S))
            lhs = torch.eye(C, device=q.device, dtype=torch.float32) + B.unsqueeze(-1) * A
            U = torch.linalg.solve_triangular(lhs, rhs, upper=False, unitriangular=True)
            out[c0:c1] = (eG * (Q @ S) + (M * (Q @ K.transpose(-1, -2))) @ U).transpose(0, 1)
            tail = (G[:, -1:] - G).exp().unsqueeze(-1)                          # exp(G_C - G_j)
            S = G[:, -1].exp().view(H, 1, 1) * S + (tail * K).transpose(-1, -2) @ U
        state[slot] = S.to(state.dtype)
        off += n
    return out.to(v.dtype)
