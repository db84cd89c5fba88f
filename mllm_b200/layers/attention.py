"""Model-side attention layer over the slot-indexed KV pool.

Holds head counts, scale and the layer index (as pymllm/layers/attention/radix_attention.py:24-171)
and runs the fused prologue (per-head QK-norm, rotary embedding, cache write) followed by
the prefill or decode attention kernel chosen by the batch's forward mode.  The kernels read
the request->slot table directly, so there is no per-step planning or index flattening.
"""

from __future__ import annotations

import math
from typing import Optional

import torch
from torch import nn

from .. import ops


class RadixAttention(nn.Module):
    def __init__(self, num_heads: int, head_dim: int, scaling: float, num_kv_heads: int, layer_id: int,
                 rope_theta: float = 1e6, rms_eps: float = 1e-6, mrope_sections=None,
                 mrope_interleaved: bool = False, rope_scaling: Optional[dict] = None,
                 sliding_window: Optional[int] = None, logit_cap: float = 0.0) -> None:
        super().__init__()
        self.rope_scaling = rope_scaling
        # each query attends to its last `sliding_window` keys (itself included); scores soft-capped at logit_cap
        self.sliding_window = int(sliding_window) if sliding_window else None
        self.logit_cap = float(logit_cap or 0.0)
        self.num_heads, self.num_kv_heads, self.head_dim = num_heads, num_kv_heads, head_dim
        # yarn / longrope checkpoints scale cos and sin by a constant: q.k grows by its square
        self.scaling, self.layer_id = scaling * ops.rope_attention_factor(rope_scaling) ** 2, layer_id
        self.rope_theta, self.rms_eps = rope_theta, rms_eps
        self.mrope_sections, self.mrope_interleaved = mrope_sections, mrope_interleaved
        self._inv_freq: Optional[torch.Tensor] = None
        self._axis_map: Optional[torch.Tensor] = None

    def _tables(self, device):
        if self._inv_freq is None or self._inv_freq.device != device:
            self._inv_freq = ops.rope_inv_freq(self.head_dim, self.rope_theta, device, self.rope_scaling)
            if self.mrope_sections is not None:
                self._axis_map = ops.mrope_axis_map(self.head_dim, self.mrope_sections, self.mrope_interleaved, device)
        return self._inv_freq, self._axis_map

    def forward(self, qkv: torch.Tensor, q_norm_w, k_norm_w, forward_batch) -> torch.Tensor:
        """``qkv`` [T, (Hq+2Hkv)*D] fused projection output -> attention output [T, Hq*D]."""
        fb = forward_batch
        T = qkv.shape[0]
        if fb.forward_mode.is_idle() or T == 0:
            return qkv.new_zeros((T, self.num_heads * self.head_dim))
        k_cache, v_cache = fb.token_to_kv_pool.get_kv_buffer(self.layer_id)
        inv_freq, axis_map = self._tables(qkv.device)
        use_mrope = self.mrope_sections is not None and fb.mrope_positions is not None
        ops.qk_norm_rope_kv_write(
            qkv, q_norm_w, k_norm_w, fb.mrope_positions if use_mrope else fb.positions, fb.out_cache_loc,
            k_cache, v_cache, self.num_heads, self.num_kv_heads, self.head_dim, self.rope_theta, self.rms_eps,
            self.mrope_sections if use_mrope else None, self.mrope_interleaved,
            inv_freq=inv_freq, axis_map=axis_map if use_mrope else None,
        )
        q = qkv[:, : self.num_heads * self.head_dim].view(T, self.num_heads, self.head_dim)
        out = torch.empty((T, self.num_heads, self.head_dim), dtype=qkv.dtype, device=qkv.device)
        if fb.forward_mode.is_decode():
            ops.attention_decode(q, k_cache, v_cache, fb.req_to_token_pool.req_to_token, fb.req_pool_indices,
                                 fb.seq_lens, self.scaling, out=out, max_seq_len=fb.max_seq_len,
                                 window=self.sliding_window, logit_cap=self.logit_cap)
        else:
            ops.attention_prefill(q, k_cache, v_cache, fb.req_to_token_pool.req_to_token, fb.req_pool_indices,
                                  fb.seq_lens, fb.extend_prefix_lens, fb.extend_start_loc, self.scaling, out=out,
                                  max_q_len=fb.max_extend_len, window=self.sliding_window, logit_cap=self.logit_cap)
        return out.view(T, self.num_heads * self.head_dim)


def query_rows(fb):
    """(request-table row int32 [T], position int64 [T]) of every query row of a batch; cached in ``fb.extra``."""
    got = fb.extra.get("query_rows")
    if got is None:
        req = fb.req_pool_indices.to(torch.int32)
        if not fb.forward_mode.is_decode():
            req = torch.repeat_interleave(req, fb.extend_seq_lens.long(), output_size=fb.input_ids.shape[0])
        got = fb.extra["query_rows"] = (req, fb.positions.to(torch.int64))
    return got


def rotation_frequencies(dims: int, base: float, scaling: Optional[dict] = None) -> torch.Tensor:
    """One fp64 frequency per rotated pair, ``base^(-2i / dims)``.  ``scaling`` (factor, low, high, original): frequencies
    whose wave is longer than ``original / low`` are divided by ``factor``, waves shorter than ``original / high`` stay, with
    a linear blend (in original / wave) between.  ``scaling`` with (factor, original, fast, slow) is YaRN's: pair i is divided by
    ``factor`` to a degree that rises linearly from 0 at the pair that makes ``fast`` turns over ``original`` positions to 1 at
    the pair that makes ``slow``."""
    i = torch.arange(dims // 2, dtype=torch.float64)
    f = torch.pow(torch.tensor(base, dtype=torch.float64), -2.0 * i / max(1, dims))
    if scaling and "fast" in scaling:
        def pair_of(turns: float) -> float:
            return dims * math.log(float(scaling["original"]) / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

        lo, hi = max(math.floor(pair_of(float(scaling["fast"]))), 0), min(math.ceil(pair_of(float(scaling["slow"]))), dims - 1)
        ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
        return f / float(scaling["factor"]) * ramp + f * (1.0 - ramp)
    if scaling:
        factor, lo, hi, old = (float(scaling[k]) for k in ("factor", "low", "high", "original"))
        turns = old * f / (2.0 * math.pi)                   # over the original length: original / wavelength
        keep = torch.where(turns > hi, 1.0, torch.where(turns < lo, 0.0, (turns - lo) / (hi - lo)))
        f = (1.0 - keep) * f / factor + keep * f
    return f


def rotation_magnitude(scaling: Optional[dict]) -> float:
    """Factor of the sines and cosines that comes with YaRN's frequencies."""
    return 0.1 * math.log(float(scaling["factor"])) + 1.0 if scaling and "fast" in scaling else 1.0


class SizedAttention(nn.Module):
    """Causal attention core for layers that give their own sizes: grouped query heads, keys of ``dim`` and values of
    ``vdim`` features, rotation of part of each head, any score scale, an optional sliding window or chunks of positions, an
    optional sink per head, an optional gate per head (``gate_at``: the column of its logits).  It reads the projected rows that ``shards`` names and writes the concatenated heads; projections belong to the
    mixer around it.  Subclasses have the prologue (:meth:`prepare`): norms, rotation, cache write.

    16-bit runs use the attention kernels of the other models, with heads zero-padded to 64 / 128 / 256 features in the
    cache and in the rows that leave (``width``); fp32 runs and wider heads take the row kernel, unpadded."""

    folds_scale = False       # the output is linear in V only: a scale on it belongs to what follows
    biased: tuple = ()

    def __init__(self, heads: int, kv_heads: int, dim: int, vdim: int, scale: float, eps: float, kv_index: int, rot_dims: int = 0,
                 rot_base: float = 1e4, rot_scaling: Optional[dict] = None, window: Optional[int] = None,
                 dtype: torch.dtype = torch.bfloat16, chunk: Optional[int] = None) -> None:
        super().__init__()
        if heads % kv_heads or rot_dims % 2 or rot_dims > dim:
            raise ValueError(f"attention: {heads} heads over {kv_heads}, {rot_dims} of {dim} features rotated")
        self.heads, self.kv_heads, self.dim, self.vdim = heads, kv_heads, dim, vdim
        self.scale, self.eps, self.kv_index, self.window, self.chunk = float(scale), float(eps), kv_index, window, chunk
        self.gate_at: Optional[int] = None
        self.rot_dims, self.rot_base, self.rot_scaling = rot_dims, float(rot_base), rot_scaling
        self.width = None if dtype == torch.float32 or heads // kv_heads > 128 else next(
            (w for w in (64, 128, 256) if w >= max(dim, vdim) and ops.attention_kernels_cover(w, dtype, dtype)), None)
        self.register_parameter("sink", None)
        self._inv_freq: Optional[torch.Tensor] = None

    @property
    def kv_shape(self):
        """(kv heads, key width, value width) of the layer's cache rows."""
        return self.kv_heads, self.width or self.dim, self.width or self.vdim

    @property
    def out_width(self) -> int:
        return self.heads * (self.width or self.vdim)

    def expand_columns(self, w: torch.Tensor) -> torch.Tensor:
        """An output projection's columns [.., heads * vdim] spread to the padded heads."""
        if self.width in (None, self.vdim):
            return w
        out = torch.zeros(w.shape[0], self.heads, self.width, dtype=w.dtype, device=w.device)
        out[:, :, : self.vdim] = w.view(w.shape[0], self.heads, self.vdim)
        return out.view(w.shape[0], -1)

    def inv_freq(self, device) -> torch.Tensor:
        if self._inv_freq is None or self._inv_freq.device != device:
            self._inv_freq = rotation_frequencies(self.rot_dims, self.rot_base, self.rot_scaling).to(device)
        return self._inv_freq

    def prepare(self, row: torch.Tensor, fb, q: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor) -> None:
        """Queries of ``row`` into ``q`` [T, heads, key width], keys and values into the cache slots of the batch."""
        raise NotImplementedError

    def forward(self, row: torch.Tensor, fb, out: torch.Tensor) -> None:
        """``row`` [T, >= the shards], ``out`` [T, out_width] (a column slice of a wider matrix will do)."""
        T = row.shape[0]
        kw, vw = self.kv_shape[1:]
        k_cache, v_cache = fb.token_to_kv_pool.get_kv_buffer(self.kv_index)
        rtt = fb.req_to_token_pool.req_to_token
        q = torch.empty((T, self.heads, kw), dtype=row.dtype, device=row.device)
        self.prepare(row, fb, q, k_cache, v_cache)
        o = out.unflatten(1, (self.heads, vw))
        if self.width is None or not row.is_cuda:
            ops.attention_rows(q, k_cache, v_cache, rtt, *query_rows(fb), self.scale, o, window=self.window, sink=self.sink, chunk=self.chunk)
        elif fb.forward_mode.is_decode():
            ops.attention_decode(q, k_cache, v_cache, rtt, fb.req_pool_indices, fb.seq_lens, self.scale, out=o, max_seq_len=fb.max_seq_len,
                                 window=self.window, sink=self.sink, chunk=self.chunk)
        else:
            ops.attention_prefill(q, k_cache, v_cache, rtt, fb.req_pool_indices, fb.seq_lens, fb.extend_prefix_lens, fb.extend_start_loc,
                                  self.scale, out=o, max_q_len=fb.max_extend_len, window=self.window, sink=self.sink,
                                  chunk=self.chunk)
        if self.gate_at is not None:
            ops.gate_heads(o, row[:, self.gate_at: self.gate_at + self.heads], out=o)


class RowNormAttention(SizedAttention):
    """With a query / key norm that spans all heads of the row, then rotation of neighbouring features; rows are
    ``[q | k | v]``."""

    def __init__(self, heads: int, kv_heads: int, dim: int, vdim: int, scale: float, eps: float, kv_index: int, rot_dims: int = 0,
                 rot_base: float = 1e4, window: Optional[int] = None, dtype: torch.dtype = torch.bfloat16, biased: bool = True) -> None:
        super().__init__(heads, kv_heads, dim, vdim, scale, eps, kv_index, rot_dims, rot_base, None, window, dtype)
        self.shards = {"q": heads * dim, "k": kv_heads * dim, "v": kv_heads * vdim}
        self.biased = tuple(self.shards) if biased else ()
        self.q_norm, self.k_norm = nn.Module(), nn.Module()
        self.q_norm.weight = nn.Parameter(torch.ones(heads * dim, dtype=torch.float32), requires_grad=False)
        self.k_norm.weight = nn.Parameter(torch.ones(kv_heads * dim, dtype=torch.float32), requires_grad=False)

    def prepare(self, row, fb, q, k_cache, v_cache) -> None:
        ops.rownorm_rope_kv(row, self.q_norm.weight, self.k_norm.weight, self.inv_freq(row.device), fb.positions, fb.out_cache_loc, q,
                            k_cache, v_cache, self.heads, self.kv_heads, self.dim, self.vdim, self.eps)


class HeadNormAttention(SizedAttention):
    """Query and key heads turn (``halves``: feature i with the one half the rotated features on, else neighbours) and are
    then divided by their root mean square.  Rows are ``[q | k | v]``, or ``[q | k]`` with ``tied``: the values are the keys
    as projected.  ``sinks``: a logit per head that joins the softmax denominator only."""

    def __init__(self, heads: int, kv_heads: int, dim: int, vdim: int, scale: float, eps: float, kv_index: int, rot_dims: int = 0,
                 rot_base: float = 1e4, rot_scaling: Optional[dict] = None, halves: bool = True, tied: bool = False, sinks: bool = False,
                 window: Optional[int] = None, dtype: torch.dtype = torch.bfloat16) -> None:
        super().__init__(heads, kv_heads, dim, vdim, scale, eps, kv_index, rot_dims, rot_base, rot_scaling, window, dtype)
        if tied and vdim != dim:
            raise ValueError(f"attention: values that are the keys have {dim} features, not {vdim}")
        self.halves, self.tied = halves, tied
        self.shards = {"q": heads * dim, "k": kv_heads * dim}
        self.v_at = heads * dim
        if not tied:
            self.v_at += kv_heads * dim
            self.shards["v"] = kv_heads * vdim
        if sinks:
            self.sink = nn.Parameter(torch.zeros(heads, dtype=torch.float32), requires_grad=False)

    def prepare(self, row, fb, q, k_cache, v_cache) -> None:
        ops.headnorm_rope_kv(row, self.inv_freq(row.device), fb.positions, fb.out_cache_loc, q, k_cache, v_cache, self.heads, self.kv_heads,
                             self.dim, self.vdim, self.v_at, self.halves, self.eps)


class RotaryAttention(SizedAttention):
    """Query and key heads turn (feature i with the one half the rotated features on) and keep their length, up to the
    magnitude that comes with scaled frequencies.  Rows are ``[q | k | v]``, with ``gated`` ``[q | k | v | g]``: each head's output
    is multiplied by the logistic function of its own logit."""

    def __init__(self, heads: int, kv_heads: int, dim: int, vdim: int, scale: float, kv_index: int, rot_dims: int = 0, rot_base: float = 1e4,
                 rot_scaling: Optional[dict] = None, window: Optional[int] = None, chunk: Optional[int] = None, gated: bool = False,
                 dtype: torch.dtype = torch.bfloat16) -> None:
        super().__init__(heads, kv_heads, dim, vdim, scale, 0.0, kv_index, rot_dims, rot_base, rot_scaling, window, dtype, chunk)
        self.shards = {"q": heads * dim, "k": kv_heads * dim, "v": kv_heads * vdim}
        self.v_at = (heads + kv_heads) * dim
        self.magnitude = rotation_magnitude(rot_scaling)
        if gated:
            self.shards["g"] = heads
            self.gate_at = self.v_at + kv_heads * vdim

    def prepare(self, row, fb, q, k_cache, v_cache) -> None:
        ops.headnorm_rope_kv(row, self.inv_freq(row.device), fb.positions, fb.out_cache_loc, q, k_cache, v_cache, self.heads, self.kv_heads,
                             self.dim, self.vdim, self.v_at, True, 0.0, norm=False, magnitude=self.magnitude)
