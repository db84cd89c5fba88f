"""Model-side attention layer over the slot-indexed KV pool.

Holds head counts, scale and the layer index (as pymllm/layers/attention/radix_attention.py:24-171)
and runs the fused prologue (per-head QK-norm, rotary embedding, cache write) followed by
the prefill or decode attention kernel chosen by the batch's forward mode.  The kernels read
the request->slot table directly, so there is no per-step planning or index flattening.
"""

from __future__ import annotations

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


class RowNormAttention(nn.Module):
    """Causal attention core for layers that give their own sizes: grouped query heads, keys of ``dim`` and values of
    ``vdim`` features, a query / key norm that spans all heads of the row, rotation of neighbouring features on the
    first ``rot_dims`` of each head, any score scale, an optional sliding window.  It reads the projected rows
    ``[q | k | v]`` and writes the concatenated heads; projections belong to the mixer around it.

    16-bit runs use the attention kernels of the other models, with heads zero-padded to 64 / 128 / 256 features in the
    cache and in the rows that leave (``width``); fp32 runs and wider heads take the row kernel, unpadded."""

    folds_scale = False       # the output is linear in V only: a scale on it belongs to what follows

    def __init__(self, heads: int, kv_heads: int, dim: int, vdim: int, scale: float, eps: float, kv_index: int, rot_dims: int = 0,
                 rot_base: float = 1e4, window: Optional[int] = None, dtype: torch.dtype = torch.bfloat16, biased: bool = True) -> None:
        super().__init__()
        if heads % kv_heads or rot_dims % 2 or rot_dims > dim:
            raise ValueError(f"attention: {heads} heads over {kv_heads}, {rot_dims} of {dim} features rotated")
        self.heads, self.kv_heads, self.dim, self.vdim = heads, kv_heads, dim, vdim
        self.scale, self.eps, self.kv_index, self.window = float(scale), float(eps), kv_index, window
        self.rot_dims, self.rot_base = rot_dims, float(rot_base)
        self.shards = {"q": heads * dim, "k": kv_heads * dim, "v": kv_heads * vdim}
        self.biased = tuple(self.shards) if biased else ()
        self.width = None if dtype == torch.float32 or heads // kv_heads > 128 else next(
            (w for w in (64, 128, 256) if w >= max(dim, vdim) and ops.attention_kernels_cover(w, dtype, dtype)), None)
        self.q_norm, self.k_norm = nn.Module(), nn.Module()
        self.q_norm.weight = nn.Parameter(torch.ones(heads * dim, dtype=torch.float32), requires_grad=False)
        self.k_norm.weight = nn.Parameter(torch.ones(kv_heads * dim, dtype=torch.float32), requires_grad=False)
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
        """One fp64 frequency per rotated pair: ``rot_base^(-2i / rot_dims)``."""
        if self._inv_freq is None or self._inv_freq.device != device:
            i = torch.arange(self.rot_dims // 2, dtype=torch.float64)
            self._inv_freq = torch.pow(torch.tensor(self.rot_base, dtype=torch.float64), -2.0 * i / max(1, self.rot_dims)).to(device)
        return self._inv_freq

    def forward(self, row: torch.Tensor, fb, out: torch.Tensor) -> None:
        """``row`` [T, >= q | k | v], ``out`` [T, out_width] (a column slice of a wider matrix will do)."""
        T = row.shape[0]
        kw, vw = self.kv_shape[1:]
        k_cache, v_cache = fb.token_to_kv_pool.get_kv_buffer(self.kv_index)
        rtt = fb.req_to_token_pool.req_to_token
        q = torch.empty((T, self.heads, kw), dtype=row.dtype, device=row.device)
        ops.rownorm_rope_kv(row, self.q_norm.weight, self.k_norm.weight, self.inv_freq(row.device), fb.positions, fb.out_cache_loc, q,
                            k_cache, v_cache, self.heads, self.kv_heads, self.dim, self.vdim, self.eps)
        o = out.unflatten(1, (self.heads, vw))
        if self.width is None or not row.is_cuda:
            ops.attention_rows(q, k_cache, v_cache, rtt, *query_rows(fb), self.scale, o, window=self.window)
        elif fb.forward_mode.is_decode():
            ops.attention_decode(q, k_cache, v_cache, rtt, fb.req_pool_indices, fb.seq_lens, self.scale, out=o, max_seq_len=fb.max_seq_len,
                                 window=self.window)
        else:
            ops.attention_prefill(q, k_cache, v_cache, rtt, fb.req_pool_indices, fb.seq_lens, fb.extend_prefix_lens, fb.extend_start_loc,
                                  self.scale, out=o, max_q_len=fb.max_extend_len, window=self.window)
