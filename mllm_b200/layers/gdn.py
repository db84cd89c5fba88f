"""Gated DeltaNet token mixers.  :class:`GatedDeltaNet` is that of the Qwen3.5 hybrid models (roles of pymllm/layers/gated_delta_net.py,
layers/attention/gdn_backend.py and rms_norm_gated.py; math of HF ``Qwen3_5GatedDeltaNet``):

    qkv = conv1d_silu(in_proj_qkv(x))      depth-wise causal conv over the last 4 inputs, SiLU
    beta = sigmoid(in_proj_b(x)),  g = -exp(A_log) * softplus(in_proj_a(x) + dt_bias)
    S <- S * exp(g);  S <- S + k (x) ((v - S^T k) * beta);  o = S^T q      (q, k l2-normalised, q / sqrt(Dk))
    y = out_proj( rmsnorm(o) * w * silu(in_proj_z(x)) )

State (recurrent matrix and conv history) lives in a :class:`GDNPool` row per request, so prefill of a
continuation (chunked prefill) and decode both resume from it.

:class:`ChannelDeltaNet` is the rule with a decay per key channel.  :class:`FusedGatedDeltaNet` is the same rule for models that give its sizes per layer: one projection for everything
that is taken of the layer input, gates formed inside the rule's kernel, 32-bit products in the recurrence.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, Optional

import torch
from torch import nn

from .. import ops
from ..parallel import state as pstate


@dataclass
class GdnBatch:
    """What the delta-net kernels need to know about a batch, shared by all layers of a forward pass."""

    slots: torch.Tensor       # [B] state row of each request
    lens: torch.Tensor        # [B] new tokens
    has_state: torch.Tensor   # [B] 1 where earlier tokens left a state
    q_start: Optional[torch.Tensor]   # [B] first row of each request
    max_len: int              # longest run of new tokens (0: not known on the host)


def gdn_batch(fb) -> GdnBatch:
    got = fb.extra.get("gdn_batch")
    if got is None:
        slots = fb.req_pool_indices.to(torch.int32)
        if fb.forward_mode.is_decode():
            ones = torch.ones(fb.batch_size, dtype=torch.int32, device=slots.device)
            got = GdnBatch(slots, ones, ones, torch.arange(fb.batch_size, dtype=torch.int32, device=slots.device), 1)
        else:
            start = fb.extend_start_loc
            got = GdnBatch(slots, fb.extend_seq_lens.to(torch.int32), (fb.extend_prefix_lens > 0).to(torch.int32),
                           None if start is None else start.to(torch.int32), int(fb.max_extend_len or 0))
        fb.extra["gdn_batch"] = got
    return got


class GatedDeltaNet(nn.Module):
    def __init__(self, config, layer_id: int, gdn_index: int, params_dtype=None, prefix: str = "") -> None:
        super().__init__()
        dt = params_dtype or torch.get_default_dtype()
        H = config.hidden_size
        self.layer_id, self.gdn_index = layer_id, gdn_index
        # tensor parallelism: every rank owns num_heads / tp value heads with their key heads (the
        # recurrent state, the convolution channels and the gates are per head, so nothing is exchanged
        # until the row-parallel output projection, whose partial sums are all-reduced)
        self.tp, self.tp_rank = pstate.get_tensor_model_parallel_world_size(), pstate.get_tensor_model_parallel_rank()
        hv, hk = config.linear_num_value_heads, config.linear_num_key_heads
        if hv % self.tp or hk % self.tp:
            raise ValueError(f"gated delta net: {hk} key / {hv} value heads do not divide over {self.tp} ranks")
        self.total_k_heads, self.total_v_heads = hk, hv
        self.num_v_heads, self.num_k_heads = hv // self.tp, hk // self.tp
        self.head_k_dim, self.head_v_dim = config.linear_key_head_dim, config.linear_value_head_dim
        self.key_dim, self.value_dim = self.head_k_dim * self.num_k_heads, self.head_v_dim * self.num_v_heads
        self.conv_dim = 2 * self.key_dim + self.value_dim
        self.conv_kernel = config.linear_conv_kernel_dim
        self.eps = getattr(config, "rms_norm_eps", 1e-6)

        def w(*shape, loader=None, dtype=dt, init=None):
            t = torch.empty(*shape, dtype=dtype) if init is None else torch.full(shape, init, dtype=dtype)
            p = nn.Parameter(t, requires_grad=False)
            if loader is not None:
                p.weight_loader = loader
            return p

        self.in_proj_qkv = nn.Module()
        self.in_proj_qkv.weight = w(self.conv_dim, H, loader=self._load_qkv_rows)
        self.in_proj_z = nn.Module()
        self.in_proj_z.weight = w(self.value_dim, H, loader=self._load_v_rows)
        self.in_proj_b = nn.Module()
        self.in_proj_b.weight = w(self.num_v_heads, H, loader=self._load_v_rows)
        self.in_proj_a = nn.Module()
        self.in_proj_a.weight = w(self.num_v_heads, H, loader=self._load_v_rows)
        self.conv1d = nn.Module()
        self.conv1d.weight = w(self.conv_dim, self.conv_kernel, loader=self._load_qkv_rows)
        self.dt_bias = w(self.num_v_heads, loader=self._load_v_rows, dtype=torch.float32, init=1.0)
        self.A_log = w(self.num_v_heads, loader=self._load_v_rows, dtype=torch.float32, init=0.0)
        self.norm = nn.Module()
        self.norm.weight = nn.Parameter(torch.ones(self.head_v_dim, dtype=dt), requires_grad=False)
        self.out_proj = nn.Module()
        self.out_proj.weight = w(H, self.value_dim, loader=self._load_v_cols)

    # ---- loading: slices of the full (unsharded) checkpoint tensors ----
    def _load_qkv_rows(self, param, full, shard_id=None) -> None:
        """Rows are [q heads | k heads | v heads]; take this rank's heads of each block (also the layout
        of the convolution channels, whose checkpoint shape is [C, 1, K])."""
        full = full.reshape(full.shape[0], -1)
        kd, vd = self.head_k_dim * self.total_k_heads, self.head_v_dim * self.total_v_heads
        q, k, v = full[:kd], full[kd:2 * kd], full[2 * kd:2 * kd + vd]
        r = self.tp_rank
        param.data.copy_(torch.cat([q[r * self.key_dim:(r + 1) * self.key_dim], k[r * self.key_dim:(r + 1) * self.key_dim],
                                    v[r * self.value_dim:(r + 1) * self.value_dim]], 0).reshape(param.shape))

    def _load_v_rows(self, param, full, shard_id=None) -> None:
        n = param.shape[0]
        param.data.copy_(full[self.tp_rank * n:(self.tp_rank + 1) * n].reshape(param.shape))

    def _load_v_cols(self, param, full, shard_id=None) -> None:
        n = param.shape[1]
        param.data.copy_(full[:, self.tp_rank * n:(self.tp_rank + 1) * n])

    def forward(self, x: torch.Tensor, fb) -> torch.Tensor:
        pool = fb.extra["gdn_pool"]
        recurrent, conv = pool.layer(self.gdn_index)
        T = x.shape[0]
        m = gdn_batch(fb)
        qkv = ops.linear(x, self.in_proj_qkv.weight)
        z = ops.linear(x, self.in_proj_z.weight)
        ba = ops.linear(x, torch.cat([self.in_proj_b.weight, self.in_proj_a.weight], 0)) if not hasattr(self, "_ba") else \
            ops.linear(x, self._ba)
        b, a = ba[:, : self.num_v_heads], ba[:, self.num_v_heads:]
        qkv = ops.causal_conv1d_silu(qkv, self.conv1d.weight, conv, m.slots, m.lens, m.has_state, m.q_start, m.max_len)
        q, k, v = torch.split(qkv, [self.key_dim, self.key_dim, self.value_dim], dim=-1)
        # views of the convolution's rows; value head h uses query / key head h // (value heads / key heads)
        q = q.unflatten(1, (self.num_k_heads, self.head_k_dim))
        k = k.unflatten(1, (self.num_k_heads, self.head_k_dim))
        v = v.unflatten(1, (self.num_v_heads, self.head_v_dim))
        beta = torch.sigmoid(b.float())
        g = -torch.exp(self.A_log.float()) * torch.nn.functional.softplus(a.float() + self.dt_bias.float())
        o = ops.gated_delta_rule(q, k, v, g, beta, recurrent, m.slots, m.lens, m.has_state, m.q_start)
        o = ops.rmsnorm_gated(o.reshape(-1, self.head_v_dim), z.reshape(-1, self.head_v_dim), self.norm.weight, self.eps)
        y = ops.linear(o.reshape(T, self.value_dim), self.out_proj.weight)
        return pstate.tensor_model_parallel_all_reduce(y) if self.tp > 1 else y

    def fuse_small_projections(self) -> None:
        """One GEMM for the beta / decay projections (call after loading)."""
        self._ba = torch.cat([self.in_proj_b.weight.data, self.in_proj_a.weight.data], 0).contiguous()


class FusedGatedDeltaNet(nn.Module):
    """One delta-net mixer with its own sizes.  The projections of the layer input are the row blocks
    ``[q | k | v | gate | b | a]`` of one matrix (zero rows up to a multiple of 8); q and k have ``kv_heads`` heads and
    value head ``h`` uses head ``h // (heads / kv_heads)``.  Unit norms, gates and the recurrence are fp32."""

    def __init__(self, hidden_size: int, heads: int, kv_heads: int, dim: int, vdim: int, conv: int, eps: float, gdn_index: int,
                 params_dtype: torch.dtype) -> None:
        super().__init__()
        if heads % kv_heads:
            raise ValueError(f"delta net: {heads} value heads over {kv_heads} key heads")
        self.heads, self.kv_heads, self.dim, self.vdim, self.conv_kernel = heads, kv_heads, dim, vdim, conv
        self.eps, self.gdn_index = eps, gdn_index
        self.key_dim, self.value_dim = kv_heads * dim, heads * vdim
        self.conv_dim = 2 * self.key_dim + self.value_dim
        self.shards = {"q": self.key_dim, "k": self.key_dim, "v": self.value_dim, "g": self.value_dim, "b": heads, "a": heads}
        self.offset, rows = {}, 0
        for name, n in self.shards.items():
            self.offset[name] = rows
            rows += n

        def p(*shape, dtype=params_dtype):
            return nn.Parameter(torch.zeros(*shape, dtype=dtype), requires_grad=False)

        self.in_proj = nn.Module()
        self.in_proj.weight = p(-(-rows // 8) * 8, hidden_size)
        self.conv1d = nn.Module()
        self.conv1d.weight = p(self.conv_dim, conv)
        self.A_log = p(heads, dtype=torch.float32)
        self.dt_bias = p(heads, dtype=torch.float32)
        self.norm = nn.Module()
        self.norm.weight = nn.Parameter(torch.ones(vdim, dtype=params_dtype), requires_grad=False)
        self.out_proj = nn.Module()
        self.out_proj.weight = p(hidden_size, self.value_dim)

    @property
    def state_shape(self):
        """(value heads, key features, value features, convolution channels, taps) of a request's state."""
        return self.heads, self.dim, self.vdim, self.conv_dim, self.conv_kernel

    def load_projection(self, name: str, full: torch.Tensor) -> None:
        o = self.offset[name]
        self.in_proj.weight.data[o:o + self.shards[name]].copy_(full)

    def load_conv(self, name: str, full: torch.Tensor) -> None:
        o = self.offset[name]
        self.conv1d.weight.data[o:o + self.shards[name]].copy_(full.reshape(self.shards[name], self.conv_kernel))

    def forward(self, x: torch.Tensor, fb) -> torch.Tensor:
        recurrent, conv = fb.extra["gdn_pool"].layer(self.gdn_index)
        m = gdn_batch(fb)
        o, C = self.offset, self.conv_dim
        y = ops.linear(x, self.in_proj.weight)
        qkv = ops.causal_conv1d_silu(y[:, :C], self.conv1d.weight, conv, m.slots, m.lens, m.has_state, m.q_start, m.max_len)
        q = qkv[:, : o["k"]].unflatten(1, (self.kv_heads, self.dim))
        k = qkv[:, o["k"]: o["v"]].unflatten(1, (self.kv_heads, self.dim))
        v = qkv[:, o["v"]:].unflatten(1, (self.heads, self.vdim))
        gates = (y[:, o["b"]: o["b"] + self.heads], y[:, o["a"]: o["a"] + self.heads], self.A_log, self.dt_bias)
        r = ops.gated_delta_rule(q, k, v, None, None, recurrent, m.slots, m.lens, m.has_state, m.q_start, raw_gates=gates,
                                 split_tf32=True)
        r = ops.rmsnorm_gated(r.reshape(-1, self.value_dim), y[:, o["g"]: o["g"] + self.value_dim], self.norm.weight, self.eps,
                              round_norm=False)
        return ops.linear(r, self.out_proj.weight)


class ChannelDeltaNet(nn.Module):
    """One delta-net mixer whose state decays by a factor per key channel:

        q, k, v = silu(conv1d(W x));  beta = sigmoid(W_b x);  g = -exp(A_log) * softplus(W_a2 W_a1 x + dt_bias)
        S <- diag(exp(g)) S;  S <- S + k (beta (v - S^T k))^T;  o = S^T q          (q, k unit vectors, q / sqrt(dim))
        y = W_o (rmsnorm(o) * w * sigmoid(W_g2 W_g1 x))

    The projections of the input are the row blocks ``[q | k | v | b | a1 | g1]`` of one matrix; the second factors of the decays
    and of the gates are one product with a matrix of two blocks.  Blocks begin at multiples of 8.  q and k have ``kv_heads``
    heads and value head ``h`` uses head ``h // (heads / kv_heads)``.  Unit norms, gates and the recurrence are fp32."""

    def __init__(self, hidden_size: int, heads: int, kv_heads: int, dim: int, vdim: int, conv: int, a_rank: int, g_rank: int, eps: float,
                 gdn_index: int, params_dtype: torch.dtype) -> None:
        super().__init__()
        if heads % kv_heads:
            raise ValueError(f"delta net: {heads} value heads over {kv_heads} key heads")
        self.heads, self.kv_heads, self.dim, self.vdim, self.conv_kernel = heads, kv_heads, dim, vdim, conv
        self.eps, self.gdn_index, self.dtype = eps, gdn_index, params_dtype
        self.key_dim, self.value_dim, self.decay_dim = kv_heads * dim, heads * vdim, heads * dim
        self.conv_dim = 2 * self.key_dim + self.value_dim
        self.hidden_size = hidden_size

        def p(*shape, dtype=params_dtype):
            old = getattr(getattr(self, "in_proj", None), "weight", None)       # later calls stay on the module's device
            return nn.Parameter(torch.zeros(*shape, dtype=dtype, device=None if old is None else old.device), requires_grad=False)

        self._p = p
        self._low_rank: Dict[str, torch.Tensor] = {}
        self.in_proj, self.low_rank, self.conv1d, self.norm, self.out_proj = (nn.Module() for _ in range(5))
        self.set_ranks(a_rank, g_rank)
        self.conv1d.weight = p(self.conv_dim, conv)
        self.A_log = p(heads, dtype=torch.float32)
        self.dt_bias = p(self.decay_dim, dtype=torch.float32)
        self.norm.weight = nn.Parameter(torch.ones(vdim, dtype=params_dtype), requires_grad=False)
        self.out_proj.weight = p(hidden_size, self.value_dim)

    def set_ranks(self, a_rank: int, g_rank: int) -> None:
        """Inner sizes of the decays' and of the gates' projections.  Rows of the other projections that were loaded stay."""
        old = getattr(self.in_proj, "weight", None)
        self.shards = {"q": self.key_dim, "k": self.key_dim, "v": self.value_dim, "b": self.heads, "a1": a_rank, "g1": g_rank}
        self.offset, rows = {}, 0
        for name, n in self.shards.items():
            if name not in ("k", "v"):        # q, k and v are neighbours: one convolution
                rows = -(-rows // 8) * 8
            self.offset[name] = rows
            rows += n
        self.in_proj.weight = self._p(-(-rows // 8) * 8, self.hidden_size)
        if old is not None:
            self.in_proj.weight.data[: self.offset["a1"]].copy_(old.data[: self.offset["a1"]])
        self.inner = slice(self.offset["a1"], -(-rows // 8) * 8)
        self.gate_at = -(-self.decay_dim // 8) * 8
        self.low_rank.weight = self._p(self.gate_at + -(-self.value_dim // 8) * 8, self.inner.stop - self.inner.start)

    @property
    def state_shape(self):
        """(value heads, key features, value features, convolution channels, taps) of a request's state."""
        return self.heads, self.dim, self.vdim, self.conv_dim, self.conv_kernel

    def load_projection(self, name: str, full: torch.Tensor) -> None:
        self._fit(self.in_proj.weight.data[self.offset[name]: self.offset[name] + self.shards[name]], full)

    def load_low_rank(self, name: str, full: torch.Tensor) -> None:
        """``name``: a1, a2 (decays), g1 or g2 (gates).  Their shapes alone give the inner sizes, so the four are placed together."""
        parts = self._low_rank
        parts[name] = full
        if len(parts) < 4:
            return
        self.set_ranks(parts["a1"].shape[0], parts["g1"].shape[0])
        for first, second, row, rows in (("a1", "a2", 0, self.decay_dim), ("g1", "g2", self.gate_at, self.value_dim)):
            self.load_projection(first, parts[first])
            col = self.offset[first] - self.inner.start
            self._fit(self.low_rank.weight.data[row: row + rows, col: col + self.shards[first]], parts[second])
        parts.clear()

    @staticmethod
    def _fit(dst: torch.Tensor, full: torch.Tensor) -> None:
        if dst.shape != full.shape:
            raise ValueError(f"a tensor of shape {tuple(full.shape)} does not fit {tuple(dst.shape)}")
        dst.copy_(full)

    def load_conv(self, name: str, full: torch.Tensor) -> None:
        self._fit(self.conv1d.weight.data[self.offset[name]: self.offset[name] + self.shards[name]], full)

    def forward(self, x: torch.Tensor, fb) -> torch.Tensor:
        recurrent, conv = fb.extra["gdn_pool"].layer(self.gdn_index)
        m = gdn_batch(fb)
        o, C = self.offset, self.conv_dim
        y = ops.linear(x, self.in_proj.weight)
        second = ops.linear(y[:, self.inner], self.low_rank.weight)
        qkv = ops.causal_conv1d_silu(y[:, :C], self.conv1d.weight, conv, m.slots, m.lens, m.has_state, m.q_start, m.max_len)
        q = qkv[:, : o["k"]].unflatten(1, (self.kv_heads, self.dim))
        k = qkv[:, o["k"]: o["v"]].unflatten(1, (self.kv_heads, self.dim))
        v = qkv[:, o["v"]:].unflatten(1, (self.heads, self.vdim))
        r = ops.channel_delta_rule(q, k, v, y[:, o["b"]: o["b"] + self.heads], second[:, : self.decay_dim], self.A_log, self.dt_bias,
                                   recurrent, m.slots, m.lens, m.has_state, m.q_start, m.max_len)
        r = ops.rmsnorm_gated(r.reshape(-1, self.value_dim), second[:, self.gate_at: self.gate_at + self.value_dim], self.norm.weight,
                              self.eps, round_norm=False, sigmoid=True)
        return ops.linear(r, self.out_proj.weight)


class CausalConvolution(nn.Module):
    """``x + conv(x)``, a causal convolution over time on each channel without an activation.  The last taps - 1 inputs of a
    request live in its row of the state pool.  A decode step may leave the work to the kernel that writes ``x``
    (:meth:`step`)."""

    def __init__(self, channels: int, taps: int, gdn_index: int, params_dtype: torch.dtype) -> None:
        super().__init__()
        self.channels, self.taps, self.gdn_index = channels, taps, gdn_index
        self.weight = nn.Parameter(torch.zeros(channels, taps, dtype=params_dtype), requires_grad=False)

    @property
    def state_shape(self):
        return 0, 0, 0, self.channels, self.taps

    def step(self, fb) -> Optional["ops.ConvStep"]:
        """What the kernel in front needs to apply the convolution itself; None where rows have neighbours in the batch."""
        if not fb.forward_mode.is_decode():
            return None
        return ops.ConvStep(self.weight, fb.extra["gdn_pool"].layer(self.gdn_index)[1], gdn_batch(fb).slots)

    def forward(self, x: torch.Tensor, fb) -> torch.Tensor:
        m = gdn_batch(fb)
        return ops.causal_conv1d_silu(x, self.weight, fb.extra["gdn_pool"].layer(self.gdn_index)[1], m.slots, m.lens, m.has_state, m.q_start,
                                      m.max_len, add_input=True)
