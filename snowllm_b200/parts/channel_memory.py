"""Matrix memories with a decay per head and key channel and a state of fixed size per request
(csrc/channel_memory.cu).  Per head a float matrix S [dk, dv], zero for a fresh request:

    S <- diag(a_t) S;   S <- S + k_t w_t^T;   o_t = S^T q_t

* ``gated_linear`` (gated linear attention): w = v; a_t = sigmoid(z)^(1/tau) with z = W_b (W_a x) + bias; q = W_q x *
  dk^(-1/2), k = W_k x, v = W_v x.  Each head's o is divided by its root mean square and weighted by ``norm`` [dv]
  (shared by the heads), multiplied by silu(W_g x), then the output product.
* ``delta_rule`` (the gated delta rule): the memory takes off what it already answers to a key before it writes, w =
  beta_t (v_t - S^T k_t).  q, k ([kv heads, dk]) and v ([heads, dv]) pass a short causal convolution over time
  (depthwise; the last ``conv_taps`` - 1 projected rows of a request are state) and silu; q and k become unit vectors per
  head, q times dk^(-1/2).  beta = sigmoid of a logit per head, a = exp(-exp(a_log) softplus(W_b (W_a x) + dt_bias)).
  Each head's o is divided by its root mean square, weighted by ``norm`` [dv], multiplied by sigmoid of a second
  low-rank product, and projected out.

Lengths, decays, betas, state, sums and the per-head statistics are float in every dtype; the projections and the
convolved rows are in the compute dtype."""
from __future__ import annotations

import torch

from ..errors import ConfigError
from ..ops import kernels, linear
from .attention_maps import pad_rows
from .base import Part
from .decay_memory import MAX_HEAD_DIM, memory_pieces
from .registry import register_mixer
from .spec import INIT_BIAS, INIT_CONV, INIT_ONES, KEEP_F32, SlotStateSpec, TensorSpec

MAX_CONV_TAPS = 16


class LowRank:
    """W_b W_a for two thin matrices [r, in] and [out, r], kept apart; r is padded with zeros to a multiple of 8, the
    length the tensor-core products take.  Several pairs share the two launches: their W_a side by side, their W_b on the
    diagonal of one matrix (the zeros between them add nothing)."""

    def __init__(self, pairs, what: str):
        for a, b in pairs:
            if a.shape[0] != b.shape[1]:
                raise ConfigError(f"{what}: low-rank matrices of ranks {a.shape[0]} and {b.shape[1]}")
        self.a = pad_rows(torch.cat([a for a, _ in pairs], 0), 8)
        n, r = sum(b.shape[0] for _, b in pairs), self.a.shape[0]
        self.b = self.a.new_zeros(n, r)
        row = col = 0
        for _, b in pairs:
            self.b[row:row + b.shape[0], col:col + b.shape[1]] = b
            row, col = row + b.shape[0], col + b.shape[1]

    def __call__(self, x):
        """Float [M, out], the pairs' outputs side by side."""
        return linear(linear(x, self.a), self.b, out_dtype=torch.float32)


class _ChannelMemory(Part):
    DEFAULT_RANK = 16          # of drawn weights when the configuration names none

    def __init__(self, dtype, names, *, hidden_size: int, num_heads: int, head_dim: int, v_head_dim: int,
                 head_norm_eps: float, decay_rank: int | None = None):
        super().__init__(dtype, names)
        if not 1 <= head_dim <= MAX_HEAD_DIM:
            raise ConfigError(f"memory heads of {head_dim} rows: the kernels keep up to {MAX_HEAD_DIM}")
        self.hidden_size, self.num_heads, self.head_dim, self.v_head_dim = hidden_size, num_heads, head_dim, v_head_dim
        self.head_norm_eps, self.decay_rank = float(head_norm_eps), decay_rank
        self.w_in = self.wo = self.low = self.norm = self._rides = None

    def ride_in(self, host) -> None:
        """Let another part's first product on the same rows form the projections (``Part``)."""
        self._rides = (host, host.append_input_rows(self.w_in))
        self.w_in = None

    def _projected(self, ctx, x):
        """(the projection's rows in the compute dtype, the first of their columns)."""
        if self._rides is not None:
            host, col = self._rides
            return host.input_rows(ctx), col
        return linear(x, self.w_in), 0

    def _low_rank(self, rank) -> tuple:
        """(rank as a tensor dimension, what a TensorSpec says about it): the checkpoint's to choose unless given."""
        return (rank if rank is not None else -1), dict(free_default=self.DEFAULT_RANK)


class GatedLinear(_ChannelMemory):
    libraries = ("gemm", "gemm_skinny", "gemm_tc", "gemm_tc2", "channel_memory", "sublayer")

    def __init__(self, dtype, names, *, tau: float, **kw):
        super().__init__(dtype, names, **kw)
        self.tau = float(tau)
        self.decay_bias = None

    def cache_spec(self):
        return SlotStateSpec(((self.num_heads, self.head_dim, self.v_head_dim),), ("f32",))

    def declare(self, has):
        W, H, dk, dv, n = self.hidden_size, self.num_heads, self.head_dim, self.v_head_dim, self.names
        r, low = self._low_rank(self.decay_rank)
        return [TensorSpec("q_proj", n["q_proj"], (H * dk, W)), TensorSpec("k_proj", n["k_proj"], (H * dk, W)),
                TensorSpec("v_proj", n["v_proj"], (H * dv, W)), TensorSpec("gate_proj", n["gate_proj"], (H * dv, W)),
                TensorSpec("decay_a", n["decay_a"], (r, W), **low),
                TensorSpec("decay_b", n["decay_b"], (H * dk, r), **low),
                TensorSpec("decay_bias", n["decay_bias"], (H * dk,), INIT_BIAS, KEEP_F32),
                TensorSpec("norm", n["norm"], (dv,), INIT_ONES, KEEP_F32),
                TensorSpec("out_proj", n["out_proj"], (W, H * dv))]

    def bind(self, tensors):
        self.w_in = pad_rows(torch.cat([tensors[k] for k in ("q_proj", "k_proj", "v_proj", "gate_proj")], 0), 16)
        self.low = LowRank([(tensors["decay_a"], tensors["decay_b"])], "gated linear attention")
        self.wo, self.decay_bias = tensors["out_proj"], tensors["decay_bias"].contiguous()
        self.norm = tensors["norm"].repeat(self.num_heads).contiguous()      # one weight for every head

    def forward(self, ctx, x, cache, owns_cache=True):
        H, dk, dv = self.num_heads, self.head_dim, self.v_head_dim
        proj, col = self._projected(ctx, x)
        raw = kernels.channel_memory(proj, col, col + H * dk, col + 2 * H * dk, self.low(x), 0, self.decay_bias, ctx.cu_seqlens,
                                     ctx.seg_start, ctx.seg_slot, cache.tensors[0], H, max(ctx.host_seg_len),
                                     sharp=1.0 / self.tau, q_scale=dk ** -0.5,
                                     pieces=memory_pieces(ctx, kernels.MEMORY_CHUNK))
        ctx.tap("memory_raw", raw)
        heads = kernels.head_norm_gate(raw, H, dv, self.head_norm_eps, self.dtype, weight=self.norm, gate=proj,
                                       gate_col=col + 2 * H * dk + H * dv, gate_act="silu")
        return linear(heads, self.wo, out_dtype=torch.float32)


class DeltaRule(_ChannelMemory):
    libraries = ("gemm", "gemm_skinny", "gemm_tc", "gemm_tc2", "short_conv", "channel_memory", "sublayer")

    def __init__(self, dtype, names, *, num_kv_heads: int, conv_taps: int, unit_eps: float, gate_rank: int | None = None,
                 **kw):
        super().__init__(dtype, names, **kw)
        if self.num_heads % num_kv_heads:
            raise ConfigError(f"{self.num_heads} memory heads over {num_kv_heads} q/k heads")
        if not 1 <= conv_taps <= MAX_CONV_TAPS:
            raise ConfigError(f"conv_taps={conv_taps}: the kernel takes up to {MAX_CONV_TAPS}")
        self.num_kv_heads, self.conv_taps, self.unit_eps, self.gate_rank = num_kv_heads, conv_taps, float(unit_eps), gate_rank
        self.conv_w = self.dt_bias = self.rate = None

    @property
    def conv_channels(self) -> int:
        return 2 * self.num_kv_heads * self.head_dim + self.num_heads * self.v_head_dim

    def cache_spec(self):
        state = (self.num_heads, self.head_dim, self.v_head_dim)
        if self.conv_taps <= 1:
            return SlotStateSpec((state,), ("f32",))
        return SlotStateSpec((state, (self.conv_taps - 1, self.conv_channels)), ("f32", "compute"))

    def declare(self, has):
        W, H, G, n = self.hidden_size, self.num_heads, self.num_kv_heads, self.names
        dk, dv, L = self.head_dim, self.v_head_dim, self.conv_taps
        (rd, low), (rg, _) = self._low_rank(self.decay_rank), self._low_rank(self.gate_rank)
        return [TensorSpec("q_proj", n["q_proj"], (G * dk, W)), TensorSpec("k_proj", n["k_proj"], (G * dk, W)),
                TensorSpec("v_proj", n["v_proj"], (H * dv, W)), TensorSpec("beta_proj", n["beta_proj"], (H, W)),
                TensorSpec("q_conv", n["q_conv"], (G * dk, L), INIT_CONV, KEEP_F32),
                TensorSpec("k_conv", n["k_conv"], (G * dk, L), INIT_CONV, KEEP_F32),
                TensorSpec("v_conv", n["v_conv"], (H * dv, L), INIT_CONV, KEEP_F32),
                TensorSpec("decay_a", n["decay_a"], (rd, W), **low), TensorSpec("decay_b", n["decay_b"], (H * dk, rd), **low),
                TensorSpec("gate_a", n["gate_a"], (rg, W), **low), TensorSpec("gate_b", n["gate_b"], (H * dv, rg), **low),
                TensorSpec("a_log", n["a_log"], (H,), INIT_BIAS, KEEP_F32),
                TensorSpec("dt_bias", n["dt_bias"], (H * dk,), INIT_BIAS, KEEP_F32),
                TensorSpec("norm", n["norm"], (dv,), INIT_ONES, KEEP_F32),
                TensorSpec("out_proj", n["out_proj"], (W, H * dv))]

    def bind(self, tensors):
        self.w_in = pad_rows(torch.cat([tensors[k] for k in ("q_proj", "k_proj", "v_proj", "beta_proj")], 0), 16)
        self.conv_w = torch.cat([tensors[k] for k in ("q_conv", "k_conv", "v_conv")], 0).contiguous()
        self.low = LowRank([(tensors["decay_a"], tensors["decay_b"]), (tensors["gate_a"], tensors["gate_b"])], "delta rule")
        self.wo, self.dt_bias = tensors["out_proj"], tensors["dt_bias"].contiguous()
        self.rate = (-torch.exp(tensors["a_log"])).contiguous()
        self.norm = tensors["norm"].repeat(self.num_heads).contiguous()      # one weight for every head

    def forward(self, ctx, x, cache, owns_cache=True):
        H, G, dk, dv, C = self.num_heads, self.num_kv_heads, self.head_dim, self.v_head_dim, self.conv_channels
        (proj, col), low = self._projected(ctx, x), self.low(x)
        history = cache.tensors[1] if self.conv_taps > 1 else proj.new_empty(1, 0, C)
        u = kernels.causal_conv(proj, C, self.conv_w, history, ctx.cu_seqlens, ctx.seg_start, ctx.seg_slot, ctx.row_seg,
                                silu=True, col=col)
        ctx.tap("memory_in", u)
        raw = kernels.channel_memory(u, 0, G * dk, 2 * G * dk, low, 0, self.dt_bias, ctx.cu_seqlens, ctx.seg_start,
                                     ctx.seg_slot, cache.tensors[0], G, max(ctx.host_seg_len), rate=self.rate, beta=proj,
                                     beta_col=col + C, q_scale=dk ** -0.5, unit_eps=self.unit_eps,
                                     pieces=memory_pieces(ctx, kernels.MEMORY_CHUNK))
        ctx.tap("memory_raw", raw)
        heads = kernels.head_norm_gate(raw, H, dv, self.head_norm_eps, self.dtype, weight=self.norm, gate=low,
                                       gate_col=H * dk)
        return linear(heads, self.wo, out_dtype=torch.float32)


register_mixer("gated_linear", GatedLinear)
register_mixer("delta_rule", DeltaRule)
