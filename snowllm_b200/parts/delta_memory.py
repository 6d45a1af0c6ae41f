"""The gated delta rule (kind ``delta_rule``): a matrix memory with a decay per key channel that takes off what it already
answers to a key before it writes, with a state of fixed size per request (csrc/delta_memory.cu).

One fused product gives q, k ([kv heads, dk]), v ([heads, dv]) and a logit per head.  q, k and v pass a short causal
convolution over time (depthwise; the last ``conv_taps`` - 1 projected rows of a request are state) and silu; q and k
become unit vectors per head, q times dk^(-1/2).  Per head a float matrix S [dk, dv], zero for a fresh request:

    S <- diag(a_t) S;   u = beta_t (v_t - S^T k_t);   S <- S + k_t u^T;   o_t = S^T q_t

beta = sigmoid of the logit, a = exp(-exp(a_log) softplus(W_b (W_a x) + dt_bias)) per head and channel.  Each head's o is
divided by its root mean square, weighted by ``norm`` [dv] (shared by the heads), multiplied by sigmoid of a second
low-rank product, and projected out.  Lengths, decays, betas, state, sums and the per-head statistics are float in every
dtype; the projections and the convolved rows are in the compute dtype."""
from __future__ import annotations

import torch

from ..errors import ConfigError
from ..ops import kernels, linear
from .attention_maps import pad_rows
from .base import Part
from .decay_memory import MAX_HEAD_DIM, LowRank
from .registry import register_mixer
from .spec import INIT_BIAS, INIT_CONV, INIT_ONES, KEEP_F32, SlotStateSpec, TensorSpec

MAX_CONV_TAPS = 16


class DeltaRule(Part):
    libraries = ("gemm", "gemm_skinny", "gemm_tc", "gemm_tc2", "short_conv", "delta_memory", "sublayer")
    DEFAULT_RANK = 16          # of drawn weights when the configuration names none

    def __init__(self, dtype, names, *, hidden_size: int, num_heads: int, num_kv_heads: int, head_dim: int,
                 v_head_dim: int, conv_taps: int, unit_eps: float, head_norm_eps: float, decay_rank: int | None = None,
                 gate_rank: int | None = None):
        super().__init__(dtype, names)
        if num_heads % num_kv_heads:
            raise ConfigError(f"{num_heads} memory heads over {num_kv_heads} q/k heads")
        if not 1 <= head_dim <= MAX_HEAD_DIM or not 1 <= conv_taps <= MAX_CONV_TAPS:
            raise ConfigError(f"head_dim={head_dim}, conv_taps={conv_taps}: the kernels take up to {MAX_HEAD_DIM} and "
                              f"{MAX_CONV_TAPS}")
        self.hidden_size, self.num_heads, self.num_kv_heads = hidden_size, num_heads, num_kv_heads
        self.head_dim, self.v_head_dim, self.conv_taps = head_dim, v_head_dim, conv_taps
        self.unit_eps, self.head_norm_eps = float(unit_eps), float(head_norm_eps)
        self.decay_rank, self.gate_rank = decay_rank, gate_rank
        self.w_in = self.wo = self.conv_w = self.low = self.norm = self.dt_bias = self.rate = None

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
        rd, rg = (r if r is not None else -1 for r in (self.decay_rank, self.gate_rank))
        low = dict(free_default=self.DEFAULT_RANK)
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
        proj, low = linear(x, self.w_in), self.low(x)
        history = cache.tensors[1] if self.conv_taps > 1 else proj.new_empty(1, 0, C)
        u = kernels.causal_conv(proj, C, self.conv_w, history, ctx.cu_seqlens, ctx.seg_start, ctx.seg_slot, ctx.row_seg,
                                silu=True)
        ctx.tap("memory_in", u)
        raw = kernels.delta_memory(u, 0, G * dk, 2 * G * dk, low, 0, self.dt_bias, self.rate, proj, C, ctx.cu_seqlens,
                                   ctx.seg_start, ctx.seg_slot, cache.tensors[0], G, max(ctx.host_seg_len),
                                   unit_eps=self.unit_eps, q_scale=dk ** -0.5)
        ctx.tap("memory_raw", raw)
        heads = kernels.head_norm_gate(raw, H, dv, self.head_norm_eps, self.dtype, weight=self.norm, gate=low,
                                       gate_col=H * dk)
        return linear(heads, self.wo, out_dtype=torch.float32)


register_mixer("delta_rule", DeltaRule)
