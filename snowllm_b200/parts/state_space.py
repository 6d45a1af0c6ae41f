"""Selective state-space mixer (Mamba-2, kind ``mamba2``) with a state of fixed size per request
(csrc/state_space.cu).

One fused product gives z, x, B, C and dt.  x, B and C pass a short causal convolution over time (depthwise, with a
bias; the last ``conv_taps`` - 1 projected rows of a request are state) and silu.  Per head a float matrix S
[state_size, head_dim], zero for a fresh request:

    step = softplus(dt + dt_bias);  S_t = exp(-exp(a_log) step) S_(t-1) + step B_t x_t^T;  y_t = S_t^T C_t + skip x_t

(B and C are shared by the heads of a group).  y times silu(z) is divided by its root mean square in ``norm_groups``
equal parts, weighted and projected out.  Steps, decays, state, sums, gate and norm are float in every dtype; the
projection and the convolved rows are in the compute dtype."""
from __future__ import annotations

import torch

from ..errors import ConfigError
from ..ops import kernels, linear
from .attention_maps import pad_rows
from .base import Part
from .registry import register_mixer
from .spec import INIT_BIAS, INIT_CONV, INIT_ONES, KEEP_F32, KEEP_SMALL, SlotStateSpec, TensorSpec

MAX_STATE = 256
MAX_CONV_TAPS = 16


class Mamba2(Part):
    libraries = ("gemm", "gemm_skinny", "gemm_tc", "gemm_tc2", "short_conv", "state_space")
    _lends_rows = False        # whether the projection carries rows of another part (``append_input_rows``)

    def __init__(self, dtype, names, *, hidden_size: int, num_heads: int, head_dim: int, state_size: int,
                 num_groups: int = 1, norm_groups: int = 1, conv_taps: int = 4, norm_eps: float):
        super().__init__(dtype, names)
        if num_heads % num_groups:
            raise ConfigError(f"{num_heads} state-space heads in {num_groups} groups")
        if (num_heads * head_dim) % norm_groups:
            raise ConfigError(f"a norm over {num_heads * head_dim} in {norm_groups} parts")
        if not 1 <= state_size <= MAX_STATE or not 1 <= conv_taps <= MAX_CONV_TAPS:
            raise ConfigError(f"state_size={state_size}, conv_taps={conv_taps}: the kernels take up to {MAX_STATE} and "
                              f"{MAX_CONV_TAPS}")
        self.hidden_size, self.num_heads, self.head_dim = hidden_size, num_heads, head_dim
        self.state_size, self.num_groups, self.norm_groups = state_size, num_groups, norm_groups
        self.conv_taps, self.norm_eps = conv_taps, float(norm_eps)
        self.w_in = self.wo = self.conv_w = self.conv_b = self.norm = None
        self.dt_bias = self.rate = self.skip = None

    @property
    def inner(self) -> int:
        return self.num_heads * self.head_dim

    @property
    def conv_channels(self) -> int:
        return self.inner + 2 * self.num_groups * self.state_size

    def _columns(self):
        """Columns of the projection as it is kept: (z, dt); the convolved ones (x, B, C) come first."""
        z = self.conv_channels
        return z, z + self.inner

    def cache_spec(self):
        state = (self.num_heads, self.state_size, self.head_dim)
        if self.conv_taps <= 1:
            return SlotStateSpec((state,), ("f32",))
        return SlotStateSpec((state, (self.conv_taps - 1, self.conv_channels)), ("f32", "compute"))

    def declare(self, has):
        W, H, n = self.hidden_size, self.num_heads, self.names
        C = self.conv_channels
        return [TensorSpec("in_proj", n["in_proj"], (self.inner + C + H, W)),
                TensorSpec("conv", n["conv"], (C, self.conv_taps), INIT_CONV, KEEP_F32),
                TensorSpec("conv_bias", n["conv_bias"], (C,), INIT_BIAS, KEEP_F32),
                TensorSpec("dt_bias", n["dt_bias"], (H,), INIT_BIAS, KEEP_F32),
                TensorSpec("a_log", n["a_log"], (H,), INIT_BIAS, KEEP_F32),
                TensorSpec("skip", n["skip"], (H,), INIT_ONES, KEEP_F32),
                TensorSpec("norm", n["norm"], (self.inner,), INIT_ONES, KEEP_SMALL),
                TensorSpec("out_proj", n["out_proj"], (W, self.inner))]

    def bind(self, tensors):
        inner, C = self.inner, self.conv_channels
        z, xbc, dt = torch.split(tensors["in_proj"], [inner, C, self.num_heads], 0)
        self.w_in = pad_rows(torch.cat((xbc, z, dt), 0), 16)
        self.wo, self.norm = tensors["out_proj"], tensors["norm"]
        self.conv_w, self.conv_b = tensors["conv"].contiguous(), tensors["conv_bias"].contiguous()
        self.dt_bias, self.skip = tensors["dt_bias"].contiguous(), tensors["skip"].contiguous()
        self.rate = (-torch.exp(tensors["a_log"].float())).contiguous()

    def append_input_rows(self, weight) -> int:
        """Further rows for the projection (``Part``): the column their outputs start at."""
        col = self.w_in.shape[0]
        self.w_in = pad_rows(torch.cat((self.w_in, weight), 0), 16)
        self._lends_rows = True
        return col

    def input_rows(self, ctx):
        return ctx.memo.pop(("input_rows", id(self)))

    def forward(self, ctx, x, cache, owns_cache=True):
        proj = linear(x, self.w_in)
        if self._lends_rows:
            ctx.memo[("input_rows", id(self))] = proj
        z_col, dt_col = self._columns()
        state = cache.tensors[0]
        history = cache.tensors[1] if self.conv_taps > 1 else proj.new_empty(1, 0, self.conv_channels)
        u = kernels.causal_conv(proj, self.conv_channels, self.conv_w, history, ctx.cu_seqlens, ctx.seg_start,
                                ctx.seg_slot, ctx.row_seg, bias=self.conv_b, silu=True)
        ctx.tap("state_space_in", u)
        b_off = self.inner
        y = kernels.state_space(u, 0, b_off, b_off + self.num_groups * self.state_size, proj, dt_col, self.dt_bias,
                                self.rate, self.skip, ctx.cu_seqlens, ctx.seg_start, ctx.seg_slot, state,
                                self.num_groups, max(ctx.host_seg_len))
        ctx.tap("state_space_out", y)
        heads = kernels.gate_group_norm(y, proj, z_col, self.norm, self.norm_groups, self.norm_eps)
        return linear(heads, self.wo, out_dtype=torch.float32)


register_mixer("mamba2", Mamba2)
