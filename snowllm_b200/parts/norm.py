"""Norms over the hidden size, fused with the residual sum that precedes them: RMSNorm
(snowllm/ops/norm.py:11-30; snowllm/models/lfm2/layers.py:99-104) and Dynamic Tanh, which computes no
statistics at all: tanh(alpha * x) * weight + bias with one learned number alpha; the RMS norm in groups,
which also reads a residual stream that is kept as several streams; and the layer norm (centred, a weight, no bias)."""
from __future__ import annotations

import torch

from ..errors import ConfigError
from ..ops import kernels
from .base import Part
from .registry import register_norm
from .spec import INIT_BIAS, INIT_ONES, KEEP_F32, KEEP_SMALL, TensorSpec


class RMSNorm(Part):
    libraries = ("elementwise",)
    fusable_rms = True     # x * rsqrt(mean(x^2) + eps) * weight over the whole width: what a part that fuses
                           # the norm before it into its own first kernel may take over (weight, eps)

    def __init__(self, dtype, names, *, size: int, eps: float, offset: float = 0.0):
        """``offset``: a constant added to the stored weight (1 for weights stored around zero); the sum is kept in
        float."""
        super().__init__(dtype, names)
        self.size, self.eps, self.offset = size, eps, float(offset)
        self.weight = None

    def declare(self, has):
        if self.offset:
            return [TensorSpec("weight", self.names["weight"], (self.size,), INIT_BIAS, KEEP_F32)]
        return [TensorSpec("weight", self.names["weight"], (self.size,), INIT_ONES, KEEP_SMALL)]

    def bind(self, tensors):
        self.weight = tensors["weight"] + self.offset if self.offset else tensors["weight"]

    def forward(self, ctx, residual, delta=None, rows=None):
        """``residual += delta`` in float, then the norm of the sum in the compute dtype.  With
        ``rows`` (int32 row numbers) only those rows come out and the residual stays untouched.  A
        ``kernels.NormedDelta`` is applied with its own norm, gate and depth average."""
        return kernels.add_rmsnorm(residual, delta, self.weight, self.eps, self.dtype, rows=rows)

    def add_normed(self, ctx, residual, y):
        """``residual += norm(y)`` for a sublayer's float output ``y`` (the norm on the output side);
        returns the new residual in the compute dtype (the residual itself when that is float)."""
        same = residual.dtype == self.dtype
        x = kernels.norm_add(residual, y, self.weight, self.eps, self.dtype, want_x=not same)
        return residual if same else x


class DynamicTanh(Part):
    """tanh(alpha * x) * weight + bias, elementwise, in float: no mean, no variance, no eps.  Tensors:
    ``weight`` [size], ``bias`` [size], ``alpha`` (one number)."""
    libraries = ("sublayer",)
    fusable_rms = False

    def __init__(self, dtype, names, *, size: int):
        super().__init__(dtype, names)
        self.size = size
        self.weight = self.bias = self.alpha = None

    def declare(self, has):
        n = self.names
        return [TensorSpec("weight", n["weight"], (self.size,), INIT_ONES, KEEP_SMALL),
                TensorSpec("bias", n["bias"], (self.size,), INIT_BIAS, KEEP_SMALL),
                TensorSpec("alpha", n["alpha"], (), INIT_ONES, KEEP_SMALL)]

    def bind(self, tensors):
        self.weight, self.bias, self.alpha = tensors["weight"], tensors["bias"], tensors["alpha"]

    def forward(self, ctx, residual, delta=None, rows=None):
        """``residual += delta`` in float (a tensor, an ``ExpertSum`` or the ``DeltaSum`` of a layer whose
        two sublayers ran side by side), then the norm of the sum in the compute dtype.  With ``rows`` only
        those rows come out and the residual stays untouched."""
        return kernels.add_dyt(residual, delta, self.weight, self.bias, self.alpha, self.dtype, rows=rows)


class GroupRMSNorm(Part):
    """RMS norm in ``groups`` equal consecutive parts of the width: each part over its own
    sqrt(mean(part^2) + eps), the whole times ``weight``.  ``groups`` 1 is the plain RMS norm.  It reads a plain
    float residual (``residual += delta`` first) or, when ``delta`` is a ``kernels.StreamsDelta``, a stream
    kept as several streams: the pending update is applied and the streams are read with ``read`` weights
    (None: their plain sum), all in the one kernel."""
    libraries = ("streams",)
    fusable_rms = False

    def __init__(self, dtype, names, *, size: int, eps: float, groups: int = 1):
        super().__init__(dtype, names)
        if groups < 1 or size % groups:
            raise ConfigError(f"a norm over {size} in {groups} groups: the width must be a multiple of the groups")
        self.size, self.eps, self.groups = size, float(eps), int(groups)
        self.weight = None

    def declare(self, has):
        return [TensorSpec("weight", self.names["weight"], (self.size,), INIT_ONES, KEEP_SMALL)]

    def bind(self, tensors):
        self.weight = tensors["weight"]

    def read_streams(self, ctx, streams, *, init=None, update=None, read=None, rows=None):
        """The norm of sum_s read[s] X[s] after ``init`` and the pending ``update`` have been applied."""
        return kernels.streams_norm(streams, self.weight, self.groups, self.eps, self.dtype, init=init,
                                    update=update, read=read, rows=rows)

    def forward(self, ctx, residual, delta=None, rows=None):
        if isinstance(delta, kernels.StreamsDelta):
            return self.read_streams(ctx, delta.streams, update=delta, rows=rows)
        # one stream: the residual itself, with the identity as its update
        M, W = residual.shape
        one = ctx.memo.get("streams_identity")
        if one is None:
            one = ctx.memo["streams_identity"] = torch.ones(1, 1, dtype=torch.float32, device=residual.device)
        streams, update = residual.view(M, 1, W), None
        if delta is not None:
            update = kernels.StreamsDelta(streams, delta, one, one.view(1))
        return self.read_streams(ctx, streams, update=update, rows=rows)


class LayerNorm(Part):
    """(x - mean) / sqrt(mean((x - mean)^2) + eps) * weight * gain, statistics and weight in float.  ``gain``: a constant
    on the output (a model that scales its logits puts the factor into the norm before its head)."""
    libraries = ("layer_norm",)
    fusable_rms = False

    def __init__(self, dtype, names, *, size: int, eps: float, gain: float = 1.0):
        super().__init__(dtype, names)
        self.size, self.eps, self.gain = size, float(eps), float(gain)
        self.weight = None

    def declare(self, has):
        return [TensorSpec("weight", self.names["weight"], (self.size,), INIT_ONES, KEEP_F32)]

    def bind(self, tensors):
        self.weight = tensors["weight"]

    def forward(self, ctx, residual, delta=None, rows=None):
        """``residual += delta`` in float (a tensor, any of the deltas in pieces, or a ``kernels.NormedDelta`` with a norm
        of its own), then the norm of the sum in the compute dtype.  With ``rows`` only those rows come out and the
        residual stays untouched."""
        return kernels.layer_norm(residual, delta, self.weight, self.eps, self.dtype, gain=self.gain, rows=rows)


register_norm("layernorm", LayerNorm)
register_norm("rmsnorm", RMSNorm)
register_norm("group_rmsnorm", GroupRMSNorm)
register_norm("dyt", DynamicTanh)
