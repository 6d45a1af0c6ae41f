"""An input of a layer's own from the token ids, added after the layer's sublayers.

The embedding keeps a second table with one row per token (``Embedding(side_size=)``); layer ``index`` owns the columns
[index * dim, (index + 1) * dim) of it, e.  With x the residual stream:

    y = W_proj (gelu(W_gate x) * e),      x <- x + y / rms(y) * norm

The block calls ``forward`` in place of leaving its last delta to the next norm: x is brought up to date, rounded to the
compute dtype for the gate's product, and the update stays pending as a ``kernels.NormedDelta``."""
from __future__ import annotations

import torch

from ..errors import KernelError
from ..ops import kernels, linear
from .base import Part
from .spec import INIT_ONES, KEEP_F32, TensorSpec

TABLE = "token_side_table"          # the memo key under which the embedding leaves its second table


class TokenSide(Part):
    libraries = ("gemm", "gemm_skinny", "gemm_tc", "gemm_tc2", "layer_norm")

    def __init__(self, dtype, names, *, hidden_size: int, dim: int, index: int, eps: float):
        super().__init__(dtype, names)
        self.hidden_size, self.dim, self.index, self.eps = hidden_size, int(dim), int(index), float(eps)
        self.gate = self.proj = self.norm = None

    def declare(self, has):
        W, d, n = self.hidden_size, self.dim, self.names
        return [TensorSpec("gate", n["gate"], (d, W)), TensorSpec("proj", n["proj"], (W, d)),
                TensorSpec("norm", n["norm"], (W,), INIT_ONES, KEEP_F32)]

    def bind(self, tensors):
        self.gate, self.proj, self.norm = tensors["gate"], tensors["proj"], tensors["norm"]

    def forward(self, ctx, residual, delta):
        """``residual += delta`` at once; this part's own update is returned pending."""
        if TABLE not in ctx.memo:
            raise KernelError("a layer with an input from the token ids needs an embedding with side rows")
        x = kernels.layer_norm(residual, delta, None, 0.0, self.dtype)
        g = linear(x, self.gate, out_dtype=torch.float32)
        act = kernels.side_gate(g, ctx.memo[TABLE], ctx.token_ids, self.index * self.dim, self.dtype,
                                pending=ctx.pending_tokens)
        ctx.tap("token_side_gate", act)
        return kernels.NormedDelta(linear(act, self.proj, out_dtype=torch.float32), weight=self.norm, eps=self.eps)
