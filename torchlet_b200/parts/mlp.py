"""A feed-forward without a gate: y = W_down act(W_up x + b_up) + b_down, act = the square of relu.

In bfloat16 the first product runs with its bias and the activation in the tcgen05 kernel's epilogue; in float32, and at
sizes that kernel does not take, the activation is a kernel of its own behind the product.

Parameters: ``hidden_size``, ``intermediate_size``, ``activation`` ("relu_squared"), ``bias`` (default False), and the
tensors' names below the prefix: ``up_name``, ``down_name`` (defaults "up", "down"; a bias is the matrix's name +
``bias_suffix``, default ".b").
"""
from __future__ import annotations

import torch

from .. import ops
from ..config.spec import PartSpec
from .base import FEED_FORWARDS, FeedForward, TensorSpec
from .linear import Linear


@FEED_FORWARDS.register("mlp")
class MLP(FeedForward):
    def __init__(self, spec: PartSpec):
        super().__init__(spec)
        p = spec.params
        self.hidden_size = int(p["hidden_size"])
        self.intermediate_size = int(p["intermediate_size"])
        self.bias = bool(p.get("bias", False))
        if p.get("activation", "relu_squared") != "relu_squared":
            raise ValueError(f"unknown activation {p['activation']!r} (known: relu_squared)")
        self.up_proj: Linear | None = None
        self.down_proj: Linear | None = None

    @classmethod
    def _names(cls, spec: PartSpec, prefix: str):
        p = spec.params
        return prefix + p.get("up_name", "up"), prefix + p.get("down_name", "down"), p.get("bias_suffix", ".b")

    @classmethod
    def expected_tensors(cls, spec: PartSpec, prefix: str) -> list[TensorSpec]:
        hidden, inter = int(spec.params["hidden_size"]), int(spec.params["intermediate_size"])
        up, down, suffix = cls._names(spec, prefix)
        out = [TensorSpec(up, (inter, hidden)), TensorSpec(down, (hidden, inter))]
        if spec.params.get("bias", False):
            out += [TensorSpec(up + suffix, (inter,), init="zeros"), TensorSpec(down + suffix, (hidden,), init="zeros")]
        return out

    def load(self, tensors: dict, prefix: str, device, dtype) -> None:
        up, down, suffix = self._names(self.spec, prefix)
        self.up_proj = Linear(tensors[up], tensors[up + suffix] if self.bias else None, device, dtype)
        self.down_proj = Linear(tensors[down], tensors[down + suffix] if self.bias else None, device, dtype)

    def forward(self, ctx, x, acc) -> None:
        act = ctx.buffer("mlp.act", (x.shape[0], self.intermediate_size), ctx.dtype)
        if ctx.dtype == torch.bfloat16 and ops.gemm_tc_supported(x, self.up_proj.weight):
            ops.gemm_tc(x, self.up_proj.weight, act, self.up_proj.bias, ops.EPI_RELU2_BF16)
        else:
            self.up_proj.forward(x, act)
            ops.relu_squared_(act)
        if not self.down_proj.accumulate_later(ctx, act, acc):
            self.down_proj.forward(act, acc, accumulate=True)
