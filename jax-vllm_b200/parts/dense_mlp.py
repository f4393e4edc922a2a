"""A feed-forward without a gate: down(act(up(x))), no bias, act by name: relu(z)^2, the exact gelu, tanh, or "poly_norm",
a N(z) + b N(z^2) + c N(z^3) + e with four numbers of a tensor, which norms a token's whole vector (csrc/poly_norm.cu).

Like the attention mixers it offers its two products to an arrangement that packs them with another part's
(`in_weight`, `from_projection`, `out_weight`)."""

from __future__ import annotations

import torch

from .. import ops
from .base import Part, TensorSpec
from .registry import register_feed_forward


class DenseMLP(Part):
    kernels = ("activation", "gemm_simt")

    def __init__(self, spec, prefix, ctx):
        self.poly = spec.activation == "poly_norm"
        if not self.poly and spec.activation not in ops.UNARY_ACTIVATIONS:
            raise ValueError(f"feed-forward: activation {spec.activation!r} is not built "
                             f"({', '.join(ops.UNARY_ACTIVATIONS)} and poly_norm are)")
        if self.poly:
            self.kernels = ("poly_norm", "gemm_simt")
        self.spec, self.ctx = spec, ctx
        self.prefix = f"{prefix}.{spec.prefix}" if spec.prefix else prefix
        self.in_rows = self.heads_out = spec.intermediate_size
        self.w_up = self.w_down = self.coef = None

    def _names(self):
        return tuple(f"{self.prefix}.{n}" for n in self.spec.names)

    def tensor_specs(self):
        up, down, act = self._names()
        s = self.spec
        out = {up: TensorSpec((s.intermediate_size, s.hidden_size)), down: TensorSpec((s.hidden_size, s.intermediate_size))}
        if self.poly:
            out[act] = TensorSpec((4,), kind="vector", init="ones_normal")
        return out

    def bind(self, tensors):
        up, down, act = self._names()
        if self.poly:
            self.coef = tensors[act].contiguous()
        self.w_up = self.compute_weight(tensors[up], self.ctx).contiguous()
        self.w_down = self.compute_weight(tensors[down], self.ctx).contiguous()

    def in_weight(self) -> torch.Tensor:
        return self.w_up

    def out_weight(self) -> torch.Tensor:
        return self.w_down

    def from_projection(self, z, step, out=None):
        if self.poly:
            return ops.poly_norm(z, self.coef, self.spec.norm_eps, out, out_dtype=self.ctx.dtype)
        return ops.unary_act(z, self.spec.activation, out)

    def forward(self, x, step):
        dt = self.ctx.dtype
        z = ops.linear(x, self.w_up, dt, parts_ok=self.poly)      # a few rows: maybe parts of a sum, added as they are read
        return ops.linear(self.from_projection(z, step), self.w_down, dt, parts_ok=True)


register_feed_forward("dense_mlp", DenseMLP)
