"""A gated recurrence whose gates read only the current token, element by element (csrc/min_gru.cu).

    z = sigmoid(W_z x + b_z),  y = W_x x + b_x,  candidate = y + 1/2 where y >= 0, sigmoid(y) elsewhere
    S <- (1 - z) S + z * candidate;   out = W_o (output_scale * S * silu(W_g x))

The state is a row of float32 in the request's state slot (`FixedStateNeed`, zero at a sequence's start); everything
from the projections on is 32-bit.  One product serves the three input matrices; the part offers its products to an
arrangement that packs them (`in_weight`, `from_projection`, `out_weight`).
"""

from __future__ import annotations

import torch

from .. import ops
from .base import FixedStateNeed, Part, TensorSpec
from .registry import register_mixer


class MinGRU(Part):
    kernels = ("min_gru", "gemm_simt")

    def __init__(self, spec, prefix, ctx):
        self.spec, self.ctx = spec, ctx
        self.prefix = f"{prefix}.{spec.prefix}" if spec.prefix else prefix
        self.c = int(spec.width)
        if self.c < 1:
            raise ValueError(f"{self.prefix}: a recurrence of {self.c} elements is not built")
        self.names = {k: f"{self.prefix}.{n}" for k, n in zip(("z", "z_b", "x", "x_b", "g", "o"), spec.names)}
        self.in_rows, self.heads_out = 3 * self.c, self.c
        self.w_in = self.w_o = self.z_bias = self.x_bias = None

    def tensor_specs(self):
        n, W, C = self.names, self.spec.hidden_size, self.c
        return {n["z"]: TensorSpec((C, W)), n["z_b"]: TensorSpec((C,), kind="vector", init="normal"),
                n["x"]: TensorSpec((C, W)), n["x_b"]: TensorSpec((C,), kind="vector", init="normal"),
                n["g"]: TensorSpec((C, W)), n["o"]: TensorSpec((W, C))}

    def bind(self, tensors):
        n = self.names
        mats = [self.compute_weight(tensors[n[k]], self.ctx) for k in ("z", "x", "g")]
        if len({m.dtype for m in mats}) > 1:
            mats = [m.to(torch.float32) for m in mats]
        self.w_in = torch.cat(mats, dim=0).contiguous()
        self.w_o = self.compute_weight(tensors[n["o"]], self.ctx).contiguous()
        self.z_bias = tensors[n["z_b"]].contiguous()
        self.x_bias = tensors[n["x_b"]].to(self.z_bias.dtype).contiguous()

    def cache_need(self):
        return FixedStateNeed((self.c,), torch.float32)

    def in_weight(self) -> torch.Tensor:
        return self.w_in

    def out_weight(self) -> torch.Tensor:
        return self.w_o

    def from_projection(self, row, step, cache, out):
        """`row` [n, 3 * width] (the packed projection, possibly a column range) -> the gated state, written to `out`
        [n, width] (possibly a column range)."""
        return ops.min_gru(row, 0, self.c, 2 * self.c, self.z_bias, self.x_bias, cache.state, step.cu_seqlens,
                           step.state_slots, step.n_entries, self.c, out, float(self.spec.output_scale))

    def forward_projected(self, row, step, cache):
        out = torch.empty((step.n_tokens, self.c), dtype=self.ctx.dtype, device=row.device)
        self.from_projection(row, step, cache, out)
        return ops.linear(out, self.w_o, self.ctx.dtype)

    def forward(self, x, step, cache):
        return self.forward_projected(ops.linear(x, self.w_in, self.ctx.dtype), step, cache)


register_mixer("min_gru", MinGRU)
