"""A mixture of small feed-forward experts, each down(act(up(x))), no biases; or, with the activation
"clamped_glu", experts with a gate matrix: g = min(W_gate x, limit), u = clamp(W_up x, -limit, limit),
down(g * sigmoid(1.702 g) * (u + 1)), or with "swiglu" down(silu(W_gate x) * (W_up x)) (the two matrices are stacked, the
activation is a kernel of its own).

    z        = x @ W_router^T           32-bit accumulation and result (ops.linear)
    ids, w   = route(z)                 softmax scores in 32-bit, group-limited choice of the top_k (csrc/moe_route.cu)
               or, with `scoring` "table", no router: a table names each token id's experts, all weights 1 / top_k
    order    = pairs sorted by expert   every expert's rows padded to a row tile (csrc/moe_route.cu, jv_moe_align)
    a        = act(x[token] @ W_up_e^T) grouped product, rows gathered as they are read, activation in its epilogue
    y        = a @ W_down_e^T           grouped product
    out[t]   = sum_k w[t, k] * y[pos(t, k)]     added up in 32-bit, k ascending, by the reader of the result

Options of the router: a correction per expert added to the scores for the choice only; identity experts behind the
others, whose output is x itself (the sum of their chosen weights goes with x: `PickedRows.own`).  A shared expert
(`shared_size`), down(silu(gate x) * (up x)) for every token, is added: its down product may be joined with another part's
(`out_weight`, `inner`); alone it gives an `ops.BranchSum`.

The result is handed on as an `ops.PickedRows` (rows of y, which to pick and with which weight): the norm that
follows adds them up as it reads them.  The expert matrices are kept stacked, [experts, out, in].
"""

from __future__ import annotations

import torch

from .. import ops
from ..config.model_spec import GatedMLPSpec
from .base import Part, TensorSpec
from .feed_forward import GatedMLP
from .registry import register_feed_forward


class RoutedExperts(Part):
    kernels = ("moe_route", "moe_gemm_simt", "gemm_simt")

    def __init__(self, spec, prefix, ctx):
        if spec.activation not in ("gelu", "clamped_glu", "swiglu"):
            raise ValueError(f"routed experts: activation {spec.activation!r} is not built (gelu, clamped_glu and swiglu are)")
        self.by_table = spec.scoring == "table"
        if (spec.scoring not in ops.ROUTER_SCORINGS and not self.by_table) or spec.group_score not in ops.GROUP_SCORES:
            raise ValueError(f"routed experts: scoring {spec.scoring!r} with group score {spec.group_score!r} is not "
                             f"built ({', '.join(ops.ROUTER_SCORINGS)}, table; {', '.join(ops.GROUP_SCORES)})")
        if self.by_table and (spec.n_groups != 1 or spec.vocab_size < 1):
            raise ValueError("routed experts: a table has a row per token id and knows no groups")
        self.gated = spec.activation in ("clamped_glu", "swiglu")
        if spec.activation == "clamped_glu" and not spec.limit > 0:
            raise ValueError("routed experts: the clamped activation needs a positive limit")
        if self.gated:
            self.kernels = ("moe_route", "moe_gemm_simt", "gemm_simt", "activation")
        if self.by_table and (spec.correction is not None or spec.identity):
            raise ValueError("routed experts: a table knows no correction and no identity experts")
        # the router's experts: those with tensors, then the identity experts
        E, n, keep = spec.num_experts + spec.identity, spec.n_groups, spec.keep_groups
        if E % n or not 1 <= keep <= n or not 1 <= spec.top_k <= keep * (E // n):
            raise ValueError(f"routed experts: {E} experts, {n} groups, {keep} kept, top {spec.top_k} do not fit")
        self.spec, self.ctx = spec, ctx
        self.prefix = f"{prefix}.{spec.prefix}" if spec.prefix else prefix
        self.w_router = self.table = self.w_up = self.w_down = self.correction = self.shared = None
        self.inner_size = int(spec.shared_size)
        if self.inner_size:
            self.shared = GatedMLP(GatedMLPSpec(spec.hidden_size, self.inner_size, prefix="shared",
                                                names=("gate", "up", "down")), self.prefix, ctx)

    def tensor_specs(self):
        p, s = self.prefix, self.spec
        if self.by_table:
            out = {f"{p}.table": TensorSpec((s.vocab_size, s.top_k), kind="table", below=s.num_experts)}
        else:
            out = {f"{p}.router": TensorSpec((s.num_experts + s.identity, s.hidden_size))}
            if s.correction is not None:
                out[f"{p}.{s.correction}"] = TensorSpec((s.num_experts + s.identity,), kind="vector", init="normal")
        for e in range(s.num_experts):
            if self.gated:
                out[f"{p}.e{e}.gate"] = TensorSpec((s.expert_size, s.hidden_size))
            out[f"{p}.e{e}.up"] = TensorSpec((s.expert_size, s.hidden_size))
            out[f"{p}.e{e}.down"] = TensorSpec((s.hidden_size, s.expert_size))
        if self.shared is not None:
            out.update(self.shared.tensor_specs())
        return out

    def bind(self, tensors):
        p, s = self.prefix, self.spec
        if self.by_table:
            self.table = tensors[f"{p}.table"].to(torch.int32).contiguous()
        else:
            self.w_router = self.compute_weight(tensors[f"{p}.router"], self.ctx).contiguous()
            if s.correction is not None:
                self.correction = tensors[f"{p}.{s.correction}"].to(torch.float32).contiguous()
        ups = [self.compute_weight(tensors[f"{p}.e{e}.up"], self.ctx) for e in range(s.num_experts)]
        if self.gated:      # [gate; up] of an expert stacked: one grouped product makes both
            gates = [self.compute_weight(tensors[f"{p}.e{e}.gate"], self.ctx) for e in range(s.num_experts)]
            if len({m.dtype for m in ups + gates}) > 1:
                ups, gates = [m.float() for m in ups], [m.float() for m in gates]
            ups = [torch.cat([g, u], dim=0) for g, u in zip(gates, ups)]
        downs = [self.compute_weight(tensors[f"{p}.e{e}.down"], self.ctx) for e in range(s.num_experts)]
        if len({m.dtype for m in ups + downs}) > 1:
            ups, downs = [m.float() for m in ups], [m.float() for m in downs]
        self.w_up = torch.stack(ups).contiguous()
        self.w_down = torch.stack(downs).contiguous()
        if self._tensor_cores():
            self.kernels = ("moe_route", "gemm_tcgen05", "gemm_simt") + (("activation",) if self.gated else ())
        if self.shared is not None:
            self.shared.bind(tensors)
            self.kernels += tuple(k for k in self.shared.kernels if k not in self.kernels)

    # The grouped tcgen05 product works on 128-row tiles of 256 columns: it is taken for bfloat16 experts whose inner
    # sizes it can address (multiples of 8) and whose matrices are at least this wide; smaller ones, and the 32-bit
    # path, go to the CUDA-core product with its 32-row tiles.
    TCGEN05_MIN_SIZE = 128

    def _tensor_cores(self) -> bool:
        s = self.spec
        return (ops.moe_gemm_tcgen05_supports(self.ctx.dtype, self.w_up) and ops.moe_gemm_tcgen05_supports(self.ctx.dtype, self.w_down)
                and min(s.expert_size, s.hidden_size) >= self.TCGEN05_MIN_SIZE)

    def _choose(self, x, step):
        """(experts, weights) [n, top_k] of every token, and with identity experts the weight [n] of the token itself."""
        s = self.spec
        if self.by_table:
            return ops.moe_route_table(step.token_ids, self.table, s.num_experts)
        logits = ops.linear(x, self.w_router, torch.float32)       # 32-bit accumulation, 32-bit result
        return ops.moe_route(logits, s.top_k, s.n_groups, s.keep_groups, s.renormalize, s.scoring, s.group_score,
                             s.renorm_eps, s.weight_scale, correction=self.correction, identity=s.identity)

    def _gate(self, gu):
        """The activation of experts with a gate matrix, from rows [gate | up]."""
        return ops.swiglu(gu) if self.spec.activation == "swiglu" else ops.glu_clamped(gu, self.spec.limit)

    def out_weight(self):
        return None if self.shared is None else self.shared.out_weight()

    def inner(self, x, step, out):
        """The shared expert's activation (if there is one) to `out`; the routed experts' rows are the result."""
        if self.shared is not None:
            self.shared.inner(x, step, out)
        return self._routed(x, step)

    def forward(self, x, step):
        y = self._routed(x, step)
        return y if self.shared is None else ops.BranchSum(self.shared.forward(x, step), y)

    def _routed(self, x, step):
        s, dt = self.spec, self.ctx.dtype
        ids, weights, *own = self._choose(x, step)
        own = (x, own[0]) if own else (None, None)
        first = None if self.gated else "gelu"
        if self._tensor_cores():
            _, pos_of, tile_expert, used = ops.moe_align(ids, s.num_experts, ops.MOE_TCGEN05_TILE, s.identity)
            rows = ops.moe_gather_rows(x, pos_of, tile_expert.numel() * ops.MOE_TCGEN05_TILE)
            act = ops.moe_gemm_tcgen05(rows, self.w_up, tile_expert, act=first, used_tiles=used)
            if self.gated:
                act = self._gate(act)
            return ops.PickedRows(ops.moe_gemm_tcgen05(act, self.w_down, tile_expert, used_tiles=used), pos_of, weights, *own)
        sorted_token, pos_of, tile_expert, _ = ops.moe_align(ids, s.num_experts, ops.moe_gemm_simt_tile(), s.identity)
        act = ops.moe_gemm_simt(x, sorted_token, self.w_up, tile_expert, dt, act=first)
        if self.gated:
            act = self._gate(act)
        y = ops.moe_gemm_simt(act, None, self.w_down, tile_expert, dt)
        return ops.PickedRows(y, pos_of, weights, *own)


register_feed_forward("routed_experts", RoutedExperts)
