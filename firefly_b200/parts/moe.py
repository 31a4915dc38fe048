"""Routed experts with group-limited choice and a shared expert.

    z = W_router x (32-bit);  s = softmax(z) over all experts
    experts form `groups` equal groups of neighbours; a group's score is its largest s; only experts
    of the `keep` best groups may be chosen; of those, the `top` with the largest s are
    weights = chosen s / (their sum + 1e-20)
    expert(x) = W_down (g * sigmoid(1.702 g) * (u + 1)),  g = min(W_gate x, limit),  u = clamp(W_up x, -limit, limit)
    out = sum of weight * expert(x) over the chosen experts  (+ shared expert(x), with sizes and limit of its own)

All of it stays on the device (``csrc/moe.cu``): the router's choice, a plan that sorts the step's
(token, choice) pairs by expert, two grouped products over the experts' stacked matrices (the first with
the activation in its epilogue; bfloat16 on tensor cores) and one kernel that forms the weighted sum, adds the shared expert and
adds the whole, times the block's multiplier, into the 32-bit residual.  No count is read by the host,
so steps with routed experts are captured into CUDA graphs like any other.

Parameters (``shared_limit`` and ``limit`` where the form has them): hidden_size, experts, top, groups, keep, ff, limit, shared_ff (0: no shared expert),
shared_limit.  Tensors: router [experts, W]; e<i>.gate, e<i>.up [ff, W]; e<i>.down [W, ff];
shared.gate, shared.up [shared_ff, W]; shared.down [W, shared_ff].

What the lines above fix can be chosen by further parameters (the defaults are the above):
    score          "softmax" | "sigmoid": s = sigmoid(z), each expert by itself
                   | "chosen_softmax": the choice is by z itself and the weights are the softmax over the chosen z alone
    router_bias    the leaf of a tensor [experts] added to z (None: none)
    correction     True: a tensor ``correction`` [experts] is added to s for the choice (of groups and of experts);
                   the weights stay the plain s
    group_score    "best" | "two_best": a group's score is the sum of its two largest choice scores
    renormalize    False: the weights are the chosen s as they are
    activation     "clamped_swish" | "silu": expert(x) = W_down (silu(W_gate x) * (W_up x)), no clamps, no limit
                   | "relu2": expert(x) = W_down relu(W_up x)^2, no gate matrices at all (the shared expert likewise)
    weight_on_input  True: a choice's weight multiplies the expert's input: out = sum of expert(weight * x).  The first
                   product is linear in the input, so the weight goes onto its 32-bit result, in front of the activation
    shared_gate    True: the shared expert's output is multiplied by sigmoid(w x), w the tensor ``shared.sg`` [1, W]; its
                   logit is one more row of the router's product
Experts outside the open groups count as minus infinity in the choice (choice scores may be negative).
"""
from __future__ import annotations

from typing import List, Mapping

import torch

from ..ops import kernels as K
from ..weights.arena import FusedSpec, Piece
from ..weights.loader import WeightSpec
from .base import Part, register_part
from .linear import apply_linear, linear_relu2


class RoutedRows:
    """A step's routed output that has not been summed: token t's is sum_k wts[t, k] rows[row_of[t, k]] + shared[t]."""

    def __init__(self, rows: torch.Tensor, row_of: torch.Tensor, wts: torch.Tensor, shared):
        self.rows, self.row_of, self.wts, self.shared = rows, row_of, wts, shared


class GroupedExperts(Part):
    adds_into_residual = True        # forward(accumulate_into=...)
    hands_on_rows = True             # forward(as_rows=...)
    scales_residual = True           # forward(residual_scale=...)

    def __init__(self, spec, rt):
        super().__init__(spec, rt)
        self.hidden = int(self.p("hidden_size"))
        self.E = int(self.p("experts"))
        self.top = int(self.p("top"))
        self.groups = int(self.p("groups", 1))
        self.keep = int(self.p("keep", self.groups))
        self.ff = int(self.p("ff"))
        act = str(self.p("activation", "clamped_swish"))
        self.gated = act != "relu2"
        self.activation = {"clamped_swish": K.GLU_CLAMPED_SWISH, "silu": K.GLU_SILU, "relu2": 0}[act]
        self.limit = float(self.p("limit", 0.0 if act != "clamped_swish" else ...))
        self.weight_on_input = bool(self.p("weight_on_input", False))
        self.shared_gate = bool(self.p("shared_gate", False))
        self.score = {"softmax": K.ROUTE_SOFTMAX, "sigmoid": K.ROUTE_SIGMOID, "chosen_softmax": K.ROUTE_CHOSEN_SOFTMAX}[str(self.p("score", "softmax"))]
        self.group_score = {"best": K.GROUP_BY_BEST, "two_best": K.GROUP_BY_TWO_BEST}[str(self.p("group_score", "best"))]
        self.renormalize = bool(self.p("renormalize", True))
        self.has_correction = bool(self.p("correction", False))
        self.correction = None
        self.router_bias_leaf = self.p("router_bias", None)
        self.router_bias = None
        self.shared_ff = int(self.p("shared_ff", 0))
        self.shared_limit = float(self.p("shared_limit", self.limit))
        if self.E % self.groups or not (0 < self.keep <= self.groups) or not (0 < self.top <= self.keep * (self.E // self.groups)):
            raise ValueError(f"{self.prefix}: {self.top} of {self.E} experts in {self.keep} of {self.groups} groups cannot be chosen")
        if self.shared_gate and not self.shared_ff:
            raise ValueError(f"{self.prefix}: a gate for a shared expert that is not there")
        if self.shared_ff and self.gated and self.activation != K.GLU_CLAMPED_SWISH:
            raise ValueError(f"{self.prefix}: a shared expert is of the clamped or of the ungated form")
        self.router = self.w_gate = self.w_up = self.w_down = self.w_sh_gu = self.w_sh_down = None

    def weight_specs(self) -> List[WeightSpec]:
        n, W = self.name, self.hidden
        out = [WeightSpec(n("router"), (self.E, W))]
        if self.router_bias_leaf is not None:
            out.append(WeightSpec(n(self.router_bias_leaf), (self.E,), init="zeros", as_float32=True))
        if self.has_correction:
            out.append(WeightSpec(n("correction"), (self.E,), init="zeros", as_float32=True))
        for e in range(self.E):
            if self.gated:
                out.append(WeightSpec(n(f"e{e}.gate"), (self.ff, W)))
            out += [WeightSpec(n(f"e{e}.up"), (self.ff, W)), WeightSpec(n(f"e{e}.down"), (W, self.ff))]
        if self.shared_ff:
            if self.gated:
                out.append(WeightSpec(n("shared.gate"), (self.shared_ff, W)))
            out += [WeightSpec(n("shared.up"), (self.shared_ff, W)), WeightSpec(n("shared.down"), (W, self.shared_ff))]
            if self.shared_gate:
                out.append(WeightSpec(n("shared.sg"), (1, W)))
        return out

    def fused_layout(self, dtype_of) -> List[FusedSpec]:
        """The experts' matrices stacked, [experts * rows, columns] each kind; the shared expert's gate over up; the shared
        gate's row under the router's."""
        n, W = self.name, self.hidden
        out = []
        if self.gated:
            out.append(FusedSpec(n("experts.gate"), (self.E * self.ff, W), tuple(Piece(n(f"e{e}.gate"), e * self.ff) for e in range(self.E))))
        if self.shared_gate:
            out.append(FusedSpec(n("router_sg"), (self.E + 1, W), (Piece(n("router"), 0), Piece(n("shared.sg"), self.E))))
        out += [FusedSpec(n("experts.up"), (self.E * self.ff, W), tuple(Piece(n(f"e{e}.up"), e * self.ff) for e in range(self.E))),
               FusedSpec(n("experts.down"), (self.E * W, self.ff), tuple(Piece(n(f"e{e}.down"), e * W) for e in range(self.E)))]
        if self.shared_ff and self.gated:
            out.append(FusedSpec(n("shared.gate_up"), (2 * self.shared_ff, W),
                                 (Piece(n("shared.gate"), 0), Piece(n("shared.up"), self.shared_ff))))
        return out

    def _stacked(self, tensors, fused: str, leaves: List[str]) -> torch.Tensor:
        if self.name(fused) in tensors:
            return self._matrix(tensors[self.name(fused)])
        mats = [self._matrix(tensors[self.name(leaf)]) for leaf in leaves]
        if len({m.dtype for m in mats}) != 1:
            mats = [m.to(torch.float32) for m in mats]
        return torch.cat(mats, dim=0).contiguous()

    def bind(self, tensors: Mapping[str, torch.Tensor]) -> None:
        E, W = self.E, self.hidden
        self.router = self._stacked(tensors, "router_sg", ["router", "shared.sg"]) if self.shared_gate \
            else self._matrix(tensors[self.name("router")])
        if self.router_bias_leaf is not None:
            self.router_bias = self._vector32(tensors[self.name(self.router_bias_leaf)])
        if self.has_correction:
            self.correction = self._vector32(tensors[self.name("correction")])
        if self.gated:
            self.w_gate = self._stacked(tensors, "experts.gate", [f"e{e}.gate" for e in range(E)]).view(E, self.ff, W)
        self.w_up = self._stacked(tensors, "experts.up", [f"e{e}.up" for e in range(E)]).view(E, self.ff, W)
        self.w_down = self._stacked(tensors, "experts.down", [f"e{e}.down" for e in range(E)]).view(E, W, self.ff)
        if len({m.dtype for m in (self.w_gate, self.w_up, self.w_down) if m is not None}) != 1:
            self.w_gate, self.w_up, self.w_down = (m.to(torch.float32) if m is not None else None
                                                   for m in (self.w_gate, self.w_up, self.w_down))
        if self.shared_ff:
            self.w_sh_gu = self._stacked(tensors, "shared.gate_up", ["shared.gate", "shared.up"]) if self.gated \
                else self._matrix(tensors[self.name("shared.up")])
            self.w_sh_down = self._matrix(tensors[self.name("shared.down")])

    def forward(self, x, ctx, accumulate_into=None, residual_scale: float = 1.0, as_rows: bool = False):
        T, ws, W, top = x.shape[0], ctx.workspace, self.hidden, self.top
        dt = self.w_up.dtype
        if x.dtype != dt:
            raise K.KernelError(f"{self.prefix}: activations {x.dtype} against expert matrices {dt}")
        # the router: logits, scores and the choice in 32-bit
        z = ws.get("moe.z", (T, self.E + (1 if self.shared_gate else 0)), torch.float32)
        apply_linear(x, self.router, z, ctx, "moe.z")
        ids = ws.get("moe.ids", (T, top), torch.int32)
        wts = ws.get("moe.wts", (T, top), torch.float32)
        K.moe_route(z[:, : self.E], ids, wts, self.groups, self.keep, score=self.score, correction=self.correction,
                    group_score=self.group_score, renormalize=self.renormalize, bias=self.router_bias)
        rows = T * top
        tc = K.moe_on_tensor_cores(dt, (W, self.ff))       # which grouped kernel runs: the plan's row tile is its
        max_tiles = K.moe_max_tiles(rows, self.E, tc)
        seg = ws.get("moe.seg", (self.E + 1,), torch.int32)
        row_of = ws.get("moe.row_of", (rows,), torch.int32)
        src_tok = ws.get("moe.src_tok", (rows,), torch.int32)
        tile_e = ws.get("moe.tile_e", (max_tiles,), torch.int32)
        tile_r = ws.get("moe.tile_r", (max_tiles,), torch.int32)
        n_tiles = ws.get("moe.n_tiles", (1,), torch.int32)
        row_w = ws.get("moe.row_w", (rows,), torch.float32) if self.weight_on_input else None
        K.moe_plan(ids, self.E, seg, row_of, src_tok, tile_e, tile_r, n_tiles, tc, wts if self.weight_on_input else None, row_w)
        plan = (seg, tile_e, tile_r, n_tiles, max_tiles)
        act = ws.get("moe.act", (rows, self.ff), dt)
        if self.gated:
            K.moe_grouped(x, src_tok, self.w_gate, self.w_up, plan, act, self.limit, tc, self.activation, row_w=row_w, status=ctx.status)
        else:
            K.moe_grouped(x, src_tok, self.w_up, None, plan, act, 0.0, tc, kind=K.MOE_UP, row_w=row_w, status=ctx.status)
        outs = ws.get("moe.rows", (rows, W), torch.float32)
        K.moe_grouped(act, src_tok, self.w_down, None, plan, outs, 0.0, tc, status=ctx.status)
        shared = None
        if self.shared_ff:
            sact = ws.get("moe.sh_act", (T, self.shared_ff), dt)
            if self.gated:
                gu = ws.get("moe.sh_gu", (T, 2 * self.shared_ff), dt)
                apply_linear(x, self.w_sh_gu, gu, ctx, "moe.sh_gu")
                K.clamped_glu(gu, sact, self.shared_limit)
            else:
                linear_relu2(x, self.w_sh_gu, sact, ctx, "moe.sh_up")
            shared = ws.get("moe.sh_out", (T, W), torch.float32)
            apply_linear(sact, self.w_sh_down, shared, ctx, "moe.sh_out")
        if as_rows and accumulate_into is None and not self.weight_on_input and not self.shared_gate:
            return RoutedRows(outs, row_of, wts, shared)
        into = accumulate_into if accumulate_into is not None else ws.get("moe.delta", (T, W), torch.float32)
        K.moe_combine(into, outs, row_of, None if self.weight_on_input else wts, shared, residual_scale if accumulate_into is not None else 1.0,
                      top=top, shared_z=z[:, self.E] if self.shared_gate else None, overwrite=accumulate_into is None)
        return None if accumulate_into is not None else into


register_part("feed_forward", "grouped_experts", GroupedExperts)
