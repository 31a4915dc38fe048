"""Grouped-query attention over the paged cache.

Order of operations as in the reference's layer (src/model/qwen_model.cu:113-160):
q, k, v projections; RMSNorm of each q and k head over its ``head_dim`` elements
(weight [head_dim] shared by the heads, before the rotation, :124-128); rotary
encoding of q and k at the tokens' absolute positions (:136); k and v into the
cache (:139-143); attention with scale 1/sqrt(head_dim) where q head h reads kv
head h // (num_heads/num_kv_heads) (src/kernels/attention.cu:44,304,458);
output projection.  The three projections are one product against the
concatenated matrix; norm, rotation and cache write are one kernel.

Unlike the reference, whose prefill attends only inside the portion it is given
(src/model/qwen_model.cu:147-151), every query attends the cache from position 0
(or the start of its window) to itself, so a prompt may be cut anywhere.

Parameters: hidden_size, num_heads, num_kv_heads, head_dim, qk_norm (bool),
qk_norm_eps, window (None = all keys, W = the last W keys including the query's
own), scale (None = 1/sqrt(head_dim)), has_kv (False: the layer has no k/v
projections and only ever reads another run's cache), cache_block_size (tokens per
cache page if this layer wants a page size of its own; None: the engine's).

Further parameters, for designs that differ from the above (defaults: as above):
    value_dim       size of a value head if it is not head_dim.  The cache and the kernels keep heads of
                    max(head_dim, value_dim) elements; the shorter kind is filled up with zero rows (of W_q, W_k
                    or W_v) and zero columns (of W_o) when the matrices are bound, so nothing else changes
    chunk           C: a query sees key j <= i only if floor(i / C) = floor(j / C), chunks counted from position 0
                    of the sequence (not together with ``window``)
    unit_norm_after_rotation   q and k are divided by their root mean square over head_dim (no weight, eps =
                    qk_norm_eps) behind the rotation instead of a weighted norm in front of it; the rotation may
                    cover only the head's first elements and be rescaled (``position``'s parameters)
    q_leaf, k_leaf, v_leaf, o_leaf   the tensors' leaves under the prefix
    bias_suffix     q, k and v have biases (the tensor's leaf + this suffix), added in 32-bit by the kernel that
                    finishes the heads
    softcap         c > 0: the scaled score s becomes c tanh(s / c)
    sink            True: one more entry in every softmax's denominator, of score 0 and without a value
    sink_leaf       the tensor [num_heads] of such an entry's score, a number a head (not scaled)
    qk_norm_over    "head" (default) or "all": with ``qk_norm`` one norm over all query heads together and one over all key
                    heads, weights [num_heads * head_dim] and [num_kv_heads * head_dim]
    value_is_key    True: there is no W_v; the values are the keys as projected (before norm and rotation)
    q_temp          (coef, every): q at position p is multiplied by 1 + coef ln(floor((p + 1) / every) + 1)
    gate_leaf       the tensor [num_heads, hidden] of one output gate a head: head h's output is multiplied by
                    sigmoid(W_g x)_h before the output projection; its rows are part of the first product
    q_norm_leaf, k_norm_leaf   the leaves of the per-head norms' weights (``qk_norm``)
A position part whose ``pairing`` is "interleaved" (element 2i turns with element 2i + 1) or that has no table of positions
is served by the same head-finishing kernel as the unit norm, which forms the angles itself from the frequencies.
"""
from __future__ import annotations

import math
from typing import List, Mapping

import torch

from ..cache.spec import PagedKVSpec
from ..ops import kernels as K
from ..weights.arena import FusedSpec, Piece
from ..weights.loader import WeightSpec
from .base import Part, register_part
from .linear import apply_linear, linear_into_residual, scaled_linear_into_residual


class GQAttention(Part):
    adds_into_residual = True        # forward(accumulate_into=...)
    folds_next_norm = True           # forward(then_norm=...)
    accepts_folded_norm = True       # its first operation is a product that can finish a folded norm
    scales_residual = True           # forward(residual_scale=...)

    def __init__(self, spec, rt, position=None):
        super().__init__(spec, rt)
        self.hidden = int(self.p("hidden_size"))
        self.nq = int(self.p("num_heads"))
        self.nkv = int(self.p("num_kv_heads"))
        self.d = int(self.p("head_dim"))
        self.qk_norm = bool(self.p("qk_norm", False))
        self.eps = float(self.p("qk_norm_eps", 1e-6))
        self.window = self.p("window", None)
        scale = self.p("scale", None)
        self.scale = 1.0 / math.sqrt(self.d) if scale is None else float(scale)
        self.has_kv = bool(self.p("has_kv", True))
        self.cache_block_size = self.p("cache_block_size", None)
        self.position = position
        self.dv = int(self.p("value_dim", self.d))
        self.dk = self.d                                  # true size of a query / key head
        self.d = max(self.dk, self.dv)                    # size of a head in the projection, the cache and the kernels
        self.chunk = self.p("chunk", None)
        self.unit_norm = bool(self.p("unit_norm_after_rotation", False))
        self.leaf = {k: self.p(k + "_leaf", k + "_proj.weight") for k in "qkvo"}
        self.bias_suffix = self.p("bias_suffix", None)
        self.softcap = float(self.p("softcap", 0.0) or 0.0)
        if self.softcap < 0:
            raise ValueError("softcap must be positive (or absent)")
        self.sink = bool(self.p("sink", False))
        self.sink_leaf = self.p("sink_leaf", None)
        self.sinks = None                                 # float32 [num_heads] once bound
        over = str(self.p("qk_norm_over", "head"))
        if over not in ("head", "all") or (over == "all" and not self.qk_norm):
            raise ValueError("qk_norm_over is 'head' or, with qk_norm, 'all'")
        self.norm_all = over == "all"
        self.value_is_key = bool(self.p("value_is_key", False))
        q_temp = self.p("q_temp", None)
        self.q_temp = None if q_temp is None else (float(q_temp[0]), int(q_temp[1]))
        self.gate_leaf = self.p("gate_leaf", None)
        # the gates' rows stand behind the heads in the first product, filled up so that its rows stay 16-byte aligned
        self.gate_rows = 0 if self.gate_leaf is None else -(-self.nq // 8) * 8
        self.norm_leaf = {k: self.p(f"{k}_norm_leaf", f"{k}_norm.weight") for k in "qk"}
        if self.q_temp is not None and self.q_temp[1] <= 0:
            raise ValueError("q_temp: 'every' must be positive")
        if self.value_is_key and (self.dk != self.dv or not self.has_kv):
            raise ValueError("value_is_key needs keys of its own, of the values' size")
        interleaved = getattr(position, "pairing", "half") == "interleaved"
        no_table = position is not None and hasattr(position, "frequencies") and getattr(position, "max_positions", 1) == 0
        # the kernel that forms the angles from the frequencies also adds biases, takes either pairing, a temperature, ...
        self.by_frequencies = self.unit_norm or interleaved or self.bias_suffix is not None or no_table \
            or self.q_temp is not None or self.value_is_key or (self.qk_norm and self.dk != self.d) or self.norm_all
        if self.by_frequencies and position is not None and not hasattr(position, "frequencies"):
            raise ValueError("this attention needs a position encoding that gives its frequencies")
        self.interleaved = interleaved
        self.bias = None
        if self.chunk is not None and (self.window is not None or int(self.chunk) <= 0):
            raise ValueError("chunk must be positive and excludes window")
        if self.unit_norm and self.qk_norm:
            raise ValueError("qk_norm (in front of the rotation) and unit_norm_after_rotation exclude each other")
        if self.unit_norm and position is not None and not hasattr(position, "frequencies"):
            raise ValueError("unit_norm_after_rotation needs a position encoding that gives its frequencies")
        if self.nq % self.nkv:
            raise ValueError(f"num_heads {self.nq} is not a multiple of num_kv_heads {self.nkv}")
        if self.d > 256:
            raise ValueError(f"head_dim {self.d} > 256 is not supported by the attention kernels")
        if self.window is not None and int(self.window) <= 0:
            raise ValueError("window must be positive")
        self.w_qkv = self.w_o = self.q_norm_w = self.k_norm_w = None

    # -- cache ------------------------------------------------------------------
    def cache_spec(self):
        return PagedKVSpec(self.nkv, self.d, None if self.window is None else int(self.window),
                           None if self.cache_block_size is None else int(self.cache_block_size))

    # -- weights ------------------------------------------------------------------
    def weight_specs(self) -> List[WeightSpec]:
        L = self.leaf
        out = [WeightSpec(self.name(L["q"]), (self.nq * self.dk, self.hidden))]
        if self.has_kv:
            out += [WeightSpec(self.name(L["k"]), (self.nkv * self.dk, self.hidden)),
                    *([] if self.value_is_key else [WeightSpec(self.name(L["v"]), (self.nkv * self.dv, self.hidden))])]
        out.append(WeightSpec(self.name(L["o"]), (self.hidden, self.nq * self.dv)))
        if self.gate_leaf is not None:
            out.append(WeightSpec(self.name(self.gate_leaf), (self.nq, self.hidden)))
        if self.bias_suffix is not None:
            sfx = self.bias_suffix
            out.append(WeightSpec(self.name(L["q"]) + sfx, (self.nq * self.dk,), init="zeros", as_float32=True))
            if self.has_kv:
                out += [WeightSpec(self.name(L["k"]) + sfx, (self.nkv * self.dk,), init="zeros", as_float32=True),
                        *([] if self.value_is_key else
                          [WeightSpec(self.name(L["v"]) + sfx, (self.nkv * self.dv,), init="zeros", as_float32=True)])]
        if self.qk_norm:
            for kind in ("q", "k") if self.has_kv else ("q",):
                heads = (self.nq if kind == "q" else self.nkv) if self.norm_all else 1
                out.append(WeightSpec(self.name(self.norm_leaf[kind]), (heads * self.dk,), init="norm", as_float32=True))
        if self.sink_leaf is not None:
            out.append(WeightSpec(self.name(self.sink_leaf), (self.nq,), init="zeros", as_float32=True))
        return out

    def fused_layout(self, dtype_of) -> List[FusedSpec]:
        """q, k, v (unless the values are the keys) and the heads' gates stacked into one matrix, the projections' rows in
        this order."""
        if not self.has_kv or self.dk != self.dv or self.gate_rows not in (0, self.nq):
            return []                                   # what is filled up is put together when bound
        sources = [(self.leaf["q"], self.nq * self.d), (self.leaf["k"], self.nkv * self.d)]
        if not self.value_is_key:
            sources.append((self.leaf["v"], self.nkv * self.d))
        if self.gate_leaf is not None:
            sources.append((self.gate_leaf, self.nq))
        pieces, at = [], 0
        for leaf, rows in sources:
            pieces.append(Piece(self.name(leaf), at))
            at += rows
        return [FusedSpec(self.name("qkv_proj.weight"), (at, self.hidden), tuple(pieces))]

    def _filled(self, m: torch.Tensor, heads: int, size: int) -> torch.Tensor:
        """Rows of `heads` heads of `size` rows each, every head filled up to self.d rows with zeros."""
        if size == self.d:
            return m
        out = torch.zeros((heads, self.d, m.shape[1]), dtype=m.dtype, device=m.device)
        out[:, :size] = m.view(heads, size, m.shape[1])
        return out.view(heads * self.d, m.shape[1])

    def bind(self, tensors: Mapping[str, torch.Tensor]) -> None:
        fused = self.name("qkv_proj.weight")
        if fused in tensors:
            self.w_qkv = self._matrix(tensors[fused])
        else:
            mats = [self._filled(self._matrix(tensors[self.name(self.leaf["q"])]), self.nq, self.dk)]
            if self.has_kv:
                mats.append(self._filled(self._matrix(tensors[self.name(self.leaf["k"])]), self.nkv, self.dk))
                if not self.value_is_key:
                    mats.append(self._filled(self._matrix(tensors[self.name(self.leaf["v"])]), self.nkv, self.dv))
            if self.gate_leaf is not None:
                g = self._matrix(tensors[self.name(self.gate_leaf)])
                mats.append(torch.cat([g, torch.zeros((self.gate_rows - self.nq, self.hidden), dtype=g.dtype, device=g.device)]))
            if len({m.dtype for m in mats}) != 1:
                mats = [m.to(torch.float32) for m in mats]
            self.w_qkv = torch.cat(mats, dim=0).contiguous() if len(mats) > 1 else mats[0].contiguous()
        self.w_o = self._matrix(tensors[self.name(self.leaf["o"])])
        if self.dv != self.d:          # zero columns where the kernels' value heads are longer than the true ones
            wo = torch.zeros((self.hidden, self.nq, self.d), dtype=self.w_o.dtype, device=self.w_o.device)
            wo[:, :, : self.dv] = self.w_o.view(self.hidden, self.nq, self.dv)
            self.w_o = wo.view(self.hidden, self.nq * self.d).contiguous()
        if self.bias_suffix is not None:       # one row in the projection's layout, heads filled up with zeros
            sfx = self.bias_suffix
            parts = [(self.leaf["q"], self.nq, self.dk)]
            if self.has_kv:
                parts.append((self.leaf["k"], self.nkv, self.dk))
                if not self.value_is_key:
                    parts.append((self.leaf["v"], self.nkv, self.dv))
            rows = []
            for leaf, heads, size in parts:
                b = self._vector32(tensors[self.name(leaf) + sfx]).view(heads, size)
                full = torch.zeros((heads, self.d), dtype=torch.float32, device=b.device)
                full[:, :size] = b
                rows.append(full.view(-1))
            self.bias = torch.cat(rows).contiguous()
        if self.sink_leaf is not None:
            self.sinks = self._vector32(tensors[self.name(self.sink_leaf)])
        elif self.sink:
            self.sinks = torch.zeros((self.nq,), dtype=torch.float32, device=self.w_o.device)
        if self.qk_norm:
            self.q_norm_w = self._norm_row(tensors, "q")
            if self.has_kv:
                self.k_norm_w = self._norm_row(tensors, "k")

    def _norm_row(self, tensors, kind: str) -> torch.Tensor:
        w = self._vector32(tensors[self.name(self.norm_leaf[kind])])
        if self.dk == self.d:
            return w
        w = w.view(-1, self.dk)                                                   # one head's weights, or every head's
        full = torch.zeros((w.shape[0], self.d), dtype=torch.float32, device=w.device)      # heads filled up with zeros
        full[:, : self.dk] = w
        return full.view(-1)

    # -- run ------------------------------------------------------------------
    def _mask(self) -> int:
        """The kernels' one mask argument: W > 0 a window of W keys, -C < 0 chunks of C positions, 0 every key."""
        if self.chunk is not None:
            return -int(self.chunk)
        return 0 if self.window is None else int(self.window)

    def forward(self, x, ctx, slot: int, write_cache: bool, accumulate_into=None, then_norm=None,
                residual_scale: float = 1.0):
        T = x.shape[0]
        ws = ctx.workspace
        if write_cache and not self.has_kv:
            raise RuntimeError(f"{self.prefix}: a layer without k/v projections cannot write a cache")
        nkv_w = self.nkv if write_cache else 0
        width = (self.nq + (1 if self.value_is_key else 2) * nkv_w) * self.d
        gate = None
        if write_cache or not self.has_kv:
            w = self.w_qkv
            gate_col, width = width, width + self.gate_rows
        else:                                    # a run that only reads a cache: the queries' rows, and the gates' by themselves
            w = self.w_qkv[: self.nq * self.d]
            if self.gate_leaf is not None:
                gm = ws.get("attn.gate", (T, self.gate_rows), ctx.dtype)
                apply_linear(x, self.w_qkv[self.w_qkv.shape[0] - self.gate_rows:], gm, ctx, "attn.gate")
                gate = (gm, 0)
        qkv = ws.get("attn.qkv", (T, width), ctx.dtype)
        apply_linear(x, w, qkv, ctx, "attn.qkv")
        if self.gate_leaf is not None and gate is None:
            gate = (qkv, gate_col)
        pages, table = ctx.kv(slot)
        rot = self.position.rotary_table() if self.position is not None and not self.by_frequencies else None
        cos_sin, rotary_dim = rot if rot is not None else (None, 0)
        att = ws.get("attn.out", (T, self.nq * self.d), ctx.dtype)
        turns = self.position is not None and hasattr(self.position, "frequencies")
        if write_cache and self.chunk is None and not self.softcap and self.dk == self.d and not self.unit_norm \
                and self.bias is None and not self.norm_all and not (self.by_frequencies and turns) and (self.qk_norm or self.q_temp is None) \
                and K.decode_finishes_heads(ctx, ctx.dtype, self.nq, self.nkv, self.d, rotary_dim):
            # a step of single tokens: the attention kernel finishes the heads itself
            K.attn_decode_heads(qkv, pages, table, ctx, att, self.nq, self.nkv, self.d, self.scale,
                                0 if self.window is None else int(self.window), self.q_norm_w,
                                self.k_norm_w, self.eps, cos_sin, sink=self.sinks, q_temp=self.q_temp,
                                value_is_key=self.value_is_key)
        elif self.by_frequencies:
            freq, mag = (self.position.frequencies(), self.position.magnitude) if turns else (None, 1.0)
            bias = self.bias if (self.bias is None or write_cache or not self.has_kv) else self.bias[: self.nq * self.d]
            K.head_finish(qkv, self.nq, nkv_w, self.d, self.dk, self.eps, freq, mag, ctx,
                          table if write_cache else None, pages if write_cache else None,
                          interleaved=self.interleaved, normalize=self.unit_norm, bias=bias, q_norm_w=self.q_norm_w,
                          k_norm_w=self.k_norm_w if write_cache else None, q_temp=self.q_temp,
                          value_is_key=self.value_is_key, norm_all=self.norm_all)
            self._attend(qkv, width, pages, table, ctx, att)
        else:
            K.qk_norm_rope_store(qkv, self.nq, nkv_w, self.d, self.q_norm_w,
                                 self.k_norm_w if write_cache else None, self.eps, cos_sin, rotary_dim,
                                 ctx.positions, ctx.token_seq, table if write_cache else None,
                                 pages if write_cache else None, ctx.status)
            self._attend(qkv, width, pages, table, ctx, att)
        if gate is not None:
            gated = ws.get("attn.gated", (T, self.nq * self.d), ctx.dtype)
            K.head_gate(att, gate, gated, self.nq, self.d, self.d, per_head=True)
            att = gated
        if residual_scale != 1.0:
            return scaled_linear_into_residual(att, self.w_o, accumulate_into, residual_scale, ctx, "attn.proj")
        return linear_into_residual(att, self.w_o, accumulate_into, ctx, "attn.proj", then_norm)

    def _attend(self, qkv, width, pages, table, ctx, att) -> None:
        K.paged_attention(qkv, width, pages, table, ctx, att, self.nq, self.nkv, self.d, self.scale,
                          self._mask(), softcap=self.softcap, sink=self.sinks)


register_part("mixer", "gqa_attention", GQAttention)
