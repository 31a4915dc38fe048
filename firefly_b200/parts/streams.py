"""Hyper-connections: the residual is several streams side by side, and every part reads and writes all of them.

With S streams x_1 .. x_S, all equal to the embedding output at the start, a part (a mixer or a feed-forward) runs as

    u = sum_s in[s] x_s;   y = part(norm(u));   x_t <- sum_s mix[s, t] x_s + out[t] y     (all from the old streams)

and the model ends with norm(sum_s x_s).  The streams are 32-bit, [T, S, W].

``hyper_connections`` is the arrangement of a layer in this form (two parts, or a mixer only).  A part's output is not
written into the streams at once: it is handed on as a ``StreamWrite``, and the seam in front of the next part (the next
block's, or the model's end) does the write, the next read and the norm in one pass over a token's rows
(``csrc/stream_seam.cu``).  A feed-forward of routed experts hands on its experts' rows with their weights
(``RoutedRows``), whose sum the same pass forms.  As long as nothing has been written, the streams are the embedding
output itself, [T, W], and are never spread out.

``stream_sum`` is the norm part at the model's end: the last write, the sum over the streams and the norm it wraps, for
the rows whose logits are asked for.
"""
from __future__ import annotations

from typing import List, Mapping, Optional

import torch

from ..config.base import ConfigError
from ..ops import kernels as K
from ..weights.loader import WeightSpec
from .base import Part, Runtime, build_part, declared, register_part
from .block import Block
from .moe import RoutedRows
from .norm import LayerNorm, RMSNorm


class Connection:
    """One part's tie to the streams: the tensors ``<prefix>.in`` [S], ``.out`` [S] and ``.mix`` [S, S] (from, to)."""

    def __init__(self, prefix: str, streams: int):
        self.prefix, self.streams = prefix, int(streams)
        if not (0 < self.streams <= 32):
            raise ConfigError(f"{prefix}: {streams} streams; 1 to 32 are supported")
        self.w_in = self.w_out = self.mix = None

    def weight_specs(self) -> List[WeightSpec]:
        S, p = self.streams, self.prefix
        return [WeightSpec(p + ".in", (S,), init="norm", as_float32=True), WeightSpec(p + ".out", (S,), init="norm", as_float32=True),
                WeightSpec(p + ".mix", (S, S), as_float32=True)]

    def bind(self, tensors: Mapping[str, torch.Tensor]) -> None:
        self.w_in, self.w_out, self.mix = (Part._vector32(tensors[self.prefix + leaf]) for leaf in (".in", ".out", ".mix"))


class StreamWrite:
    """A part's output that has not been written into the streams yet."""

    def __init__(self, y, connection: Connection):
        self.y, self.connection = y, connection


def _norm_args(norm) -> dict:
    return dict(w=norm.weight, b=getattr(norm, "bias", None), eps=norm.eps, center=isinstance(norm, LayerNorm))


def seam(streams: torch.Tensor, pending: Optional[StreamWrite], ctx, *, count: int, w_in=None, norm=None, row_idx=None,
         tag: str = "normed", out_dtype=None, keep: bool = True):
    """The pending write, the read with ``w_in`` (None: the plain sum) and the norm (None: none) of ``count`` streams;
    returns (rows, streams).  ``keep`` False: the written streams are not wanted."""
    T, W = streams.shape[0], streams.shape[-1]
    rows = T if row_idx is None else row_idx.numel()
    out = ctx.workspace.get(tag, (rows, W), out_dtype or ctx.dtype)
    kw = _norm_args(norm) if norm is not None else {}
    if pending is not None:
        c = pending.connection
        kw.update(mix=c.mix, out_w=c.w_out)
        if isinstance(pending.y, RoutedRows):
            kw["routed"] = pending.y.rows, pending.y.row_of, pending.y.wts, pending.y.shared
        else:
            kw["y"] = pending.y
        if keep:
            # in place, unless the streams are still the embedding output
            kw["dst"] = streams if streams.dim() == 3 else ctx.workspace.get("streams", (T, count, W), torch.float32)
    K.stream_seam(streams, out, streams=count, in_w=w_in, row_idx=row_idx, **kw)
    return out, kw.get("dst", streams)


def stream_sum(streams: torch.Tensor, pending: Optional[StreamWrite], ctx, count: int) -> torch.Tensor:
    """The sum of the streams behind the pending write, float32 [T, W]; nothing is changed."""
    return seam(streams, pending, ctx, count=count, tag="streams.sum", out_dtype=torch.float32, keep=False)[0]


class HyperConnectionBlock(Block):
    """A layer whose parts are tied to several streams.  ``params``: ``streams``, and ``connections``, one tensor prefix
    for each part.  The norms are layer norms or RMS norms."""

    def __init__(self, layer_spec, rt: Runtime):
        super().__init__(layer_spec, rt)
        self.streams = int(self.params["streams"])
        prefixes = tuple(self.params["connections"])
        if len(prefixes) != len(self.norms):
            raise ValueError(f"arrangement '{layer_spec.arrangement}' needs {len(self.norms)} connections, got {len(prefixes)}")
        if self.input_filter is not None or not all(isinstance(n, (LayerNorm, RMSNorm)) for n in self.norms):
            raise ValueError(f"arrangement '{layer_spec.arrangement}' takes layer norms or RMS norms and no input filter")
        self.connections = [Connection(p, self.streams) for p in prefixes]
        self._ffn_rows = self.feed_forward is not None and declared(self.feed_forward, "hands_on_rows")

    def weight_specs(self) -> List[WeightSpec]:
        return super().weight_specs() + [w for c in self.connections for w in c.weight_specs()]

    def bind(self, tensors: Mapping[str, torch.Tensor]) -> None:
        super().bind(tensors)
        for c in self.connections:
            c.bind(tensors)

    def _read(self, k: int, streams, pending, ctx):
        if pending is not None and not isinstance(pending, StreamWrite):
            raise RuntimeError("hyper_connections: the layer in front is of another arrangement")
        return seam(streams, pending, ctx, count=self.streams, w_in=self.connections[k].w_in, norm=self.norms[k])

    def forward(self, residual: torch.Tensor, pending, ctx, slot: int, write_cache: bool):
        x, X = self._read(0, residual, pending, ctx)
        pending = StreamWrite(self.mixer.forward(x, ctx, slot, write_cache), self.connections[0])
        if self.feed_forward is not None:
            x, X = self._read(1, X, pending, ctx)
            y = self.feed_forward.forward(x, ctx, **({"as_rows": True} if self._ffn_rows else {}))
            pending = StreamWrite(y, self.connections[1])
        return X, pending


class StreamSumNorm(Part):
    """norm(sum of the streams).  Parameters: streams, norm (the PartSpec of a layer norm or RMS norm)."""

    def __init__(self, spec, rt):
        super().__init__(spec, rt)
        self.streams = int(self.p("streams"))
        self.norm = build_part("norm", self.p("norm"), rt)
        if not isinstance(self.norm, (LayerNorm, RMSNorm)):
            raise ValueError("stream_sum wraps a layer norm or an RMS norm")

    def parts(self) -> list:
        return [self.norm]

    def weight_specs(self) -> List[WeightSpec]:
        return self.norm.weight_specs()

    def bind(self, tensors: Mapping[str, torch.Tensor]) -> None:
        self.norm.bind(tensors)

    def forward(self, residual: torch.Tensor, delta, ctx, *, tag: str = "normed", row_idx: Optional[torch.Tensor] = None):
        return seam(residual, delta, ctx, count=self.streams, norm=self.norm, row_idx=row_idx, tag=tag, keep=False)[0]


register_part("arrangement", "hyper_connections", HyperConnectionBlock)
register_part("norm", "stream_sum", StreamSumNorm)
