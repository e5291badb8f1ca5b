"""Several residual streams instead of one."""
from __future__ import annotations

from typing import Dict, Optional

import torch

from .. import kernels
from ..weights.spec import ParamSpec
from .base import BLOCKS, Block, FeedForward, Mixer, Norm, Part
from .block import UnusedTensors, _leaves


class HyperConnection(Part):
    """How a sub-layer is connected to ``streams`` residual streams: it reads sum_s in[s] x_s, and its result y makes
    x_t <- sum_s mix[s, t] x_s + out[t] y  (all streams at once from the old ones; mix is indexed [from, to]).
    The three tensors are kept in 32-bit."""

    def __init__(self, streams: int):
        self.streams = int(streams)
        self.in_ = self.out = self.mix = None

    def param_specs(self) -> Dict[str, ParamSpec]:
        S = self.streams
        return {"in": ParamSpec((S,), kind="vector", mean=1.0 / S, std=0.2 / S),
                "out": ParamSpec((S,), kind="vector", mean=1.0, std=0.3),
                "mix": ParamSpec((S, S), kind="vector", mean=1.0 / S, std=0.3 / S)}

    def bind(self, params, compute_dtype):
        self.in_, self.out, self.mix = (params[n].to(torch.float32).contiguous() for n in ("in", "out", "mix"))

    def cuda_modules(self, compute_dtype):
        return ["streams"]


class StreamsNorm(Norm):
    """A norm over a sum of the streams: norm(sum_s in[s] x_s) with a connection, norm(sum_s x_s) without.  Its tensors are the
    inner norm's (a connection's belong to the block).  Whoever updates the streams last computes it in the same pass and leaves
    the result in ``stream.prepared``; else one kernel collects and norms."""

    def __init__(self, norm: Norm, streams: int, connection: Optional[HyperConnection] = None):
        if norm.deferred_params.__func__ is Norm.deferred_params:
            raise ValueError("streams: the kernel that collects them applies RMS norms only")
        self.norm, self.streams, self.connection = norm, int(streams), connection
        self.compute_dtype = None

    def param_specs(self):
        return self.norm.param_specs()

    def bind(self, params, compute_dtype):
        self.norm.bind(params, compute_dtype)

    def cuda_modules(self, compute_dtype):
        return ["streams"]

    def coefficients(self):
        """(in, (weight, eps)) for the kernel."""
        return (None if self.connection is None else self.connection.in_), self.norm.deferred_params()

    def forward(self, ctx, stream, rows=None, deferred_ok=False):
        prepared, stream.prepared = stream.prepared, None
        if prepared is not None and prepared[0] is self and rows is None:
            return prepared[1]
        in_, norm = self.coefficients()
        return kernels.streams_update(stream.h, self.streams, ctx.compute_dtype, in_=in_, next_norm=norm, rows=rows)[1]


@BLOCKS.register("hyper_connected")
class HyperConnectedBlock(Block):
    """A pre-norm block on ``streams`` residual streams x_1 .. x_S (``stream.h`` [T, S, W], or [T, 1, W] while all are equal):
    for each of its two sub-layers, y = sublayer(norm(sum_s in[s] x_s)), then x_t <- sum_s mix[s, t] x_s + out[t] y.
    ``ffn`` (with ``norm2``) may be None: the block is then its first half.

    Sub-layers hand out their results in 32-bit (``output``: a tensor or a stack of partial sums); one kernel per sub-layer forms
    the new streams and, where the next reader is a sub-layer of such a block, that sub-layer's normed input in the same pass."""

    def __init__(self, streams: int, norm1: Norm, mixer: Mixer, norm2: Norm = None, ffn: FeedForward = None,
                 names: Dict[str, str] = None):
        if (ffn is None) != (norm2 is None):
            raise ValueError("hyper_connected block: ffn and norm2 come together or not at all")
        self.streams = int(streams)
        self.norm1, self.mixer, self.norm2, self.ffn = norm1, mixer, norm2, ffn
        self.conn1, self.conn2 = HyperConnection(streams), HyperConnection(streams)
        self.entry1 = StreamsNorm(norm1, streams, self.conn1)
        self.entry2 = StreamsNorm(norm2, streams, self.conn2) if ffn is not None else None
        self.names = dict(names)

    def sub_parts(self) -> Dict[str, Part]:
        n = self.names
        out = {n["norm1"]: self.norm1, n["conn1"]: self.conn1}
        out.update(_leaves(n["mixer"], self.mixer))
        if self.ffn is not None:
            out.update({n["norm2"]: self.norm2, n["conn2"]: self.conn2})
            out.update(_leaves(n["ffn"], self.ffn))
        else:
            # a layer without feed-forward: a folder that stores the second sub-layer's norm and connection all the same is
            # not at fault
            import dataclasses
            specs = {n["norm2"] + k: v for k, v in self.norm1.param_specs().items()}
            specs.update({n["conn2"] + k: v for k, v in self.conn2.param_specs().items()})
            out[""] = UnusedTensors({k: dataclasses.replace(v, optional=True) for k, v in specs.items()})
        return out

    def entry_norm(self):
        return self.entry1

    def _update(self, ctx, stream, result, conn: HyperConnection, reader):
        if not isinstance(result, torch.Tensor):
            raise NotImplementedError("hyper_connected block: a sub-layer hands out a tensor or a stack of partial sums")
        in_, norm = reader.coefficients() if isinstance(reader, StreamsNorm) else (None, None)
        stream.h, y = kernels.streams_update(stream.h, self.streams, ctx.compute_dtype, y=result, mix=conn.mix, out=conn.out,
                                             in_=in_, next_norm=norm)
        stream.prepared = (reader, y) if y is not None else None

    def forward(self, ctx, stream, cache_view):
        after = stream.after_block
        stream.next_norm = None
        y = self.entry1.forward(ctx, stream)
        r = self.mixer.output(ctx, y, cache_view)
        if self.ffn is None:
            self._update(ctx, stream, r, self.conn1, after)
            return
        self._update(ctx, stream, r, self.conn1, self.entry2)
        y = self.entry2.forward(ctx, stream)
        self._update(ctx, stream, self.ffn.output(ctx, y), self.conn2, after)
