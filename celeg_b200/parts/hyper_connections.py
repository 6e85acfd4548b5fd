"""Several residual streams in place of one (Zhu et al., "Hyper-Connections", 2024; here with stored weights).

    StreamCopies                 the streams of a step (float32 [tokens, count, width]) and the output owed to them; a
                                 ResidualStream whose blocks open them answers its norms from them
    connection kind "hyper"      a sublayer's weights: ``take`` (how the streams make what it reads), ``mix`` [from, to] and
                                 ``give`` (how its output enters them)
    arrangement kind "hyper_residual"   u = sum_s take[s] x_s; y = Sublayer(Norm(u)); x_t <- sum_s mix[s, t] x_s + give[t] y,
                                 for the mixer and for the feed-forward, each with its connection
                                 (``mixer_connection``, ``feed_forward_connection``)

All streams begin as the embedding row, which stays where the input part wrote it until the first sublayer's output is
mixed in. What lies between two sublayers (mixing an output in, the next weighted sum, its norm) is one launch
(csrc/hyper_connections.cu); the last norm's reader gets the norm of the streams' sum for the rows it wants. In steps of few
rows on the bfloat16 path that launch falls away too where a sublayer ends in a product and the next one begins with one:
the product mixes itself in and prepares the next norm (csrc/gemv_bf16.cu), as it does for one stream.
"""
from __future__ import annotations

from typing import Mapping, Optional

import torch

from .. import kernels
from .registry import register_part
from .runtime import ResidualStream, Runtime, StepContext, _Sink


class StreamCopies:
    def __init__(self, rt: Runtime, count: int, width: int):
        self.count, self.width = count, width
        self.streams = rt.flat_scratch("hyper.streams", rt.max_tokens * count * width, torch.float32)
        self.close()

    def close(self) -> None:
        self.open = False
        self.single: Optional[torch.Tensor] = None       # the row that stands for every stream so far
        self.owed = None                                 # (connection, output, second output, both outputs' norms)
        self.prepared = None                             # (connection or None, norm, SplitNorm) left by the last product

    def begin(self, stream: ResidualStream) -> None:
        """All streams become the stream's rows as they are."""
        if stream.pending is not None or stream.pending_b is not None or stream.prepared is not None:
            raise RuntimeError("the streams are opened from a stream that something is owed to")
        self.open, self.single, self.owed, self.prepared = True, stream.residual, None, None

    def read(self, connection: "HyperConnection", norm, out: torch.Tensor, rows: int) -> torch.Tensor:
        """out = norm(sum_s take[s] x_s), what is owed mixed in for good; or the split norm that the last product prepared
        for exactly this reader."""
        if self.prepared is not None:
            return self._prepared_for(connection, norm)
        self._pass(out, rows, norm, connection.take, None)
        return out

    def _prepared_for(self, connection, norm):
        prepared, self.prepared = self.prepared, None
        if prepared[0] is not connection or prepared[1] is not norm:
            raise RuntimeError("a norm was prepared for another reader than the one that asks")
        return prepared[2]

    def expect(self, stream: ResidualStream, buffer: torch.Tensor, connection: "HyperConnection", reader, rows: int) -> None:
        """A sublayer with weights ``connection`` is about to write its output to ``buffer``; ``reader`` = (connection or
        None, norm) of what reads the streams after it (None: it wants normalised rows)."""
        rt = stream.rt
        rt.sink = None
        if reader is None or reader[1] is None or not rt.small_batch(rows) or self.count > kernels.GEMV_MAX_STREAMS:
            return
        halves = stream.split(reader[1], stream.pieces)
        if halves is not None:
            rt.sink = _Sink(buffer, reader[1], halves[0], halves[1], copies=self)
            self.mixing, self.reader = connection, reader[0]

    def take_product(self, x, weight: torch.Tensor, rows: int, sink: _Sink, ahead) -> None:
        kernels.gemv_hyper(x, weight, rows, self.streams, self.count, self.mixing.mix, self.mixing.give,
                           self.reader.take if self.reader is not None else None, sink.split, sink.weight, single=self.single,
                           ahead=ahead)
        self.single = None
        self.prepared = (self.reader, sink.norm, sink.split)

    def closing(self, norm, out: torch.Tensor, rows: int, gather: Optional[torch.Tensor] = None):
        """norm(sum of the streams) of the rows (or the gathered ones) in ``out``, or as the last product prepared it."""
        if self.prepared is not None and gather is None:
            return self._prepared_for(None, norm)
        self.total(out, rows, norm=norm, gather=gather)
        return out

    def owe(self, connection: "HyperConnection", y: torch.Tensor, second: Optional[torch.Tensor] = None, norms=None) -> None:
        """A sublayer's output: ``y``, or the normed sum of ``y`` and ``second`` with ``norms`` = (weight, weight, eps)."""
        assert self.owed is None
        self.owed = (connection, y, second, norms)

    def total(self, out: torch.Tensor, rows: int, norm=None, gather: Optional[torch.Tensor] = None) -> None:
        """out = norm(sum of the streams) with what is owed (which stays owed); no norm: the sum."""
        self._pass(out, rows, norm, None, gather, keep=True)

    def _pass(self, out, rows, norm, take, gather, keep=False) -> None:
        weight, eps = norm.as_prologue() if norm is not None else (None, 0.0)
        mixing = {}
        if self.owed is not None:
            connection, y, second, norms = self.owed
            mixing = {"y": y, "mix": connection.mix, "give": connection.give}
            if second is not None:
                mixing.update(y2=second, y_norms=(norms[0], norms[1], norms[2], 1.0))
        kernels.hyper_connect(self.streams, self.count, out, rows, self.width, single=self.single, take=take,
                              norm_weight=weight, eps=eps, gather=gather, write=not keep, **mixing)
        if self.owed is not None and not keep:
            self.single, self.owed = None, None


@register_part("connection", "hyper")
class HyperConnection:
    def __init__(self, params: Mapping, weights: Mapping[str, torch.Tensor], parts: Mapping, rt: Runtime):
        self.streams, self.width = int(params["streams"]), int(params["width"])
        self.take, self.give = rt.vector(weights["take"].reshape(-1)), rt.vector(weights["give"].reshape(-1))
        self.mix = rt.vector(weights["mix"])
        n = self.streams
        if self.take.shape != (n,) or self.give.shape != (n,) or self.mix.shape != (n, n):
            raise ValueError(f"hyper connection of {n} streams: weights of shapes {tuple(self.take.shape)}, "
                             f"{tuple(self.give.shape)}, {tuple(self.mix.shape)}")


@register_part("arrangement", "hyper_residual")
class HyperResidual:
    """A pre-norm block over several streams. A part whose last step is a product writes float32 rows for it, and a mixer
    that ends in the normed sum of two outputs hands both over (``forward_normed_pair``), so that what is mixed into the
    streams was not rounded."""

    def __init__(self, layer_parts: Mapping, rt: Runtime):
        self.rt = rt
        self.mixer_norm, self.mixer = layer_parts["mixer_norm"], layer_parts["mixer"]
        self.ffn_norm, self.ffn = layer_parts.get("feed_forward_norm"), layer_parts.get("feed_forward")
        self.mixer_connection = layer_parts["mixer_connection"]
        self.ffn_connection = layer_parts.get("feed_forward_connection")
        if (self.ffn is None) != (self.ffn_connection is None):
            raise ValueError("hyper_residual: a feed-forward and its connection come together")
        for norm in (self.mixer_norm, self.ffn_norm):
            if norm is not None and (not hasattr(norm, "as_prologue") or norm.as_prologue() is None):
                raise ValueError("hyper_residual: the norms must be plain RMS norms")
        hidden = self.mixer_norm.width
        self.copies = StreamCopies(rt, self.mixer_connection.streams, hidden)     # (all blocks' are over the same streams)
        self.normed = rt.scratch("block.normed", hidden)
        self.output = rt.scratch("block.output", hidden, torch.float32)
        self.delta = rt.scratch("block.delta_a", hidden)

    def _sublayer(self, connection, norm, part, reader, stream: ResidualStream, copies: StreamCopies,
                  step: StepContext) -> None:
        x = copies.read(connection, norm, self.normed, step.tokens)
        self.rt.sink = None
        pair = part.forward_normed_pair(x, step) if hasattr(part, "forward_normed_pair") else None
        if pair is not None:
            first, second, norms = pair
            copies.owe(connection, first, second, norms)
            return
        if not getattr(part, "ends_with_product", False):
            part.forward(x, self.delta, step)
            copies.owe(connection, self.delta)
            return
        copies.expect(stream, self.output, connection, reader, step.tokens)
        part.forward(x, self.output, step)
        sink, self.rt.sink = self.rt.sink, None
        if sink is None or not sink.used:
            copies.owe(connection, self.output)

    @staticmethod
    def _takes_split(part, step: StepContext) -> bool:
        takes = getattr(part, "takes_split_norm", None)
        return takes is not None and takes(step)

    def entry_reader(self, step: StepContext):
        """(connection, norm) that the streams are read through first, if that reader takes a split norm."""
        return (self.mixer_connection, self.mixer_norm) if self._takes_split(self.mixer, step) else None

    def run(self, stream: ResidualStream, step: StepContext) -> None:
        copies = stream.copies
        if copies is None:
            copies = stream.copies = self.copies
        if not copies.open:
            copies.begin(stream)
        if copies.count != self.mixer_connection.streams:
            raise RuntimeError(f"a block of {self.mixer_connection.streams} streams among blocks of {copies.count}")
        after = stream.reader if stream.reader is not None else (None, stream.after_layer)
        if self.ffn is None:
            self._sublayer(self.mixer_connection, self.mixer_norm, self.mixer, after, stream, copies, step)
            return
        between = (self.ffn_connection, self.ffn_norm) if self._takes_split(self.ffn, step) else None
        self._sublayer(self.mixer_connection, self.mixer_norm, self.mixer, between, stream, copies, step)
        self._sublayer(self.ffn_connection, self.ffn_norm, self.ffn, after, stream, copies, step)
