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
(csrc/hyper_connections.cu); the last norm's reader gets the norm of the streams' sum for the rows it wants.
"""
from __future__ import annotations

from typing import Mapping, Optional

import torch

from .. import kernels
from .registry import register_part
from .runtime import ResidualStream, Runtime, StepContext


class StreamCopies:
    def __init__(self, rt: Runtime, count: int, width: int):
        self.count, self.width = count, width
        self.streams = rt.flat_scratch("hyper.streams", rt.max_tokens * count * width, torch.float32)
        self.close()

    def close(self) -> None:
        self.open = False
        self.single: Optional[torch.Tensor] = None       # the row that stands for every stream so far
        self.owed = None                                 # (connection, output, second output, both outputs' norms)

    def begin(self, stream: ResidualStream) -> None:
        """All streams become the stream's rows as they are."""
        if stream.pending is not None or stream.pending_b is not None or stream.prepared is not None:
            raise RuntimeError("the streams are opened from a stream that something is owed to")
        self.open, self.single, self.owed = True, stream.residual, None

    def read(self, connection: "HyperConnection", norm, out: torch.Tensor, rows: int) -> torch.Tensor:
        """out = norm(sum_s take[s] x_s), what is owed mixed in for good."""
        self._pass(out, rows, norm, connection.take, None)
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

    def _sublayer(self, connection, norm, part, copies: StreamCopies, step: StepContext) -> None:
        x = copies.read(connection, norm, self.normed, step.tokens)
        pair = part.forward_normed_pair(x, step) if hasattr(part, "forward_normed_pair") else None
        if pair is not None:
            first, second, norms = pair
            copies.owe(connection, first, second, norms)
            return
        output = self.output if getattr(part, "ends_with_product", False) else self.delta
        part.forward(x, output, step)
        copies.owe(connection, output)

    def run(self, stream: ResidualStream, step: StepContext) -> None:
        copies = stream.copies
        if copies is None:
            copies = stream.copies = self.copies
        if not copies.open:
            copies.begin(stream)
        if copies.count != self.mixer_connection.streams:
            raise RuntimeError(f"a block of {self.mixer_connection.streams} streams among blocks of {copies.count}")
        self._sublayer(self.mixer_connection, self.mixer_norm, self.mixer, copies, step)
        if self.ffn is not None:
            self._sublayer(self.ffn_connection, self.ffn_norm, self.ffn, copies, step)
