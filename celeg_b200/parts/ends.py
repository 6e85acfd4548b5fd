"""The two ends of a model as parts: what turns a step's token ids into rows of the residual stream
("input") and what turns the stream's wanted rows into logits ("output"). A model description that
names neither gets the two below, built from its embedding table, final norm, head and scale factors;
one that needs something else at an end (a norm after the embedding, capped logits, several heads)
names a kind of its own, registered like any other part.

An input part has ``run(stream, step, first)``: write ``stream.residual[:step.tokens]``; ``first`` is
None or ``(norm weight, SplitNorm)`` of the first block's norm, which the part may prepare (and then sets
``stream.prepared``); when ``stream.wants_rows`` it may leave the rows in the activation type in ``stream.rows`` (and then
sets ``stream.rows_current``). ``vocab_size`` is the number of token ids it takes.
An output part has ``next_norm(step, n_logits)``: the norm it applies first if it takes it split over the
last block's closing product and its own (else None), and ``run(stream, step, logit_rows, n_logits,
logits)``: float32 logits of the stream's rows ``logit_rows[:n_logits]`` (all rows in order when
``step.logits_of_all_rows``) into ``logits[:n_logits]``.

celeg's counterparts: the embedding gather and the tied or untied LM head of the packed executor
(src/backend/cuda/packed/operators.cu:19-64, src/backend/cuda/packed/logits.cu:12-77).
"""
from __future__ import annotations

from typing import Mapping

import torch

from .. import kernels
from .norms import RmsNorm
from .registry import register_part
from .runtime import Runtime, StepContext


@register_part("input", "embedding")
class EmbeddingInput:
    """rows = multiplier * table[token ids] in float32; the first half of the first block's norm when asked.
    With ``sinusoid_base`` b a vector of the token's position p is added (Vaswani et al., "Attention Is All You
    Need", 2017, with sine and cosine side by side instead of in two halves): entry 2i is sin(p b^(-2i / width)),
    entry 2i + 1 the cosine of the same angle; the frequencies are made in float64 and kept in float32, the angle
    is a float32 product."""

    def __init__(self, params: Mapping, weights: Mapping[str, torch.Tensor], parts: Mapping, rt: Runtime):
        self.rt = rt
        self.table = rt.matrix(weights["table"])
        self.vocab_size = int(self.table.shape[0])
        self.multiplier = float(params.get("multiplier", 1.0))
        base = params.get("sinusoid_base")
        self.frequencies = None
        if base is not None:
            width = int(self.table.shape[1])
            pairs = torch.arange((width + 1) // 2, dtype=torch.float64)
            self.frequencies = torch.pow(torch.tensor(float(base), dtype=torch.float64), -2.0 * pairs / width).to(
                device=rt.device, dtype=torch.float32)

    def run(self, stream, step: StepContext, first=None) -> None:
        tokens = step.token_ids[:step.tokens]
        places = {} if self.frequencies is None else {"positions": step.positions, "frequencies": self.frequencies}
        if first is not None:
            norm, (weight, split) = first
            kernels.embedding(self.table, tokens, stream.residual, self.multiplier, prepare=split, next_weight=weight,
                              **places)
            stream.prepared = (norm, split)
        elif stream.wants_rows and stream.rows is not stream.residual and not places:
            kernels.embedding(self.table, tokens, stream.residual, self.multiplier, copy=stream.rows)
            stream.rows_current = True
        else:
            kernels.embedding(self.table, tokens, stream.residual, self.multiplier, **places)


@register_part("output", "norm_head")
class NormHeadOutput:
    """logits = multiplier * (norm(stream rows) @ head^T): the nested part ``norm``, then the head matrix
    (the embedding table itself when the description ties them: the runtime places a tensor once); with
    ``softcap`` the logits are then capped smoothly: cap * tanh(logits / cap)."""

    def __init__(self, params: Mapping, weights: Mapping[str, torch.Tensor], parts: Mapping, rt: Runtime):
        self.rt = rt
        self.norm = parts["norm"]
        self.head = rt.matrix(weights["head"])
        self.multiplier = float(params.get("multiplier", 1.0))
        cap = params.get("softcap")
        self.softcap = float(cap) if cap else None        # logits <- cap * tanh(logits / cap)
        if self.multiplier != 1.0 and isinstance(self.norm, RmsNorm):      # (the norm's weight is a scale: one for both)
            self.norm.weight.mul_(self.multiplier)
            self.multiplier = 1.0
        self.normed = rt.scratch("model.final_normed", int(self.head.shape[1]))

    def next_norm(self, step: StepContext, n_logits: int):
        if n_logits > 0 and step.logits_of_all_rows and self.rt.takes_split_norm(n_logits, self.head):
            return self.norm
        return None

    def run(self, stream, step: StepContext, logit_rows: torch.Tensor, n_logits: int, logits: torch.Tensor) -> None:
        if step.logits_of_all_rows:
            normed = stream.normed(self.norm, self.normed, n_logits)
        else:
            normed = stream.normed(self.norm, self.normed, n_logits, gather=logit_rows)
        self.rt.linear(normed, self.head, logits, n_logits)
        if self.multiplier != 1.0:
            logits[:n_logits].mul_(self.multiplier)
        if self.softcap is not None:
            kernels.softcap(logits, n_logits, self.softcap)
