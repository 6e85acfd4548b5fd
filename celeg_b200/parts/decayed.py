"""Mixers whose matrix state per head decays at a rate that the token decides (kernels: csrc/decayed_scan.cu, the short
convolutions csrc/channel_conv.cu). State, decays, steps and every sum of the recurrence are float32 on both precision
paths; the projections run in the path's matrix type and leave float32 results.

    mamba2                   S' = a S + dt B x^T with one decay a = exp(-exp(A_log) dt) a token and head, read-out S'^T C + D x
                             (Dao and Gu, "Transformers are SSMs: Generalized Models and Efficient Algorithms Through
                             Structured State Space Duality", 2024)
    gated_linear_attention   S' = diag(a) S + k v^T with a decay a = sigmoid(z)^(1 / tau) a token and key channel, read-out
                             S'^T q (Yang et al., "Gated Linear Attention Transformers with Hardware-Efficient Training",
                             2024)

The single tokens at the head of a step (decoding requests) go to the decoding kernel, the portions behind them to the
chunked scan.
"""
from __future__ import annotations

from typing import Mapping, Optional

import torch

from .. import kernels
from ..cache.manager import StateNeed
from .mixers import StateBinding
from .registry import register_part
from .runtime import Runtime, StepContext


class ChunkedSpans:
    """The chunks that a step's portions are cut into: how many at most, and their plan on the device, which the first mixer
    of a run makes for all of them."""

    def __init__(self, rt: Runtime):
        self.tokens = kernels.chunk_tokens()
        self.max_chunks = rt.max_tokens // self.tokens + rt.max_requests + 48
        self.plan = rt.flat_scratch("decay.plan", 2 * self.max_chunks + rt.max_tokens + 64, torch.int32)

    def of(self, step: StepContext, single: int):
        """(plan, spans, bound of the chunks) of the spans from ``single`` on."""
        spans = step.spans - single
        chunks = (step.tokens - single) // self.tokens + spans
        if chunks > self.max_chunks:
            raise ValueError(f"{chunks} chunks of a step exceed the {self.max_chunks} that the scratch holds")
        key = ("decay.plan", single)
        if key not in step.extras:
            kernels.chunk_plan(step.span_begin[single:], spans, self.max_chunks, self.plan)
            step.extras[key] = True
        return self.plan, spans, chunks


def _padded_rows(matrix: torch.Tensor, multiple: int = 8) -> torch.Tensor:
    """Zero rows at the end, so that a product's rows stay 16-byte aligned."""
    missing = -matrix.shape[0] % multiple
    if not missing:
        return matrix
    return torch.cat([matrix, torch.zeros((missing, matrix.shape[1]), dtype=matrix.dtype)], dim=0)


@register_part("mixer", "mamba2")
class Mamba2Mixer:
    """One projection [z | x | B | C | dt] (inner = heads * vdim channels of z and x, groups * state of B and C, one step a
    head). x, B and C go through a causal convolution per channel (tensor ``conv`` [channels, taps], ``conv_bias``) and SiLU;
    dt <- softplus(dt + ``dt_bias``). Per head (head h reads group h // (heads / groups))
    S <- exp(-exp(``a_log``) dt) S + dt B x^T and y = S^T C + ``direct`` x. All heads' y times SiLU(z), RMS-normed in
    ``norm_groups`` equal parts, times ``norm`` and projected by W_o. Per-request state, float32, zero for a new request: S
    per head, then the last taps - 1 inputs of the convolution.

    Portions: projection, convolution, the chunked scan, gate and norm, projection. Decoding: the scan is one launch."""

    def __init__(self, params: Mapping, weights: Mapping[str, torch.Tensor], parts: Mapping, rt: Runtime):
        self.rt = rt
        self.hidden = int(params["hidden_size"])
        self.heads, self.vdim = int(params["heads"]), int(params["vdim"])
        self.state, self.groups = int(params["state"]), int(params["groups"])
        self.taps, self.norm_groups = int(params["taps"]), int(params["norm_groups"])
        self.eps = float(params["eps"])
        inner = self.inner = self.heads * self.vdim
        self.shared = self.groups * self.state
        self.channels = inner + 2 * self.shared
        if self.heads % self.groups or inner % self.norm_groups:
            raise ValueError(f"mamba2: {self.heads} heads in {self.groups} groups, {inner} channels in {self.norm_groups} norm "
                             f"groups")
        if not 1 <= self.taps <= 16:
            raise ValueError(f"mamba2: {self.taps} taps (1 to 16)")
        if tuple(weights["in_proj"].shape) != (inner + self.channels + self.heads, self.hidden):
            raise ValueError(f"mamba2: a projection of shape {tuple(weights['in_proj'].shape)}")
        self.w_in = rt.matrix(_padded_rows(weights["in_proj"]))
        self.w_out = rt.matrix(weights["out"])
        self.kernel = rt.vector(weights["conv"].reshape(self.channels, self.taps))
        self.conv_bias = rt.vector(weights["conv_bias"]) if "conv_bias" in weights else None
        self.dt_bias, self.a_log = rt.vector(weights["dt_bias"]), rt.vector(weights["a_log"])
        self.direct = rt.vector(weights["direct"]) if "direct" in weights else None
        self.norm = rt.vector(weights["norm"])
        self.state_elements = self.heads * self.state * self.vdim
        self.binding: Optional[StateBinding] = None
        self.carried: Optional[torch.Tensor] = None
        self.spans = ChunkedSpans(rt)
        chunks = self.spans.max_chunks
        self.projected = rt.scratch("recurrent.proj", int(self.w_in.shape[0]), torch.float32)
        self.convolved = rt.scratch("recurrent.conv", self.channels, torch.float32)
        self.cum = rt.scratch("decay.cum", 2 * self.heads, torch.float32)
        self.dt = rt.scratch("decay.dt", self.heads, torch.float32)
        self.products = rt.flat_scratch("decay.products", chunks * self.groups * self.spans.tokens ** 2, torch.float32)
        self.states = rt.flat_scratch("decay.states", chunks * self.state_elements, torch.float32)
        self.read = rt.scratch("recurrent.read", inner, torch.float32)
        self.gated = rt.scratch("recurrent.gated", inner)

    def cache_need(self):
        return StateNeed(elements=self.state_elements + (self.taps - 1) * self.channels)

    def bind_cache(self, binding: StateBinding) -> None:
        self.binding = binding
        self.carried = binding.state[:, self.state_elements:] if self.taps > 1 else None

    ends_with_product = True      # forward() writes `out` last, with rt.linear

    def takes_split_norm(self, step: StepContext) -> bool:
        return self.rt.takes_split_norm(step.tokens, self.w_in)

    def forward(self, x: torch.Tensor, out: torch.Tensor, step: StepContext) -> None:
        rt, t, b = self.rt, step.tokens, self.binding
        rt.linear(x, self.w_in, self.projected, t)
        rows, inner, conv = self.projected, self.inner, self.convolved
        alone = step.max_span == 1 and step.spans == t
        kernels.channel_conv(rows[:, inner:inner + self.channels], self.kernel, self.conv_bias, self.carried, b.slot_stride,
                             step.token_span, step.span_begin, step.span_slot, conv, t, step.spans, kernels.ACT_SILU,
                             single=alone)
        v, k = conv[:, :inner], conv[:, inner:inner + self.shared]
        q = conv[:, inner + self.shared:]
        raw = rows[:, inner + self.channels:inner + self.channels + self.heads]
        single = t if alone else step.leading_single_tokens
        if single:
            kernels.scalar_decay_decode(q, k, v, raw, self.dt_bias, self.a_log, self.direct, b.state, b.slot_stride,
                                        step.span_slot, single, self.heads, self.groups, self.state, self.vdim, self.read)
        if single < t:
            plan, spans, chunks = self.spans.of(step, single)
            kernels.scalar_decay_scan(q, k, v, raw, self.dt_bias, self.a_log, self.direct, self.cum, self.dt, self.products,
                                      self.states, self.read, b.state, b.slot_stride, step.span_slot[single:], plan,
                                      self.spans.max_chunks, spans, chunks, self.heads, self.groups, self.state, self.vdim)
        kernels.gated_head_norm(self.read, rows[:, :inner], self.norm, True, self.gated, t, self.norm_groups,
                                inner // self.norm_groups, self.eps, kernels.GATE_SILU + kernels.GATE_BEFORE_NORM)
        rt.linear(self.gated, self.w_out, out, t)


@register_part("mixer", "gated_linear_attention")
class GatedLinearAttentionMixer:
    """q = W_q x / sqrt(dim), k = W_k x (heads x dim), v = W_v x (heads x vdim); a decay per key channel
    a = sigmoid(W_2 (W_1 x) + b)^(1 / tau). Per head S <- diag(a) S + k v^T and the read-out S^T q. Each head's read-out is
    divided by its root mean square, scaled by ``norm`` (vdim, shared by the heads), gated by SiLU(W_g x) and projected by
    W_o. Per-request state: S per head, float32, zero for a new request.

    One fused [q | k | v | gate | W_1] projection leaves float32 sums. Decoding: one launch between the two projections.
    Portions: the product with W_2, the chunked scan, the heads' norm and gate. The rank of W_2 W_1 is padded with zero rows
    and columns to a multiple of eight."""

    def __init__(self, params: Mapping, weights: Mapping[str, torch.Tensor], parts: Mapping, rt: Runtime):
        self.rt = rt
        self.hidden = int(params["hidden_size"])
        self.heads, self.dim, self.vdim = int(params["heads"]), int(params["dim"]), int(params["vdim"])
        self.tau, self.eps = float(params["tau"]), float(params["eps"])
        if self.dim > kernels.DECAY_MAX_DIM:
            raise ValueError(f"gated_linear_attention: a key size of {self.dim} exceeds {kernels.DECAY_MAX_DIM}")
        if not self.tau > 0:
            raise ValueError(f"gated_linear_attention: tau {self.tau}")
        qk, vw = self.qk_width, self.v_width = self.heads * self.dim, self.heads * self.vdim
        down, up = _padded_rows(weights["decay_down"]), weights["decay_up"]
        self.rank = int(down.shape[0])
        if self.rank != up.shape[1]:
            up = torch.cat([up, torch.zeros((up.shape[0], self.rank - up.shape[1]), dtype=up.dtype)], dim=1)
        stacked = torch.cat([weights["q"], weights["k"], weights["v"], weights["gate"], down], dim=0)
        self.low_at = 2 * (qk + vw)
        self.w_in = rt.matrix(_padded_rows(stacked))
        self.w_decay, self.w_out = rt.matrix(up), rt.matrix(weights["out"])
        self.decay_bias, self.norm = rt.vector(weights["decay_bias"]), rt.vector(weights["norm"])
        if self.decay_bias.shape != (qk,) or self.norm.shape != (self.vdim,):
            raise ValueError(f"gated_linear_attention: bias and norm have shapes {tuple(self.decay_bias.shape)} and "
                             f"{tuple(self.norm.shape)}, expected ({qk},) and ({self.vdim},)")
        self.binding: Optional[StateBinding] = None
        self.spans = ChunkedSpans(rt)
        chunks = self.spans.max_chunks
        self.projected = rt.scratch("linear_attention.proj", int(self.w_in.shape[0]), torch.float32)
        self.low = rt.scratch("linear_attention.low", self.rank)
        self.z = rt.scratch("linear_attention.z", qk, torch.float32)
        self.q_taken = rt.scratch("linear_attention.q", qk, torch.float32)
        self.k_taken = rt.scratch("linear_attention.k", qk, torch.float32)
        self.total = rt.flat_scratch("linear_attention.total", chunks * qk, torch.float32)
        self.products = rt.flat_scratch("linear_attention.products", chunks * self.heads * self.spans.tokens ** 2, torch.float32)
        self.states = rt.flat_scratch("linear_attention.states", chunks * self.heads * self.dim * self.vdim, torch.float32)
        self.read = rt.scratch("linear_attention.read", vw, torch.float32)
        self.gated = rt.scratch("linear_attention.gated", vw)

    def cache_need(self):
        return StateNeed(elements=self.heads * self.dim * self.vdim)

    def bind_cache(self, binding: StateBinding) -> None:
        self.binding = binding

    ends_with_product = True      # forward() writes `out` last, with rt.linear

    def takes_split_norm(self, step: StepContext) -> bool:
        return self.rt.takes_split_norm(step.tokens, self.w_in)

    def forward(self, x: torch.Tensor, out: torch.Tensor, step: StepContext) -> None:
        rt, t, b, qk, vw = self.rt, step.tokens, self.binding, self.qk_width, self.v_width
        rt.linear(x, self.w_in, self.projected, t)
        rows = self.projected
        q, k, v = rows[:, :qk], rows[:, qk:2 * qk], rows[:, 2 * qk:2 * qk + vw]
        gate, low = rows[:, 2 * qk + vw:self.low_at], rows[:, self.low_at:self.low_at + self.rank]
        scale = self.dim ** -0.5
        single = t if step.max_span == 1 and step.spans == t else step.leading_single_tokens
        if single:
            kernels.channel_decay_decode(q, k, v, scale, low, self.w_decay, self.decay_bias, self.tau, self.norm, self.eps,
                                         gate, b.state, b.slot_stride, step.span_slot, single, self.heads, self.dim, self.vdim,
                                         self.gated)
        if single < t:
            kernels.activation_cast(low, self.low, t, -1)
            rt.linear(self.low, self.w_decay, self.z, t)
            plan, spans, chunks = self.spans.of(step, single)
            kernels.channel_decay_scan(q, k, v, self.z, self.decay_bias, self.tau, scale, self.q_taken, self.k_taken,
                                       self.total, self.products, self.states, self.read, b.state, b.slot_stride,
                                       step.span_slot[single:], plan, self.spans.max_chunks, spans, chunks, self.heads,
                                       self.dim, self.vdim)
            kernels.gated_head_norm(self.read[single:], gate[single:], self.norm, False, self.gated[single:], t - single,
                                    self.heads, self.vdim, self.eps, kernels.GATE_SILU)
        rt.linear(self.gated, self.w_out, out, t)
