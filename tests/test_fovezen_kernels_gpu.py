"""The kernels that the Fovezen design added or widened, each against the same operation written in numpy (float64): the
pass over several residual streams (as a launch of its own and in the weight-streaming product), the normed sum of two
outputs, short convolutions with carried inputs, the scans and decoding steps with token-dependent decays, norms behind a
gate, softly capped scores in all four attention kernels, and clamped gates in both gated products."""
from __future__ import annotations

import math

import numpy as np
import pytest
import torch

import plain_fovezen as plain
from test_liverax_kernels_gpu import KERNELS, Paged, bf16_round, close, gpu, kernels, run_attention

pytestmark = pytest.mark.gpu

DEVICE = "cuda:0"
DTYPES = [(torch.float32, 4e-6), (torch.bfloat16, 6e-3)]


def rounded(array, dtype):
    return bf16_round(array) if dtype == torch.bfloat16 else np.asarray(array, dtype=np.float32).astype(np.float64)


def f32(array):
    return np.asarray(array, dtype=np.float32).astype(np.float64)


# --------------------------------------------------------------------------------------------- several streams
@pytest.mark.parametrize("dtype,rel", DTYPES)
@pytest.mark.parametrize("tokens,width,count", [(5, 36, 3), (3, 64, 1), (7, 515, 2), (170, 2048, 4), (9, 2048, 3), (2, 9000, 4),
                                                (3, 20000, 2), (200, 1024, 5), (4, 256, 8), (2, 100, 16), (150, 4096, 16)])
def test_a_pass_over_the_streams(tokens, width, count, dtype, rel):
    k = kernels()
    rng = np.random.default_rng(width + count)
    eps = 1e-5
    copies = f32(rng.normal(0.5, 2.0, size=(tokens, count, width)))
    single = f32(rng.normal(size=(tokens, width)))
    first, second = f32(rng.normal(size=(tokens, width))), f32(3.0 * rng.normal(size=(tokens, width)))
    mix, give, take = (f32(rng.normal(size=size)) for size in ((count, count), count, count))
    norm, first_w, second_w = (f32(1.0 + 0.3 * rng.normal(size=width)) for _ in range(3))

    def spread(old, y):
        return np.einsum("tsw,su->tuw", old, mix) + give[None, :, None] * y[:, None, :]

    def normed(x):
        return x / np.sqrt((x ** 2).mean(-1, keepdims=True) + eps)

    pair = normed(first) * first_w + normed(second) * second_w
    weights = {"mix": gpu(mix), "give": gpu(give)}
    for tag, old, y, args in (
            ("one output", copies, first, {"y": gpu(first), **weights}),
            ("an output in the activation type", copies, rounded(first, dtype), {"y": gpu(first, dtype), **weights}),
            ("two normed outputs", copies, pair, {"y": gpu(first), "y2": gpu(second), **weights,
                                                  "y_norms": (gpu(first_w), gpu(second_w), eps, 1.0)}),
            ("one row for all", np.repeat(single[:, None], count, axis=1), first, {"y": gpu(first), "single": gpu(single), **weights}),
            ("nothing to mix in", np.repeat(single[:, None], count, axis=1), None, {"single": gpu(single)})):
        want_streams = old if y is None else spread(old, y)
        u = np.einsum("tsw,s->tw", want_streams, take)
        streams = gpu(copies)
        out = torch.zeros((tokens, width), dtype=dtype, device=DEVICE)
        k.hyper_connect(streams, count, out, tokens, width, take=gpu(take), norm_weight=gpu(norm), eps=eps, **args)
        close(out, normed(u) * norm, rel, f"{tag}: what the next sublayer reads")
        close(streams, copies if y is None else want_streams, 3e-6, f"{tag}: the streams")
        # the head's reader: the sum of the streams for gathered rows, the streams left alone
        streams = gpu(copies)
        picked = gpu([tokens - 1, 0], torch.int32)
        k.hyper_connect(streams, count, out, 2, width, norm_weight=gpu(norm), eps=eps, gather=picked, **args)
        close(out[:2], (normed(want_streams.sum(1)) * norm)[[tokens - 1, 0]], rel, f"{tag}: gathered rows")
        assert torch.equal(streams, gpu(copies))
        plain_sum = torch.zeros((tokens, width), dtype=torch.float32, device=DEVICE)
        k.hyper_connect(streams, count, plain_sum, tokens, width, write=False, **args)
        close(plain_sum, want_streams.sum(1), 5e-6, f"{tag}: the sum")
        assert torch.equal(streams, gpu(copies))


@pytest.mark.parametrize("rows,n,depth,count", [(1, 64, 64, 4), (8, 256, 96, 3), (16, 2048, 4096, 4), (9, 200, 72, 1), (5, 1040, 512, 2)])
@pytest.mark.parametrize("from_single", [False, True])
def test_the_product_that_mixes_itself_into_the_streams(rows, n, depth, count, from_single):
    k = kernels()
    rng = np.random.default_rng(n + count)
    eps = 1e-5
    x, w = bf16_round(rng.normal(size=(rows, depth))), bf16_round(rng.normal(size=(n, depth)) / math.sqrt(depth))
    copies, single = f32(rng.normal(size=(rows, count, n))), f32(rng.normal(size=(rows, n)))
    mix, give, take = (f32(rng.normal(size=size)) for size in ((count, count), count, count))
    norm = f32(1.0 + 0.3 * rng.normal(size=n))
    scaled_sums = rng.uniform(0.5, 2.0, size=(rows, 3)).astype(np.float32)
    for split_in in (False, True):
        y = x @ w.T
        operand = gpu(x, torch.bfloat16)
        if split_in:
            y = y / np.sqrt(f32(scaled_sums).sum(1, keepdims=True) / depth + eps)
            operand = k.SplitNorm(operand, gpu(scaled_sums), 3, eps, depth)
        old = np.repeat(single[:, None], count, axis=1) if from_single else copies
        want = np.einsum("tsw,su->tuw", old, mix) + give[None, :, None] * y[:, None, :]
        for weights in (take, None):
            u = want.sum(1) if weights is None else np.einsum("tsw,s->tw", want, weights)
            streams = gpu(copies)
            pieces = (n + 15) // 16
            split = k.SplitNorm(torch.zeros((rows, n), dtype=torch.bfloat16, device=DEVICE),
                                torch.zeros((rows, pieces), dtype=torch.float32, device=DEVICE), pieces, eps, n)
            k.gemv_hyper(operand, gpu(w, torch.bfloat16), rows, streams, count, gpu(mix), gpu(give),
                         None if weights is None else gpu(weights), split, gpu(norm), single=gpu(single) if from_single else None)
            close(streams, want, 1e-5, "the streams")
            close(split.xw, u * norm, 6e-3, "the prepared rows")
            close(split.sumsq.sum(1), (u ** 2).sum(-1), 1e-5, "the prepared sums")


@pytest.mark.parametrize("dtype,rel", DTYPES)
def test_the_normed_sum_of_two_outputs(dtype, rel):
    k = kernels()
    rng = np.random.default_rng(2)
    for width in (36, 700):
        a, b = f32(rng.normal(size=(5, width))), f32(20.0 * rng.normal(size=(5, width)))
        a_w, b_w = f32(rng.normal(size=width)), f32(rng.normal(size=width))
        out = torch.zeros((5, width), dtype=dtype, device=DEVICE)
        k.normed_pair(gpu(a), gpu(b), gpu(a_w), gpu(b_w), 1e-5, 0.5, out, 5)
        close(out, 0.5 * (plain.rms_scaled(a, 1e-5) * a_w + plain.rms_scaled(b, 1e-5) * b_w), rel, "normed sum")


# ------------------------------------------------------------------------------------------ short convolutions
class Spans:
    def __init__(self, lengths, stride, seed):
        rng = np.random.default_rng(seed)
        self.lengths, self.tokens, self.spans = lengths, sum(lengths), len(lengths)
        self.begin = np.concatenate([[0], np.cumsum(lengths)]).astype(np.int32)
        self.of = np.concatenate([np.full(n, s) for s, n in enumerate(lengths)]).astype(np.int32)
        self.slots = (np.arange(len(lengths)) * 2 + 1)[::-1].astype(np.int32).copy()
        self.state = rng.normal(size=(2 * len(lengths) + 1, stride)).astype(np.float32)
        self.dev = {"token_span": gpu(self.of, torch.int32), "span_begin": gpu(self.begin, torch.int32),
                    "span_slot": gpu(self.slots, torch.int32)}


@pytest.mark.parametrize("channels,offset", [(12, 0), (40, 8), (37, 3), (260, 4)])
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 5, 16])
@pytest.mark.parametrize("lengths", [[1], [1, 1, 1, 1, 1, 1, 1, 1, 1], [2, 1, 30, 3, 1, 5], [70], [1, 1, 3, 2]])
def test_short_convolutions_with_carried_inputs(channels, offset, taps, lengths):
    k = kernels()
    rng = np.random.default_rng(channels + taps)
    spans = Spans(lengths, (taps - 1) * channels + 8, 3)
    rows = rng.normal(size=(spans.tokens, channels + offset + 4)).astype(np.float32)
    w, bias = rng.normal(size=(channels, taps)).astype(np.float32), rng.normal(size=channels).astype(np.float32)
    for act, with_bias in ((-1, False), (k.ACT_SILU, True)):
        state = gpu(spans.state)
        out = torch.zeros((spans.tokens, channels), dtype=torch.float32, device=DEVICE)
        single = all(n == 1 for n in lengths)
        k.channel_conv(gpu(rows)[:, offset:offset + channels], gpu(w), gpu(bias) if with_bias else None, state,
                       spans.state.shape[1], spans.dev["token_span"], spans.dev["span_begin"], spans.dev["span_slot"], out,
                       spans.tokens, spans.spans, act, single=single)
        want_state = f32(spans.state)
        want = np.zeros((spans.tokens, channels))
        for s, slot in enumerate(spans.slots):
            mine = f32(rows[spans.begin[s]:spans.begin[s + 1], offset:offset + channels])
            before = want_state[slot, :(taps - 1) * channels].reshape(taps - 1, channels)
            joined = np.concatenate([before, mine])
            y = plain.causal_convolution(joined, f32(w), f32(bias) if with_bias else None)[taps - 1:]
            want[spans.begin[s]:spans.begin[s + 1]] = y if act < 0 else plain.silu(y)
            if taps > 1:
                want_state[slot, :(taps - 1) * channels] = joined[-(taps - 1):].reshape(-1)
        close(out, want, 3e-6, "convolved")
        assert torch.equal(state, gpu(want_state))


# --------------------------------------------------------------------------------- token-dependent decays
LENGTHS = [[1], [2], [64], [65], [200], [1, 1, 1], [3, 130, 1, 64, 9], [63, 128, 2]]


def walk(state, keys, values, decays, queries):
    """decayed_states from a given state; returns (read-outs, state after)."""
    out = np.zeros((keys.shape[0], values.shape[1]))
    for t in range(keys.shape[0]):
        state = np.reshape(decays[t], (-1, 1)) * state + np.outer(keys[t], values[t])
        out[t] = state.T @ queries[t]
    return out, state


@pytest.mark.parametrize("lengths", LENGTHS)
@pytest.mark.parametrize("heads,dim,vdim,tau", [(2, 8, 4, 16.0), (1, 5, 7, 1.0), (3, 64, 64, 4.0), (2, 33, 70, 1.0), (1, 128, 36, 16.0),
                                                (1, 250, 12, 2.0)])
def test_the_scan_and_the_decoding_step_with_a_decay_a_channel(heads, dim, vdim, tau, lengths):
    k = kernels()
    rng = np.random.default_rng(dim + len(lengths))
    elements = heads * dim * vdim
    spans = Spans(lengths, (elements + 3) // 4 * 4 + 4, 5)
    t, qk, vw = spans.tokens, heads * dim, heads * vdim
    q, key, v = (rng.normal(size=(t, n)).astype(np.float32) for n in (qk, qk, vw))
    # from decays of almost one to decays of almost nothing, which one block of tokens has everywhere
    z, bias = rng.normal(0.0, 2.0, size=(t, qk)).astype(np.float32), rng.uniform(-3.0, 4.0, size=qk).astype(np.float32)
    z[t // 3:t // 3 + 9] = -60.0
    decays = np.exp(-plain.softplus(-(f32(z) + f32(bias))) / tau)
    scale = 0.3
    want, want_state = np.zeros((t, vw)), f32(spans.state)
    for s, slot in enumerate(spans.slots):
        part = slice(spans.begin[s], spans.begin[s + 1])
        for h in range(heads):
            at, a, b = slice(h * dim * vdim, (h + 1) * dim * vdim), slice(h * dim, (h + 1) * dim), slice(h * vdim, (h + 1) * vdim)
            want[part, b], after = walk(want_state[slot, at].reshape(dim, vdim), f32(key[part, a]), f32(v[part, b]),
                                        decays[part, a], scale * f32(q[part, a]))
            want_state[slot, at] = after.reshape(-1)
    chunks = t // k.chunk_tokens() + spans.spans + 2
    plan = torch.zeros(chunks + spans.spans + 2, dtype=torch.int32, device=DEVICE)
    buffers = [torch.zeros(size, dtype=torch.float32, device=DEVICE) for size in
               ((t, qk), (t, qk), chunks * qk, chunks * heads * 4096, chunks * elements, (t, vw))]
    state = gpu(spans.state)
    k.chunk_plan(spans.dev["span_begin"], spans.spans, chunks, plan)
    k.channel_decay_scan(gpu(q), gpu(key), gpu(v), gpu(z), gpu(bias), tau, scale, *buffers, state, spans.state.shape[1],
                         spans.dev["span_slot"], plan, chunks, spans.spans, t // k.chunk_tokens() + spans.spans, heads, dim, vdim)
    close(buffers[-1], want, 3e-6, "read-outs of the scan")
    close(state, want_state, 3e-6, "states after the scan")
    if max(lengths) > 1:
        return
    # decoding: the decay through its two products, the heads' norm and the gate
    rank = 8
    low, up = rng.normal(size=(t, rank)).astype(np.float32), rng.normal(size=(qk, rank)) / 3.0
    norm, gate = rng.normal(1.0, 0.2, size=vdim).astype(np.float32), rng.normal(size=(t, vw)).astype(np.float32)
    for dtype, rel in DTYPES:
        up_r = rounded(up, dtype)
        decays = np.exp(-plain.softplus(-(f32(low) @ up_r.T + f32(bias))) / tau)
        want, want_state = np.zeros((t, vw)), f32(spans.state)
        for s, slot in enumerate(spans.slots):
            for h in range(heads):
                at, a, b = slice(h * dim * vdim, (h + 1) * dim * vdim), slice(h * dim, (h + 1) * dim), slice(h * vdim, (h + 1) * vdim)
                read, after = walk(want_state[slot, at].reshape(dim, vdim), f32(key[s:s + 1, a]), f32(v[s:s + 1, b]),
                                   decays[s:s + 1, a], scale * f32(q[s:s + 1, a]))
                want_state[slot, at] = after.reshape(-1)
                want[s, b] = plain.rms_scaled(read[0], 1e-5) * norm * plain.silu(f32(gate[s, b]))
        state = gpu(spans.state)
        out = torch.zeros((t, vw), dtype=dtype, device=DEVICE)
        k.channel_decay_decode(gpu(q), gpu(key), gpu(v), scale, gpu(low), gpu(up_r, dtype), gpu(bias), tau, gpu(norm), 1e-5,
                               gpu(gate), state, spans.state.shape[1], spans.dev["span_slot"], t, heads, dim, vdim, out)
        close(out, want, max(rel, 1e-5), "the decoding step's output")
        close(state, want_state, 3e-6, "states after the decoding step")


@pytest.mark.parametrize("lengths", LENGTHS)
@pytest.mark.parametrize("heads,groups,dim,vdim", [(4, 2, 8, 4), (3, 1, 5, 7), (4, 4, 64, 64), (6, 2, 130, 72), (8, 1, 16, 33)])
@pytest.mark.parametrize("forgets", [False, True])
def test_the_scan_and_the_decoding_step_with_a_decay_a_token(heads, groups, dim, vdim, lengths, forgets):
    k = kernels()
    rng = np.random.default_rng(dim + 7 * len(lengths))
    elements = heads * dim * vdim
    spans = Spans(lengths, (elements + 3) // 4 * 4 + 4, 6)
    t, qk, vw = spans.tokens, groups * dim, heads * vdim
    rows = rng.normal(size=(t, 2 * qk + vw + heads + 3)).astype(np.float32)
    dt_bias, a_log = rng.uniform(-4.0, 2.0, size=heads).astype(np.float32), rng.uniform(-3.0, 2.5, size=heads).astype(np.float32)
    direct = rng.normal(size=heads).astype(np.float32)
    if forgets:
        # tokens whose step is so long that nothing before them is left, among tokens that keep almost everything: the
        # running sums are large beside the differences that the later tokens need
        a_log[:] = rng.uniform(-1.0, 2.0, size=heads)
        dt_bias[:] = -6.0
        rows[1::29, 2 * qk + vw:2 * qk + vw + heads] = 3000.0
        rows[1::29, vw:vw + qk] = 0.0                        # (and they write nothing)
        direct[:] = 0.0
    v, key, q, raw = (f32(rows[:, a:b]) for a, b in ((0, vw), (vw, vw + qk), (vw + qk, vw + 2 * qk), (vw + 2 * qk, vw + 2 * qk + heads)))
    step = plain.softplus(raw + f32(dt_bias))
    decays = np.exp(-np.exp(f32(a_log)) * step)
    want, want_state = np.zeros((t, vw)), f32(spans.state)
    for s, slot in enumerate(spans.slots):
        part = slice(spans.begin[s], spans.begin[s + 1])
        for h in range(heads):
            g = h // (heads // groups)
            at, a, b = slice(h * dim * vdim, (h + 1) * dim * vdim), slice(g * dim, (g + 1) * dim), slice(h * vdim, (h + 1) * vdim)
            read, after = walk(want_state[slot, at].reshape(dim, vdim), step[part, h, None] * key[part, a], v[part, b],
                               decays[part, h], q[part, a])
            want[part, b] = read + float(direct[h]) * v[part, b]
            want_state[slot, at] = after.reshape(-1)
    dev = gpu(rows)
    views = [dev[:, a:b] for a, b in ((vw + qk, vw + 2 * qk), (vw, vw + qk), (0, vw), (vw + 2 * qk, vw + 2 * qk + heads))]
    chunks = t // k.chunk_tokens() + spans.spans + 1
    plan = torch.zeros(chunks + spans.spans + 2, dtype=torch.int32, device=DEVICE)
    buffers = [torch.zeros(size, dtype=torch.float32, device=DEVICE) for size in
               ((t, 2 * heads), (t, heads), chunks * groups * 4096, chunks * elements, (t, vw))]
    state = gpu(spans.state)
    k.chunk_plan(spans.dev["span_begin"], spans.spans, chunks, plan)
    k.scalar_decay_scan(*views, gpu(dt_bias), gpu(a_log), gpu(direct), *buffers, state, spans.state.shape[1], spans.dev["span_slot"],
                        plan, chunks, spans.spans, chunks - 1, heads, groups, dim, vdim)
    close(buffers[-1], want, 1e-5, "read-outs of the scan")
    if forgets:                                              # every token by its own measure
        size = np.abs(want).max(1, keepdims=True) + 1e-4
        close(buffers[-1] / gpu(size), want / size, 3e-5, "read-outs of the scan, token by token")
    close(state, want_state, 4e-6, "states after the scan")
    if max(lengths) == 1:
        state, out = gpu(spans.state), torch.zeros((t, vw), dtype=torch.float32, device=DEVICE)
        k.scalar_decay_decode(*views, gpu(dt_bias), gpu(a_log), gpu(direct), state, spans.state.shape[1], spans.dev["span_slot"], t,
                              heads, groups, dim, vdim, out)
        close(out, want, 4e-6, "read-outs of the decoding step")
        close(state, want_state, 4e-6, "states after the decoding step")


@pytest.mark.parametrize("dtype,rel", DTYPES)
@pytest.mark.parametrize("tokens,units,size", [(5, 3, 7), (9, 4, 64), (3, 2, 600), (2100, 1, 256), (1100, 2, 512), (2048, 1, 1024), (2050, 2, 130)])
def test_norms_before_and_behind_a_gate(tokens, units, size, dtype, rel):
    k = kernels()
    rng = np.random.default_rng(size)
    o, gate = f32(rng.normal(size=(tokens, units * size))), f32(rng.normal(size=(tokens, units * size + 4)))
    weight = f32(rng.normal(1.0, 0.2, size=units * size))
    z = gate[:, :units * size]
    for kind, act in ((k.GATE_SIGMOID, plain.sigmoid), (k.GATE_SILU, plain.silu)):
        for before in (0, k.GATE_BEFORE_NORM):
            x = o * act(z) if before else o
            want = plain.rms_scaled(x.reshape(tokens, units, size), 1e-5).reshape(tokens, -1) * weight * (1.0 if before else act(z))
            out = torch.zeros((tokens, units * size), dtype=dtype, device=DEVICE)
            k.gated_head_norm(gpu(o), gpu(gate)[:, :units * size], gpu(weight), True, out, tokens, units, size, 1e-5, kind + before)
            close(out, want, rel, f"gate {kind} + {before}")


# --------------------------------------------------------------------------------------------- capped scores
@pytest.mark.parametrize("kind", KERNELS)
@pytest.mark.parametrize("cap", [0.8, 5.0, 50.0])
@pytest.mark.parametrize("heads,groups,dim,window", [(4, 2, 64, None), (2, 1, 64, 70), (8, 1, 128, None), (3, 3, 24, 33)])
def test_capped_scores_in_every_attention_kernel(kind, cap, heads, groups, dim, window):
    """Scores far below, around and far beyond the cap (the series of tanh and its quotient in the tcgen05 kernel)."""
    if kind == "tcgen05" and dim != 64:
        pytest.skip("the tcgen05 kernel takes heads of 64")
    rng = np.random.default_rng(dim + heads)
    spans = [(450, 1), (0, 1), (129, 1), (63, 1)] if kind == "decode" else [(0, 200), (310, 3), (100, 129), (5, 1)]
    tokens = sum(new for _, new in spans)
    queries = bf16_round(rng.normal(size=(tokens, heads, dim)))
    keys = [bf16_round(rng.normal(size=(before + new, groups, dim))) for before, new in spans]
    values = [bf16_round(rng.normal(size=(before + new, groups, dim))) for before, new in spans]
    scale = 4.0 / math.sqrt(dim)
    want, without, t = [], [], 0
    for s, (before, new) in enumerate(spans):
        for pos in range(before, before + new):
            first = plain.visible_from(pos, window)
            for found, limit in ((want, cap), (without, None)):
                found.append(np.stack([plain.softmax(plain.capped(keys[s][first:pos + 1, h // (heads // groups)] @ queries[t, h] * scale, limit))
                                       @ values[s][first:pos + 1, h // (heads // groups)] for h in range(heads)]))
            t += 1
    want, without = np.stack(want), np.stack(without)
    assert np.abs(want - without).max() > (0.02 if cap > 10 else 0.2)
    for dtype, rel in ((torch.float32, 2e-5), (torch.bfloat16, 1e-2)):
        if dtype == torch.float32 and kind != "generic":
            continue
        paged = Paged(spans, groups, dim, dim, 16, dtype, 2)
        paged.fill(keys, values)
        got = run_attention(kind, paged, queries, heads, groups, dim, scale, window, None, None, dtype, softcap=cap)
        close(torch.as_tensor(got), want, rel, f"{kind} attention capped at {cap}")


@pytest.mark.parametrize("kind", KERNELS)
def test_small_scores_under_a_high_cap_take_the_series(kind):
    rng = np.random.default_rng(5)
    heads, groups, dim, scale, cap = 2, 2, 64, 0.02, 1.0
    spans = [(200, 1), (64, 1)] if kind == "decode" else [(0, 140), (70, 65)]
    tokens = sum(new for _, new in spans)
    queries = bf16_round(rng.normal(size=(tokens, heads, dim)))
    keys = [bf16_round(rng.normal(size=(before + new, groups, dim))) for before, new in spans]
    values = [bf16_round(rng.normal(size=(before + new, groups, dim))) for before, new in spans]
    want, t = [], 0
    for s, (before, new) in enumerate(spans):
        for pos in range(before, before + new):
            want.append(np.stack([plain.softmax(plain.capped(keys[s][:pos + 1, h] @ queries[t, h] * scale, cap)) @ values[s][:pos + 1, h]
                                  for h in range(heads)]))
            t += 1
    dtype = torch.float32 if kind == "generic" else torch.bfloat16
    paged = Paged(spans, groups, dim, dim, 16, dtype, 4)
    paged.fill(keys, values)
    got = run_attention(kind, paged, queries, heads, groups, dim, scale, None, None, None, dtype, softcap=cap)
    close(torch.as_tensor(got), np.stack(want), 1e-5 if dtype == torch.float32 else 1e-2, kind)


# ---------------------------------------------------------------------------------------------- clamped gates
@pytest.mark.parametrize("rows,width,inner", [(1, 64, 40), (8, 256, 512), (16, 128, 72), (300, 256, 384), (700, 512, 1024)])
def test_clamped_gates_in_the_gated_products(rows, width, inner):
    k = kernels()
    rng = np.random.default_rng(rows + inner)
    limit, slope, shift = 0.9, 1.7, 1.0
    x, w = bf16_round(rng.normal(size=(rows, width))), bf16_round(1.5 * rng.normal(size=(2 * inner, width)) / math.sqrt(width))
    g, u = np.minimum(x @ w[:inner].T, limit), np.clip(x @ w[inner:].T, -limit, limit)
    want = g * plain.sigmoid(slope * g) * (u + shift)
    dev, weight = gpu(x, torch.bfloat16), gpu(w, torch.bfloat16)
    flag = torch.zeros(1, dtype=torch.int32, device=DEVICE)
    out = torch.zeros((rows, inner), dtype=torch.bfloat16, device=DEVICE)
    if rows <= 16:
        k.gemv_bf16(dev, weight, out, rows, k.GEMV_SWIGLU, taps=1 + k.GATE_CLAMPED_SILU, gate_constants=(limit, slope, shift))
        close(out, want, 1e-2, "the weight-streaming product")
    for variant in (-1, 0, 1, 2, 3):
        out.zero_()
        k.gemm_tcgen05(dev, weight, out, rows, k.TC_GATED + k.GATE_CLAMPED_SILU, flag, variant, (limit, slope, shift))
        close(out, want, 1e-2, f"the tcgen05 product, variant {variant}")
    assert int(flag.item()) == 0
    # a product with another function after it is not touched by the constants
    if rows <= 16:
        k.gemv_bf16(dev, weight, out, rows, k.GEMV_SWIGLU)
        close(out, plain.silu(x @ w[:inner].T) * (x @ w[inner:].T), 1e-2, "SiLU as before")
