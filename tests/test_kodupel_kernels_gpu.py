"""The kernels that the Kodupel design added or widened, each against the same operation written in numpy (float64): the
step between two sublayers that norms an output and adds it (one row or a weighted sum of rows, bias, copy, prepared norm),
the embedding's copy, the generalised delta rule's chunked scan and decoding step, the preparation of q, k and v with
norms per head, pairs of neighbours and unit values, a gate per head, sigmoid router scores, clamped gated experts in all
their forms, and low scores beside the one in the denominator in all four attention kernels."""
from __future__ import annotations

import math

import numpy as np
import pytest
import torch

import plain_kodupel as plain
from test_liverax_kernels_gpu import KERNELS, Paged, bf16_round, close, gpu, kernels, plain_attention, run_attention

pytestmark = pytest.mark.gpu

DEVICE = "cuda:0"
DTYPES = [(torch.float32, 4e-6), (torch.bfloat16, 6e-3)]


def rounded(array, dtype):
    return bf16_round(array) if dtype == torch.bfloat16 else np.asarray(array, dtype=np.float32).astype(np.float64)


# -------------------------------------------------------------------------------------- between two sublayers
@pytest.mark.parametrize("dtype,rel", DTYPES)
@pytest.mark.parametrize("rows_type", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("tokens,width,top", [(5, 36, 0), (3, 64, 0), (7, 515, 3), (70, 2048, 0), (9, 2048, 4), (2, 9000, 2), (3, 20000, 0),
                                              (100, 1024, 8)])
def test_a_sublayers_output_is_normed_and_added(tokens, width, top, rows_type, dtype, rel):
    k = kernels()
    rng = np.random.default_rng(width + top)
    eps = 1e-5
    x = rng.normal(2.0, 3.0, size=(tokens, width)).astype(np.float32).astype(np.float64)
    weight, bias = (1.0 + 0.2 * rng.normal(size=width)).astype(np.float32), rng.normal(size=width).astype(np.float32)
    count = tokens * max(top, 1)
    rows = rounded(rng.normal(size=(count, width)), rows_type)
    place = rng.permutation(count).astype(np.int32)
    weights = rng.random(size=count).astype(np.float32)
    for with_bias, with_place in ((False, False), (True, top > 0)):
        if top == 0:
            y = rows.copy()
        else:
            at = place if with_place else np.arange(count)
            y = (weights.astype(np.float64)[:, None] * rows[at]).reshape(tokens, top, width).sum(1)
        if with_bias:
            y = y + bias
        want = x + y / np.sqrt((y ** 2).mean(-1, keepdims=True) + eps) * weight
        stream = gpu(x)
        out = torch.zeros((tokens, width), dtype=dtype, device=DEVICE)
        args = {}
        if top:
            args = {"weights": gpu(weights), "top": top, "place": gpu(place, torch.int32) if with_place else None}
        k.output_norm(stream, tokens, gpu(rows, rows_type), gpu(weight), eps, out, bias=gpu(bias) if with_bias else None, **args)
        close(stream, want, 3e-6, "the stream")
        close(out, want, rel, "the copy")
        if dtype == torch.bfloat16 and width <= 9000:
            following = gpu(1.0 + 0.1 * rng.normal(size=width))
            split = k.SplitNorm(torch.zeros((tokens, width), dtype=dtype, device=DEVICE),
                                torch.zeros((tokens, 3), dtype=torch.float32, device=DEVICE), 1, eps, width)
            stream = gpu(x)
            k.output_norm(stream, tokens, gpu(rows, rows_type), gpu(weight), eps, None, bias=gpu(bias) if with_bias else None,
                          prepare=split, next_weight=following, **args)
            close(split.xw, want * following.cpu().numpy(), rel, "the prepared rows")
            close(split.sumsq[:, 0], (want ** 2).sum(-1), 1e-5, "the prepared sums")
            assert not split.sumsq[:, 1:].any()


def test_the_copy_alone_and_the_embeddings_copy():
    k = kernels()
    rng = np.random.default_rng(3)
    for width in (30, 64):
        stream = gpu(rng.normal(size=(6, width)))
        out = torch.zeros((6, width), dtype=torch.bfloat16, device=DEVICE)
        before = stream.clone()
        k.output_norm(stream, 6, None, None, 0.0, out)
        assert torch.equal(out, before.to(torch.bfloat16)) and torch.equal(stream, before)
        table = gpu(rng.normal(size=(11, width)), torch.bfloat16)
        tokens = gpu([3, 0, 10, 3], torch.int32)
        rows = torch.zeros((5, width), dtype=torch.float32, device=DEVICE)
        copy = torch.full((5, width), 9.0, dtype=torch.bfloat16, device=DEVICE)
        k.embedding(table, tokens, rows, 2.5, copy=copy)
        assert torch.equal(rows[:4], table[tokens.long()].float() * 2.5)
        assert torch.equal(copy[:4], rows[:4].to(torch.bfloat16)) and torch.all(copy[4] == 9.0)


# ------------------------------------------------------------------------------------- generalised delta rule
class DeltaCase:
    """Rows of a fused projection for spans of the given lengths, states in slots, and what numpy makes of them."""

    def __init__(self, heads, dim, rank, lengths, seed, slow=False):
        rng = np.random.default_rng(seed)
        self.heads, self.dim, self.rank, self.lengths = heads, dim, rank, lengths
        self.tokens, inner = sum(lengths), heads * dim
        self.proj = rng.normal(size=(self.tokens, 5 * inner + rank)).astype(np.float32)
        self.offsets = (0, inner, 2 * inner, 3 * inner, 4 * inner, 5 * inner)      # r, k, v, gate, removal, low
        self.up = bf16_round(rng.normal(size=(inner, rank)) / math.sqrt(rank))
        self.w0 = (rng.uniform(-12.0, -8.0, size=inner) if slow else rng.uniform(-6.0, 3.0, size=inner)).astype(np.float32)
        self.a_bias, self.norm = rng.normal(size=inner).astype(np.float32), rng.normal(1.0, 0.2, size=inner).astype(np.float32)
        self.slots = (np.arange(len(lengths)) * 2 + 1)[::-1].astype(np.int32).copy()
        self.elements = heads * dim * dim
        self.stride = (self.elements + 3) // 4 * 4 + 8
        self.state = rng.normal(size=(2 * len(lengths) + 1, self.stride)).astype(np.float32)
        self.begin = np.concatenate([[0], np.cumsum(lengths)]).astype(np.int32)

    def cut(self, n):
        inner = self.heads * self.dim
        return self.proj[:, self.offsets[n]:self.offsets[n] + inner].astype(np.float64)

    def expected(self, low):
        """(raw read-outs [tokens, inner], states after the step) with the decay's product over ``low``."""
        r, k, v, a = (self.cut(n) for n in (0, 1, 2, 4))
        w = np.exp(-math.exp(-0.5) * plain.sigmoid(low @ self.up.T + self.w0))
        a = plain.sigmoid(a + self.a_bias)
        read, state = np.zeros_like(r), self.state.astype(np.float64)
        for s, slot in enumerate(self.slots):
            for h in range(self.heads):
                cut = slice(h * self.dim, (h + 1) * self.dim)
                place = slice(h * self.dim ** 2, (h + 1) * self.dim ** 2)
                S = state[slot, place].reshape(self.dim, self.dim)
                for t in range(self.begin[s], self.begin[s + 1]):
                    u = k[t, cut] / math.sqrt(float(k[t, cut] @ k[t, cut]) + 1e-6)
                    S = w[t, cut][:, None] * S - np.outer(a[t, cut] * u, u @ S) + np.outer(k[t, cut], v[t, cut])
                    read[t, cut] = S.T @ r[t, cut]
                state[slot, place] = S.reshape(-1)
        return read, state


@pytest.mark.parametrize("heads,dim,lengths,slow", [
    (2, 4, [5], False), (3, 8, [8, 1, 16], False), (2, 7, [9, 3], False), (1, 16, [1, 1, 1, 23], False), (2, 20, [7, 40], False),
    (5, 32, [15], True), (3, 64, [70, 2, 8], False), (2, 64, [129], True), (2, 72, [17, 6], False), (2, 128, [30, 11], False),
    (1, 136, [26], False), (1, 256, [19, 4], False)])
def test_delta_scan_over_spans_of_all_lengths(heads, dim, lengths, slow):
    k = kernels()
    case = DeltaCase(heads, dim, 8, lengths, 100 * dim + heads, slow)
    inner, tokens = heads * dim, case.tokens
    low = np.tanh(case.proj[:, case.offsets[5]:].astype(np.float64))
    want, want_state = case.expected(low)
    z = gpu(low @ case.up.T)
    flag = torch.zeros(1, dtype=torch.int32, device=DEVICE)
    state = gpu(case.state)
    read = torch.full((tokens, inner), 7.0, dtype=torch.float32, device=DEVICE)
    spans = np.repeat(np.arange(len(lengths)), lengths)
    filled = lambda n: torch.full((n,), float("nan"), dtype=torch.float32, device=DEVICE)
    k.general_delta_scan(gpu(case.proj), (case.offsets[0], case.offsets[1], case.offsets[2], case.offsets[4]), z, gpu(case.w0),
                         gpu(case.a_bias), 1e-6, gpu(spans, torch.int32), gpu(case.begin, torch.int32),
                         gpu(case.slots, torch.int32), filled(tokens * k.general_delta_scratch(heads, dim)), read, state,
                         case.stride, tokens, len(lengths), heads, dim, flag)
    assert int(flag.item()) == 0
    close(read, want, 3e-5, "read-outs")
    close(state, want_state, 3e-5, "states")
    untouched = np.setdiff1d(np.arange(case.state.shape[0]), case.slots)
    assert torch.equal(state[untouched.tolist()], gpu(case.state[untouched]))
    assert torch.equal(state[:, case.elements:], gpu(case.state[:, case.elements:]))


@pytest.mark.parametrize("dtype,rel", [(torch.float32, 1e-5), (torch.bfloat16, 8e-3)])
@pytest.mark.parametrize("heads,dim,rank,tokens", [(2, 4, 3, 1), (3, 20, 8, 5), (4, 64, 40, 8), (2, 72, 96, 3), (1, 128, 1, 2), (2, 256, 16, 2)])
def test_delta_decoding_step(heads, dim, rank, tokens, dtype, rel):
    k = kernels()
    case = DeltaCase(heads, dim, rank, [1] * tokens, 7 * dim + rank)
    low = np.tanh(case.proj[:, case.offsets[5]:].astype(np.float64))
    read, want_state = case.expected(low)
    eps = 1e-5
    normed = plain.rms_scaled(read.reshape(tokens, heads, dim), eps).reshape(tokens, heads * dim) * case.norm
    want = normed * plain.sigmoid(case.cut(3))
    state, out = gpu(case.state), torch.zeros((tokens, heads * dim), dtype=dtype, device=DEVICE)
    k.general_delta_decode(gpu(case.proj), case.offsets, gpu(case.up, dtype), gpu(case.w0), gpu(case.a_bias), gpu(case.norm), eps,
                           1e-6, state, case.stride, gpu(case.slots, torch.int32), tokens, heads, dim, out)
    close(out, want, rel, "results")
    close(state, want_state, 1e-5, "states")


def test_activation_of_columns_of_wider_rows():
    k = kernels()
    x = gpu(np.random.default_rng(5).normal(size=(9, 40)) * 3.0)
    for dtype, rel in DTYPES:
        out = torch.zeros((9, 12), dtype=dtype, device=DEVICE)
        k.activation_cast(x[:, 17:29], out, 9, k.ACT_TANH)
        close(out, np.tanh(x[:, 17:29].cpu().double().numpy()), rel, "tanh")


# ---------------------------------------------------------------------------------- preparation, gates, scores
@pytest.mark.parametrize("dtype,rel", [(torch.float32, 4e-6), (torch.bfloat16, 6e-3)])
@pytest.mark.parametrize("heads,groups,dim,vdim,key_store,value_store,rotary,own", [
    (4, 2, 16, 16, 16, 16, 8, True), (3, 1, 12, 7, 12, 7, 12, True), (8, 2, 64, 32, 64, 64, 64, True), (5, 5, 6, 6, 8, 8, 2, True),
    (16, 4, 64, 64, 64, 64, 32, True), (4, 2, 16, 16, 16, 16, 8, False), (7, 1, 10, 10, 16, 16, 6, False), (2, 2, 20, 20, 20, 20, 0, True)])
def test_preparation_with_norms_per_head_neighbours_and_unit_values(heads, groups, dim, vdim, key_store, value_store, rotary, own, dtype, rel):
    k = kernels()
    rng = np.random.default_rng(heads * 100 + dim)
    spans = [(0, 5), (37, 1), (1000, 9)]
    paged = Paged(spans, groups, key_store, value_store, 16, dtype, 1)
    tokens = paged.tokens
    qw, kw, vw = heads * dim, groups * dim if own else 0, groups * vdim if own else 0
    proj, bias = rng.normal(size=(tokens, qw + kw + vw + 3)), rng.normal(size=qw + kw + vw)
    q_norm, k_norm = rng.normal(1.0, 0.3, size=dim), rng.normal(1.0, 0.3, size=dim)
    frequencies = (50.0 ** (-2.0 * np.arange(rotary // 2) / max(rotary, 1))).astype(np.float32)
    magnitude, eps = 1.17, 1e-5
    positions, token_span, _, table = paged.device()
    q_out = torch.zeros((tokens, heads * key_store), dtype=dtype, device=DEVICE)
    k.qkv_prepare(gpu(proj), gpu(bias), q_out, positions, token_span, table, paged.k if own else None, paged.v if own else None,
                  tokens, heads, groups if own else 0, dim, vdim, key_store, value_store, 16, paged.flag, q_norm=gpu(q_norm),
                  k_norm=gpu(k_norm) if own else None, norm_eps=eps, norm_per_head=True, unit_values_eps=eps if own else None,
                  frequencies=gpu(frequencies) if rotary else None, rotary_dim=rotary, interleaved=True, magnitude=magnitude)
    assert int(paged.flag.item()) == 0
    x = proj.astype(np.float32).astype(np.float64)[:, :qw + kw + vw] + bias.astype(np.float32)

    def turned(rows):
        rows = rows.copy()
        angles = paged.positions[:, None].astype(np.float64) * frequencies[None, :].astype(np.float64)
        c, s = np.cos(angles)[:, None] * magnitude, np.sin(angles)[:, None] * magnitude
        a, b = rows[..., 0:rotary:2].copy(), rows[..., 1:rotary:2].copy()
        rows[..., 0:rotary:2], rows[..., 1:rotary:2] = a * c - b * s, b * c + a * s
        return rows
    scale = 60.0 * rel if dtype == torch.float32 else rel              # (a float32 angle of a thousand turns)
    q = turned(plain.rms_scaled(x[:, :qw].reshape(tokens, heads, dim), eps) * q_norm)
    got = q_out.float().cpu().numpy().reshape(tokens, heads, key_store)
    close(torch.as_tensor(got[..., :dim]), q, scale, "queries")
    assert not got[..., dim:].any()
    if not own:
        assert not paged.k.any() and not paged.v.any()
        return
    kk = turned(plain.rms_scaled(x[:, qw:qw + kw].reshape(tokens, groups, dim), eps) * k_norm)
    v = plain.rms_scaled(x[:, qw + kw:].reshape(tokens, groups, vdim), eps)
    for t in range(tokens):
        s, pos = int(paged.token_span[t]), int(paged.positions[t])
        stored_k, stored_v = paged.read(paged.k, s, pos), paged.read(paged.v, s, pos)
        close(torch.as_tensor(stored_k[:, :dim]), kk[t], scale, f"the key of token {t}")
        close(torch.as_tensor(stored_v[:, :vdim]), v[t], rel, f"the value of token {t}")
        assert not stored_k[:, dim:].any() and not stored_v[:, vdim:].any()


@pytest.mark.parametrize("dtype,rel", DTYPES)
@pytest.mark.parametrize("heads,size", [(3, 7), (4, 64), (5, 12), (1, 130)])
def test_a_gate_per_head(heads, size, dtype, rel):
    k = kernels()
    rng = np.random.default_rng(size)
    values, gate = rounded(rng.normal(size=(11, heads * size)), dtype), rng.normal(size=(11, heads + 5)).astype(np.float32) * 2.0
    held = gpu(values, dtype)
    k.sigmoid_gate(held, gpu(gate)[:, 3:3 + heads], 11, heads * size, per=size)
    want = values.reshape(11, heads, size) * plain.sigmoid(gate[:, 3:3 + heads].astype(np.float64))[:, :, None]
    close(held, want.reshape(11, -1), rel, "gated")


@pytest.mark.parametrize("kind", KERNELS)
@pytest.mark.parametrize("level", [0.0, -8.0])
def test_a_one_in_the_denominator_in_every_attention_kernel(kind, level):
    """Scores around 0 and around -8 (the weights then sum to almost nothing) beside a sink of score zero."""
    heads, groups, dim, scale = 8, 2, 64, 0.125
    spans = [(300, 1), (17, 1)] if kind == "decode" else [(0, 40), (130, 150), (16, 2)]
    rng = np.random.default_rng(31)
    tokens = sum(new for _, new in spans)
    c = 8.0 ** 0.5 if level else 0.0
    queries = bf16_round(0.5 * rng.normal(size=(tokens, heads, dim)) - c)
    keys = [bf16_round(0.5 * rng.normal(size=(before + new, groups, dim)) + c * -level / 64.0) for before, new in spans]
    values = [bf16_round(rng.normal(size=(before + new, groups, dim))) for before, new in spans]
    dtype = torch.bfloat16
    paged = Paged(spans, groups, dim, dim, 16, dtype, 5)
    paged.fill(keys, values)
    sinks = np.zeros(heads)
    want = plain_attention(queries, keys, values, spans, scale, None, None, sinks)
    got = run_attention(kind, paged, queries, heads, groups, dim, scale, None, None, sinks, dtype)
    without = plain_attention(queries, keys, values, spans, scale, None, None, None)
    close(torch.as_tensor(got), want, 2e-2, kind)
    if level:
        assert np.abs(without).max() > 1.2 * np.abs(want).max()


# ------------------------------------------------------------------------------------------- mixture of experts
@pytest.mark.parametrize("experts,top,tokens", [(4, 1, 9), (16, 3, 70), (40, 8, 33), (70, 70, 5)])
@pytest.mark.parametrize("renormalize", [False, True])
def test_router_with_sigmoid_scores(experts, top, tokens, renormalize):
    k = kernels()
    rng = np.random.default_rng(experts)
    logits, correction = rng.normal(size=(tokens, experts)).astype(np.float32) * 2.0, rng.normal(size=experts).astype(np.float32) * 0.5
    chosen = torch.zeros((tokens, top), dtype=torch.int32, device=DEVICE)
    weights = torch.zeros((tokens, top), dtype=torch.float32, device=DEVICE)
    k.moe_route(gpu(logits), experts, gpu(correction), None, chosen, weights, None, tokens, top, sigmoid_scores=True, renormalize=renormalize)
    scores = plain.sigmoid(logits.astype(np.float64))
    want = np.argsort(-(scores + correction), axis=-1, kind="stable")[:, :top]
    picked = np.take_along_axis(scores, want, axis=-1)
    if renormalize:
        picked = picked / picked.sum(-1, keepdims=True)
    assert np.array_equal(chosen.cpu().numpy(), want)
    close(weights, picked, 2e-6, "weights")


@pytest.mark.parametrize("dtype,rel", [(torch.float32, 4e-6), (torch.bfloat16, 1.5e-2)])
@pytest.mark.parametrize("form", ["clamped", "silu"])
@pytest.mark.parametrize("experts,top,width,inner,tokens", [(4, 2, 40, 24, 7), (16, 3, 256, 96, 200), (5, 5, 36, 20, 70), (40, 1, 64, 72, 130),
                                                             (3, 2, 104, 40, 90), (8, 2, 512, 384, 700), (32, 4, 512, 768, 2048), (6, 2, 128, 200, 300)])
def test_gated_experts_grouped_and_row_by_row(experts, top, width, inner, tokens, form, dtype, rel):
    """The forms of gated experts' first product (rows, tiles and an element-wise kernel, tcgen05 with the gate in its
    epilogue) against numpy."""
    k = kernels()
    rng = np.random.default_rng(inner)
    limit, slope, shift = 1.3, 1.7, 0.75
    h = rounded(rng.normal(size=(tokens, width)), dtype)
    gate, up = (rounded(1.5 * rng.normal(size=(experts, inner, width)) / np.sqrt(width), dtype) for _ in range(2))
    chosen_np = np.stack([rng.permutation(experts)[:top] for _ in range(tokens)]).astype(np.int32)
    if top == 1:
        chosen_np[rng.random(tokens) < 0.6] = 3                       # one expert far busier than the rest
    flat = chosen_np.reshape(-1)
    g, u = np.zeros((tokens * top, inner)), np.zeros((tokens * top, inner))
    for e in range(experts):
        at = np.nonzero(flat == e)[0]
        g[at], u[at] = h[at // top] @ gate[e].T, h[at // top] @ up[e].T
    if form == "clamped":
        g, u = np.minimum(g, limit), np.clip(u, -limit, limit)
        want, code, constants = g * plain.sigmoid(slope * g) * (u + shift), k.GATE_CLAMPED_SILU, (limit, slope, shift)
    else:
        want, code, constants = g * plain.sigmoid(g) * u, k.ACT_SILU, k.NO_GATE_CONSTANTS
    pairs = tokens * top
    chosen, x, w = gpu(flat, torch.int32), gpu(h, dtype), gpu(np.concatenate([gate, up], axis=1), dtype)
    flag = torch.zeros(1, dtype=torch.int32, device=DEVICE)
    for kind in ("rows", "tiles", "tcgen05"):
        if kind == "rows" and pairs > 1500:
            continue
        raised = torch.full((pairs + 200, inner), 3.0, dtype=dtype, device=DEVICE)
        gathered = torch.full((pairs + 200, width), 3.0, dtype=dtype, device=DEVICE)
        if kind == "tcgen05" and not k.expert_product_tcgen05_supported(gathered, w):
            continue
        if kind == "rows":
            k.expert_rows(x, top, chosen, w, raised, pairs, code, gated=True, constants=constants)
            got = raised[:pairs]
        else:
            tile_rows = 128 if kind == "tcgen05" else k.MOE_TILE
            place, source = (torch.zeros(pairs, dtype=torch.int32, device=DEVICE) for _ in range(2))
            tiles = k.moe_max_tiles(pairs, experts, tile_rows)
            table = torch.zeros(4 + 3 * tiles, dtype=torch.int32, device=DEVICE)
            k.moe_group(chosen, tokens, experts, top, place, source, table, tile_rows=tile_rows)
            if kind == "tcgen05":
                k.moe_gather_rows(x, source, gathered, pairs)
                k.expert_product_tcgen05(gathered, w, raised, table, tiles, code, flag, gated=True, constants=constants)
                for wide in (0, 1):
                    again = torch.full_like(raised, 3.0)
                    k.expert_product_tcgen05(gathered, w, again, table, tiles, code, flag, wide_tiles=wide, gated=True, constants=constants)
                    assert torch.equal(again, raised)
                assert int(flag.item()) == 0
            else:
                paired = torch.zeros((pairs, 2 * inner), dtype=dtype, device=DEVICE)
                k.expert_product(x, source, w, paired, table, tiles, -1)
                k.glu(paired, raised, pairs, inner, code, constants)
            got = raised[place.long()]
        close(got, want, rel, kind)
        assert torch.all(raised[pairs:] == 3.0)
