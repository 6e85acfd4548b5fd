"""The Fovezen design in the engine against the plain float64 model of ``plain_fovezen.py``: whole prompts, decoding token
by token, portions down to two tokens, batches of unequal requests, pages and slots used again, keys just inside and just
outside every window and far keys at page borders with weights that make one key show, far tokens through both recurrences
and what a strong decay forgets, the convolutions across a portion's start, the connections of several streams, repeated
layers' caches of their own, the cap, the limits, and greedy generation through ``Engine`` and the command line. float32
path to 2e-4 of the logits' spread, bfloat16 path to a few percent."""
from __future__ import annotations

import numpy as np
import pytest

import fovezen_models as fm
import plain_fovezen as plain

pytestmark = pytest.mark.gpu

LIMIT = {"float32": 2e-4, "bfloat16": 1.5e-1}
TYPICAL = {"float32": 1e-4, "bfloat16": 6e-2}


def spread_error(got: np.ndarray, want: np.ndarray) -> np.ndarray:
    """Per row: rms of the difference (mean taken off) over the rms of the wanted row (mean taken off)."""
    d = got - want
    d = d - d.mean(-1, keepdims=True)
    w = want - want.mean(-1, keepdims=True)
    return np.sqrt((d ** 2).mean(-1)) / np.sqrt((w ** 2).mean(-1))


def check(got, want, dtype, what, slack=1.0):
    err = spread_error(np.asarray(got, dtype=np.float64), want)
    worst = int(np.argmax(err))
    assert err[worst] <= slack * LIMIT[dtype], f"{what}: row {worst} differs by {err[worst]:.3e} of the row's spread"
    assert np.median(err) <= slack * TYPICAL[dtype], f"{what}: half of the rows differ by {np.median(err):.3e} and more"


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    base = tmp_path_factory.mktemp("fovezen")
    out = {}
    for name, (raw, seed) in fm.CONFIGS.items():
        folder = str(base / name)
        raw, tensors = fm.write_model(folder, raw, seed)
        out[name] = (folder, raw, plain.as_float64(tensors))
    return out


def load(folder, dtype, **kw):
    from celeg_b200.engine.loading import load_model
    args = dict(dtype=dtype, max_requests=4, cache_tokens=1024, max_batched_tokens=512, max_context=512)
    args.update(kw)
    return load_model(folder, **args)


def run_steps(loaded, steps):
    """steps: lists of (request, tokens); every place is wanted. Returns {request: [its logits rows in order]}."""
    from celeg_b200.engine.step import StepEntry
    rows = {}
    for step in steps:
        step = [(name, tokens) for name, tokens in step if len(tokens) > 0]
        entries = [StepEntry(name, list(tokens), list(range(len(tokens)))) for name, tokens in step]
        logits = loaded.step.run(entries, auto_begin=True).cpu().numpy()
        loaded.step.raise_on_device_error()
        at = 0
        for name, tokens in step:
            rows.setdefault(name, []).append(logits[at:at + len(tokens)].copy())
            at += len(tokens)
    return {name: np.concatenate(parts) for name, parts in rows.items()}


def cut(tokens, sizes):
    out, at, i = [], 0, 0
    while at < len(tokens):
        n = sizes[i % len(sizes)]
        out.append(tokens[at:at + n])
        at += n
        i += 1
    return out


def tokens_of(vocab, length, seed):
    return np.random.default_rng(seed).integers(0, vocab, size=length).tolist()


# ------------------------------------------------------------------------------------------ whole models
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(fm.CONFIGS))
def test_whole_prompt_then_token_by_token(models, name, dtype):
    folder, raw, tensors = models[name]
    tokens = tokens_of(raw["vocab"], 90, 1)
    want = plain.logits(raw, tensors, tokens)
    loaded = load(folder, dtype)
    whole = run_steps(loaded, [[("w", tokens)]])["w"]
    check(whole, want, dtype, f"{name} whole")
    loaded.step.end("w")
    decoded = run_steps(loaded, [[("d", tokens[:37])]] + [[("d", [t])] for t in tokens[37:]])["d"]
    check(decoded, want, dtype, f"{name} prompt of 37 then token by token")
    if dtype == "float32":       # how the prompt is cut changes nothing beyond rounding
        assert np.abs(decoded - whole).max() <= 1e-3 * np.abs(whole).max()


@pytest.mark.parametrize("name", list(fm.CONFIGS))
def test_the_sum_of_the_streams_after_every_layer(models, name):
    """What the engine's streams add up to after every layer that runs, in a prompt and token by token."""
    import torch
    from celeg_b200.engine.step import StepEntry
    folder, raw, tensors = models[name]
    tokens = tokens_of(raw["vocab"], 40, 21)
    want = plain.streams(raw, tensors, tokens)
    loaded = load(folder, "float32")
    model, seen = loaded.model, []

    def watched(run):
        def wrapped(stream, step):
            run(stream, step)
            total = torch.empty((step.tokens, model.hidden_size), dtype=torch.float32, device="cuda:0")
            stream.copies.total(total, step.tokens)
            seen.append(total.cpu().numpy())
        return wrapped
    for layer in model.layers:
        layer.block.run = watched(layer.block.run)
    loaded.step.run([StepEntry("w", tokens, [39])], auto_begin=True)
    for t in tokens:
        loaded.step.run([StepEntry("d", [t], [0])], auto_begin=True)
    loaded.step.raise_on_device_error()
    runs = len(want)
    assert len(seen) == runs * 41
    for n in range(runs):
        for got in (seen[n], np.concatenate(seen[runs + n::runs])):
            assert np.abs(got - want[n]).max() <= 5e-5 * np.abs(want[n]).max(), f"{name} after run {n}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(fm.CONFIGS))
def test_portions_of_several_sizes_down_to_two_tokens(models, name, dtype):
    folder, raw, tensors = models[name]
    tokens = tokens_of(raw["vocab"], 131, 2)
    want = plain.logits(raw, tensors, tokens)
    loaded = load(folder, dtype)
    for tag, sizes in (("a", [2, 3, 17, 2, 33]), ("b", [16, 16, 1, 15, 48]), ("c", [5, 2, 2, 64]), ("d", [8, 7, 9])):
        got = run_steps(loaded, [[(tag, part)] for part in cut(tokens, sizes)])[tag]
        check(got, want, dtype, f"{name} in portions of {sizes}")
        loaded.step.end(tag)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(fm.CONFIGS))
def test_batches_of_unequal_requests_equal_each_alone(models, name, dtype):
    folder, raw, tensors = models[name]
    requests = {"p": tokens_of(raw["vocab"], 70, 3), "q": tokens_of(raw["vocab"], 23, 4),
                "r": tokens_of(raw["vocab"], 120, 5), "s": tokens_of(raw["vocab"], 9, 6)}
    want = {key: plain.logits(raw, tensors, value) for key, value in requests.items()}
    # portions of some beside single tokens of others; q joins late, s is left out of steps and goes on later
    plan = {"p": [40] + [1] * 30, "q": [0, 0, 2, 19, 1, 1], "r": [3, 50, 1, 1, 1, 62, 1, 1], "s": [1, 0, 0, 1, 0, 5, 2]}
    at = {key: 0 for key in requests}
    steps = []
    for n in range(40):
        step = []
        for key in ("s", "p", "q", "r"):
            sizes = plan[key]
            count = min(sizes[n] if n < len(sizes) else 1, len(requests[key]) - at[key])
            if count > 0:
                step.append((key, requests[key][at[key]:at[key] + count]))
                at[key] += count
        if step:
            steps.append(step)
    assert all(at[key] == len(requests[key]) for key in requests)
    got = run_steps(load(folder, dtype), steps)
    for key in requests:
        check(got[key], want[key], dtype, f"{name} request {key} in a batch")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_pages_and_slots_are_used_again(models, name, dtype):
    """Two slots and a pool of 160 positions for six requests one after the other, two live at a time: every later
    request sits in a slot and in pages that an earlier one has left full of its own state."""
    folder, raw, tensors = models[name]
    loaded = load(folder, dtype, max_requests=2, cache_tokens=160)
    lengths = [75, 60, 31, 80, 17, 66]
    for turn in range(3):
        pair = {f"x{2 * turn}": tokens_of(raw["vocab"], lengths[2 * turn], 20 + turn),
                f"y{2 * turn}": tokens_of(raw["vocab"], lengths[2 * turn + 1], 30 + turn)}
        (a, ta), (b, tb) = pair.items()
        got = run_steps(loaded, [[(a, ta[:20]), (b, tb[:3])], [(a, ta[20:21]), (b, tb[3:])], [(a, ta[21:])]])
        for key, tokens in pair.items():
            check(got[key], plain.logits(raw, tensors, tokens), dtype, f"turn {turn} request {key}")
            loaded.step.end(key)
        loaded.manager.check_invariants()
    assert loaded.manager.free_slots == 2


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_long_portions_beside_short_ones(models, name, dtype):
    """Portions of hundreds of tokens (the scans walk many chunks) beside single tokens
    and short portions of other requests, from states and caches that earlier portions left."""
    folder, raw, tensors = models[name]
    requests = {"a": tokens_of(raw["vocab"], 700, 31), "b": tokens_of(raw["vocab"], 140, 32), "c": tokens_of(raw["vocab"], 300, 33)}
    want = {key: plain.logits(raw, tensors, value) for key, value in requests.items()}
    a, b, c = (requests[key] for key in "abc")
    loaded = load(folder, dtype, cache_tokens=2048, max_batched_tokens=1024, max_context=1024)
    got = run_steps(loaded, [[("b", b[:1]), ("a", a[:349])], [("b", b[1:2]), ("a", a[349:350]), ("c", c[:285])],
                             [("b", b[2:131]), ("a", a[350:677]), ("c", c[285:])], [("b", b[131:]), ("a", a[677:])]])
    for key in want:
        check(got[key], want[key], dtype, f"{name} request {key} in long portions")


@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_long_decoding_from_the_first_token(models, name):
    folder, raw, tensors = models[name]
    tokens = tokens_of(raw["vocab"], 200, 7)
    got = run_steps(load(folder, "float32"), [[("l", [t])] for t in tokens])["l"]
    check(got, plain.logits(raw, tensors, tokens), "float32", "200 tokens one by one")


def test_the_first_tokens_of_a_sequence(tmp_path):
    """Prompts of one, two and three tokens and decoding from there: states and carried inputs start from zero, the first
    token's attention has its own key alone."""
    for name, (raw, seed) in fm.CONFIGS.items():
        folder = str(tmp_path / name)
        raw, bf16 = fm.write_model(folder, raw, seed)
        tokens = tokens_of(raw["vocab"], 12, 16)
        want = plain.logits(raw, plain.as_float64(bf16), tokens)
        loaded = load(folder, "float32")
        for first in (1, 2, 3):
            got = run_steps(loaded, [[("f", tokens[:first])]] + [[("f", [t])] for t in tokens[first:]])["f"]
            check(got, want, "float32", f"{name}: a prompt of {first}")
            loaded.step.end("f")


# ------------------------------------------------------------------------- one mechanism, made to show
def single_out(bf16, token, column, value=6.0):
    """Column ``column`` of the embedding table becomes zero for every token but ``token``: in a first layer that input
    dimension then speaks for this token alone."""
    import torch
    table = bf16["embed"].float().numpy().copy()
    table[:, column] = 0.0
    table[token, column] = value
    bf16["embed"] = torch.from_numpy(table).to(torch.bfloat16)


def change(bf16, name, function):
    import torch
    bf16[name] = torch.from_numpy(np.asarray(function(bf16[name].float().numpy().copy()), dtype=np.float32)).to(torch.bfloat16)


def set_column(bf16, name, rows, column, values):
    def put(matrix):
        matrix[rows, column] = values
        return matrix
    change(bf16, name, put)


def untouched_convolution(bf16, name):
    """Taps that pass the token's own input on and nothing else."""
    def last(w):
        w[:] = 0.0
        w[:, -1] = 1.0
        return w
    change(bf16, name, last)


def open_connection(bf16):
    """The first connection reads the streams with a positive weight and lets the output through in full."""
    change(bf16, "l0.hc1.in", lambda w: 0 * w + 0.5)
    change(bf16, "l0.hc1.out", lambda w: 0 * w + 2.0)


def build_far_key(kind, sizes, far, probe, length, window=None):
    """Every head's query of ONE token (through an input dimension that only this token has) points at the key that ONE
    other token makes at place ``far``, along dimensions that do not turn. Returns (raw, bf16, sequence with that token,
    sequence with another in its place)."""
    heads, groups, dim, vdim, rot_dims = sizes
    if kind == "attention":
        raw = fm.single_layer(fm.attention(heads, groups, dim, vdim, fm.rotation(1000.0, rot_dims, factor=2.0), scale=1.5 * dim ** -0.5))
        mix = "l0.mix."
    else:
        raw = fm.single_layer(fm.parallel((heads, groups, dim, vdim, 3, window, 40.0, 4.0 * dim ** -0.5), (1, 4, 4, 2.0, 2)))
        mix = "l0.mix.left."
    bf16 = fm.make_tensors(raw, 40)
    vocab, width = raw["vocab"], raw["width"]
    key_token, probe_token, other_token = vocab - 1, vocab - 2, vocab - 3
    single_out(bf16, probe_token, width - 2)
    single_out(bf16, key_token, width - 4)
    open_connection(bf16)
    changed = np.random.default_rng(8).integers(0, vocab - 3, size=length).tolist()
    changed[probe] = probe_token
    without = list(changed)
    changed[far], without[far] = key_token, other_token
    rng = np.random.default_rng(9)
    direction = np.zeros((groups, dim))
    direction[:, rot_dims:] = rng.choice([-1.0, 1.0], size=(groups, dim - rot_dims))
    set_column(bf16, mix + "k", slice(0, groups * dim), width - 4, 2.0 * direction.reshape(-1))
    set_column(bf16, mix + "v", slice(0, groups * vdim), width - 4, 2.0 * rng.normal(size=groups * vdim))
    for head in range(heads):
        set_column(bf16, mix + "q", slice(head * dim, (head + 1) * dim), width - 2, 2.0 * direction[head // (heads // groups)])
    change(bf16, mix + "q.norm", lambda w: 0 * w + 1.7)
    change(bf16, mix + "k.norm", lambda w: 0 * w + 1.2)
    if kind != "attention":
        for name in ("q", "k", "v"):
            untouched_convolution(bf16, mix + name + ".conv")
        change(bf16, "l0.mix.right.out", lambda w: 0 * w)
        change(bf16, "l0.mix.left.out", lambda w: 0 * w + 2.0)
    return raw, bf16, changed, without


def follow(tmp_path, raw, bf16, changed, without, probe, dtype, shows, start, what):
    """The plain model tells the two sequences apart at ``probe`` (``shows``) or not at all there; the engine follows it with
    the probe inside a prompt, as the first token of a portion, and decoded alone (after a prompt and after decoded tokens)."""
    folder = str(tmp_path / "one")
    fm.write_model(folder, raw, 0, tensors=bf16)
    tensors = plain.as_float64(bf16)
    want, reference = plain.logits(raw, tensors, changed), plain.logits(raw, tensors, without)
    moved = spread_error(want[probe:probe + 1], reference[probe:probe + 1])[0]
    assert moved > 0.2 if shows else moved < 1e-9, f"the plain model itself: {moved}"
    loaded = load(folder, dtype)
    for tag, steps in (("prompt", [changed]), ("portion", [changed[:probe], changed[probe:]]),
                       ("inside", [changed[:probe - 3], changed[probe - 3:probe + 2], changed[probe + 2:]]),
                       ("decoded", [changed[:probe]] + [[t] for t in changed[probe:]]),
                       ("later", [changed[:start]] + [[t] for t in changed[start:]])):
        got = run_steps(loaded, [[(tag, part)] for part in steps if len(part)])[tag]
        check(got, want, dtype, f"{what}, {tag}")
        if shows:
            assert spread_error(got[probe:probe + 1].astype(np.float64), reference[probe:probe + 1])[0] > 0.15, tag
        loaded.step.end(tag)


FAR = [((4, 2, 8, 12, 4), 0, 317), ((4, 2, 8, 12, 4), 15, 317), ((4, 2, 8, 12, 4), 16, 240), ((17, 1, 24, 8, 6), 31, 300),
       ((17, 1, 24, 8, 6), 299, 300), ((3, 3, 12, 5, 2), 255, 256), ((8, 2, 64, 64, 16), 0, 340), ((8, 2, 64, 64, 16), 127, 390),
       ((8, 2, 64, 64, 16), 128, 390), ((8, 1, 64, 128, 32), 63, 340), ((4, 4, 128, 64, 8), 64, 389), ((2, 1, 16, 16, 4), 79, 80)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("sizes,far,probe", FAR)
def test_far_keys_at_page_borders(tmp_path, sizes, far, probe, dtype):
    raw, bf16, changed, without = build_far_key("attention", sizes, far, probe, probe + 9)
    start = max(1, min(far - 5, probe - 1), probe - 90)
    follow(tmp_path, raw, bf16, changed, without, probe, dtype, True, start, f"key at {far}, probe at {probe}")


WINDOWS = [((4, 2, 8, 12, 0), 16, 40), ((4, 2, 8, 12, 0), 17, 31), ((3, 3, 12, 12, 0), 5, 90), ((17, 1, 24, 8, 0), 33, 150),
           ((8, 2, 64, 64, 0), 64, 130), ((8, 2, 64, 64, 0), 100, 27), ((8, 1, 64, 128, 0), 128, 200), ((2, 2, 128, 128, 0), 70, 64),
           ((4, 4, 64, 72, 0), 140, 60), ((2, 1, 16, 16, 0), 1, 20)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("inside", [True, False])
@pytest.mark.parametrize("sizes,window,far", WINDOWS)
def test_keys_just_inside_and_just_outside_the_window(tmp_path, sizes, window, far, inside, dtype):
    """The last position that still sees the key at ``far`` is far + window - 1; one further the two sequences are the same
    to the layer (their recurrences, convolutions and everything else but the window's softmax count for nothing here)."""
    probe = far + window - (1 if inside else 0)
    if probe == far:
        pytest.skip("a window of one shows a token itself alone")
    raw, bf16, changed, without = build_far_key("window", sizes, far, probe, probe + 7, window)
    follow(tmp_path, raw, bf16, changed, without, probe, dtype, inside, max(1, far - 3), f"window {window}, key at {far}, probe at {probe}")


def build_far_state(kind, forget):
    """One recurrent layer: ONE token writes a large value under a key of its own, ONE probe token reads along that key 250
    tokens later. With ``forget`` a token between them has decays of almost nothing."""
    if kind == "linear":
        raw = fm.single_layer(fm.parallel((1, 1, 4, 4, 2, 2, 5.0, 0.5), (2, 16, 12, 1.0, 6)))
    else:
        raw = fm.single_layer(fm.mamba(2, 12, 16, 1, 2, 1))
    bf16 = fm.make_tensors(raw, 42)
    vocab, width = raw["vocab"], raw["width"]
    key_token, probe_token, forget_token = vocab - 1, vocab - 2, vocab - 3
    for token, column in ((key_token, width - 2), (probe_token, width - 4), (forget_token, width - 6)):
        single_out(bf16, token, column)
    open_connection(bf16)
    rng = np.random.default_rng(11)
    if kind == "linear":
        at, direction = "l0.mix.right.", rng.choice([-1.0, 1.0], size=32)
        for name in ("k", "v", "q"):
            change(bf16, at + name, lambda w: 0.15 * w)
        change(bf16, at + "a1", lambda w: 0 * w)
        change(bf16, at + "a2.b", lambda b: 0 * b + 12.0)                  # (decays of almost one)
        change(bf16, at + "a2", lambda w: 0 * w - 20.0)
        set_column(bf16, at + "a1", slice(0, 6), width - 6, 1.0)
        set_column(bf16, at + "k", slice(0, 32), width - 2, 0.5 * direction)
        set_column(bf16, at + "v", slice(0, 24), width - 2, 3.0 * rng.normal(size=24))
        set_column(bf16, at + "q", slice(0, 32), width - 4, 0.5 * direction)
        change(bf16, "l0.mix.left.out", lambda w: 0 * w)
        change(bf16, "l0.mix.right.out", lambda w: 0 * w + 2.0)
    else:
        # rows of the projection: z 24, x 24, B 16, C 16, dt 2
        at, direction = "l0.mix.", (np.arange(16) % 2).astype(np.float64)
        untouched_convolution(bf16, at + "conv")
        change(bf16, at + "conv.b", lambda b: 0 * b)
        change(bf16, at + "in", lambda w: np.concatenate([w[:24], 0.15 * w[24:80], 0 * w[80:]]))
        change(bf16, at + "dt_bias", lambda b: 0 * b - 4.0)
        change(bf16, at + "A_log", lambda b: 0 * b - 2.0)
        change(bf16, at + "D", lambda b: 0 * b + 1.0)
        set_column(bf16, at + "in", slice(24, 48), width - 2, 2.0 * np.abs(rng.normal(size=24)))
        set_column(bf16, at + "in", slice(48, 64), width - 2, 2.0 * direction)
        set_column(bf16, at + "in", slice(64, 80), width - 4, 2.0 * direction)
        set_column(bf16, at + "in", slice(80, 82), width - 2, 2.0)          # (the key's token writes in full)
        set_column(bf16, at + "in", slice(80, 82), width - 6, 60.0)         # (a step so long that nothing is kept)
    changed = np.random.default_rng(10).integers(0, vocab - 3, size=256).tolist()
    changed[3] = key_token
    for place in (250, 255):
        changed[place] = probe_token
    without = list(changed)
    if forget:
        changed[100] = forget_token
    else:
        without[3] = 0
    return raw, bf16, changed, without


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("forget", [False, True])
@pytest.mark.parametrize("kind", ["linear", "mamba2"])
def test_a_far_token_and_its_loss_show_through_the_state(tmp_path, kind, forget, dtype):
    raw, bf16, changed, without = build_far_state(kind, forget)
    folder = str(tmp_path / "one")
    fm.write_model(folder, raw, 0, tensors=bf16)
    tensors = plain.as_float64(bf16)
    want, reference = plain.logits(raw, tensors, changed), plain.logits(raw, tensors, without)
    assert spread_error(want[[250, 255]], reference[[250, 255]]).min() > 0.2, "the plain model itself"
    loaded = load(folder, dtype)
    for tag, steps in (("whole", [changed]), ("portions", cut(changed, [2, 70, 33, 16, 7])), ("at the loss", [changed[:100], changed[100:]]),
                       ("decoded", [changed[:6]] + [[t] for t in changed[6:]])):
        got = run_steps(loaded, [[(tag, part)] for part in steps])[tag]
        # (a read-out that happens to be small beside the state it is read from carries the state's rounding)
        check(got, want, dtype, f"{tag}", slack=2.0)
        assert spread_error(got[[250, 255]].astype(np.float64), reference[[250, 255]]).min() > 0.15
        loaded.step.end(tag)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("layer,names", [(fm.mamba(2, 12, 8, 2, 4, 1), ["l0.mix.conv"]), (fm.mamba(1, 20, 5, 1, 7, 2), ["l0.mix.conv"]),
                                         (fm.parallel((2, 1, 8, 12, 4, 30, 9.0, 0.5), (1, 4, 4, 2.0, 2)),
                                          ["l0.mix.left.q.conv", "l0.mix.left.k.conv", "l0.mix.left.v.conv"])])
def test_convolutions_reach_across_a_portions_start(tmp_path, layer, names, dtype):
    """Kernels whose first tap is the largest: what stood taps - 1 tokens ago speaks loudest, in whichever step it came. A
    model whose carried inputs were lost would show it (the plain model with each portion convolved alone does)."""
    raw = fm.single_layer(layer)
    bf16 = fm.make_tensors(raw, 43)
    open_connection(bf16)
    for name in names:
        def early(w):
            w *= 0.3
            w[:, 0] = np.where(w[:, 0] < 0, -1.5, 1.5)
            return w
        change(bf16, name, early)
    folder = str(tmp_path / "one")
    fm.write_model(folder, raw, 0, tensors=bf16)
    tensors = plain.as_float64(bf16)
    tokens = tokens_of(raw["vocab"], 40, 12)
    want = plain.logits(raw, tensors, tokens)
    keep = plain.causal_convolution

    def forgetful(u, taps, bias=None):
        return np.concatenate([keep(u[a:a + 5], taps, bias) for a in range(0, len(u), 5)])
    plain.causal_convolution = forgetful
    try:
        lost = plain.logits(raw, tensors, tokens)
    finally:
        plain.causal_convolution = keep
    assert np.median(spread_error(lost, want)) > 0.2
    loaded = load(folder, dtype)
    for tag, sizes in (("a", [40]), ("b", [5]), ("c", [2]), ("d", [1]), ("e", [3, 1, 1, 9, 2])):
        check(run_steps(loaded, [[(tag, part)] for part in cut(tokens, sizes)])[tag], want, dtype, f"portions of {sizes}")
        loaded.step.end(tag)


@pytest.mark.parametrize("heads,dim,vdim,tau,rank", [(1, 4, 5, 1.0, 3), (2, 8, 4, 2.0, 16), (3, 13, 30, 16.0, 1), (2, 64, 72, 8.0, 9),
                                                     (1, 130, 64, 4.0, 33), (1, 256, 8, 16.0, 8)])
def test_head_sizes_ranks_and_roots_of_gated_linear_attention(tmp_path, heads, dim, vdim, tau, rank):
    raw = fm.single_layer(fm.parallel((1, 1, 4, 4, 2, 3, 5.0, 0.5), (heads, dim, vdim, tau, rank)))
    folder = str(tmp_path / "one")
    raw, bf16 = fm.write_model(folder, raw, 44)
    tokens = tokens_of(raw["vocab"], 141, 12)
    want = plain.logits(raw, plain.as_float64(bf16), tokens)
    loaded = load(folder, "float32")
    for tag, sizes in (("a", [141]), ("b", [8, 7, 9, 1, 16]), ("c", [64, 64, 13]), ("d", [63, 1, 3, 65])):
        got = run_steps(loaded, [[(tag, part)] for part in cut(tokens, sizes)])[tag]
        check(got, want, "float32", f"{heads} heads of {dim} and {vdim}, tau {tau}, rank {rank}, portions of {sizes}")
        loaded.step.end(tag)


@pytest.mark.parametrize("heads,vdim,state,groups,taps,norm_groups", [(1, 4, 3, 1, 1, 1), (4, 8, 16, 4, 2, 2), (6, 10, 7, 3, 3, 6),
                                                                     (4, 64, 64, 1, 4, 1), (2, 70, 130, 2, 4, 2), (3, 20, 260, 1, 6, 3)])
def test_heads_states_groups_and_norm_groups_of_mamba2(tmp_path, heads, vdim, state, groups, taps, norm_groups):
    raw = fm.single_layer(fm.mamba(heads, vdim, state, groups, taps, norm_groups))
    folder = str(tmp_path / "one")
    raw, bf16 = fm.write_model(folder, raw, 45)
    tokens = tokens_of(raw["vocab"], 141, 13)
    want = plain.logits(raw, plain.as_float64(bf16), tokens)
    loaded = load(folder, "float32")
    for tag, sizes in (("a", [141]), ("b", [8, 7, 9, 1, 16]), ("c", [64, 64, 13]), ("d", [63, 1, 3, 65])):
        got = run_steps(loaded, [[(tag, part)] for part in cut(tokens, sizes)])[tag]
        check(got, want, "float32", f"{heads} heads of {vdim}, states of {state}, portions of {sizes}")
        loaded.step.end(tag)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("streams", [1, 2, 3, 4, 5, 8, 16])
@pytest.mark.parametrize("width", [64, 50])
def test_numbers_of_streams(tmp_path, streams, width, dtype):
    """Three layers (one runs twice) over one to sixteen streams, whose order and directions all matter: the plain model with
    the mixes turned around differs."""
    raw = fm.config(80, width, [fm.with_mlp(fm.mamba(2, 8, 8, 1, 3, 1), 40), fm.with_mlp(fm.attention(2, 1, 8, 8, fm.rotation(100.0, 4)), None),
                                fm.with_mlp(fm.parallel((2, 2, 8, 8, 2, 9, 6.0, 0.4), (1, 8, 8, 4.0, 8)), 32)],
                    streams=streams, loop=(1, 2, 2))
    folder = str(tmp_path / "one")
    raw, bf16 = fm.write_model(folder, raw, 46)
    tensors = plain.as_float64(bf16)
    tokens = tokens_of(raw["vocab"], 60, 14)
    want = plain.logits(raw, tensors, tokens)
    if streams > 1:
        turned = {key: value.T if key.endswith(".mix") and ".hc" in key else value for key, value in tensors.items()}
        assert np.median(spread_error(plain.logits(raw, turned, tokens), want)) > 0.005
    loaded = load(folder, dtype)
    for tag, sizes in (("w", [60]), ("p", [17, 2, 20, 1]), ("d", [30] + [1] * 30)):
        check(run_steps(loaded, [[(tag, part)] for part in cut(tokens, sizes)])[tag], want, dtype, f"{streams} streams, {sizes}")
        loaded.step.end(tag)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_repeated_layers_have_caches_and_states_of_their_own(tmp_path, dtype):
    """Each kind of layer three times in a row: passes that shared a cache, a state or carried inputs would go wrong from
    the second token on; in the plain model it shows that the passes differ."""
    for layer in (fm.mamba(2, 8, 8, 1, 3, 1), fm.attention(2, 1, 8, 8, fm.rotation(100.0, 4)),
                  fm.parallel((2, 2, 8, 8, 2, 9, 6.0, 0.4), (1, 8, 8, 4.0, 8))):
        raw = fm.config(80, 40, [fm.with_mlp(layer, 24)], streams=2, loop=(0, 1, 3))
        folder = str(tmp_path / f"one{layer['type']}")
        raw, bf16 = fm.write_model(folder, raw, 47)
        tensors = plain.as_float64(bf16)
        tokens = tokens_of(raw["vocab"], 50, 15)
        want = plain.logits(raw, tensors, tokens)
        assert np.median(spread_error(plain.logits(dict(raw, loop={"start": 0, "stop": 1, "times": 2}), tensors, tokens), want)) > 0.1
        loaded = load(folder, dtype)
        for tag, sizes in (("w", [50]), ("p", [7, 2, 20, 1]), ("d", [1])):
            check(run_steps(loaded, [[(tag, part)] for part in cut(tokens, sizes)])[tag], want, dtype, f"{layer['type']}, {sizes}")
            loaded.step.end(tag)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("sizes", [(4, 2, 16, 16), (17, 1, 12, 5), (4, 1, 64, 64), (2, 2, 128, 64)])
def test_the_cap_shows_where_scores_are_high(tmp_path, sizes, dtype):
    heads, groups, dim, vdim = sizes
    raw = fm.single_layer(fm.parallel((heads, groups, dim, vdim, 2, 50, 1.5, 8.0 * dim ** -0.5), (1, 4, 4, 2.0, 2)))
    bf16 = fm.make_tensors(raw, 41)
    open_connection(bf16)
    change(bf16, "l0.mix.right.out", lambda w: 0 * w)
    folder = str(tmp_path / "one")
    fm.write_model(folder, raw, 0, tensors=bf16)
    tensors = plain.as_float64(bf16)
    tokens = tokens_of(raw["vocab"], 80, 15)
    want = plain.logits(raw, tensors, tokens)
    keep, plain.capped = plain.capped, lambda scores, cap: scores
    try:
        without = plain.logits(raw, tensors, tokens)
    finally:
        plain.capped = keep
    assert np.median(spread_error(without, want)) > 0.2
    loaded = load(folder, dtype)
    for tag, steps in (("w", [tokens]), ("d", [tokens[:30]] + [[t] for t in tokens[30:]])):
        check(run_steps(loaded, [[(tag, part)] for part in steps])[tag], want, dtype, f"capped scores, {tag}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("ff,limit", [(24, 0.4), (40, 1.0), (136, 7.0), (20, 2.0)])
def test_limits_of_the_gated_unit(tmp_path, ff, limit, dtype):
    """Gates and up values cut off on their sides, in steps of few and of many tokens."""
    raw = fm.single_layer(fm.mamba(1, 8, 4, 1, 2, 1), ff, limit=limit)
    folder = str(tmp_path / "one")
    raw, bf16 = fm.write_model(folder, raw, 48)
    tokens = tokens_of(raw["vocab"], 150, 13)
    tensors = plain.as_float64(bf16)
    want = plain.logits(raw, tensors, tokens)
    if limit < 2.0:
        raw["layers"][0]["mlp"]["limit"] = 50.0
        assert np.median(spread_error(plain.logits(raw, tensors, tokens), want)) > 0.02
        raw["layers"][0]["mlp"]["limit"] = limit
    loaded = load(folder, dtype)
    check(run_steps(loaded, [[("w", tokens)]])["w"], want, dtype, f"{ff} inner, limit {limit}, whole")
    check(run_steps(loaded, [[("p", part)] for part in cut(tokens, [3, 16, 17, 1, 40])])["p"], want, dtype, f"limit {limit}, portions")


# ---------------------------------------------------------------------------- the engine's own entry point
def compare_greedy(raw, tensors, prompts, got, new, margin):
    """Generated tokens against greedy decoding with the plain model wherever its best two logits are not close."""
    compared = 0
    for prompt, generated in zip(prompts, got):
        assert len(generated) == new
        sequence = list(prompt)
        for token in generated:
            logits = plain.logits(raw, tensors, sequence)[-1]
            top = np.sort(logits)[-2:]
            if top[1] - top[0] > margin * (logits.max() - logits.min()):
                assert int(token) == int(np.argmax(logits))
                compared += 1
            sequence.append(int(token))
    return compared


@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_greedy_generation_through_the_engine(models, name):
    from celeg_b200 import Engine, EngineOptions
    folder, raw, tensors = models[name]
    prompts = [tokens_of(raw["vocab"], n, 50 + n) for n in (5, 41, 18)]
    engine = Engine(folder, max_context=128, dtype="float32",
                    options=EngineOptions(max_active_requests=4, max_batched_tokens=32, page_tokens=16))
    got = engine.generate(prompts, max_new_tokens=12, temperature=0.0, repetition_penalty=1.0)
    assert compare_greedy(raw, tensors, prompts, got, 12, 1e-2) >= 24


def test_greedy_generation_in_bfloat16_with_graphs(models):
    """The serving path: bfloat16, CUDA graphs, run-ahead."""
    from celeg_b200 import Engine, EngineOptions
    folder, raw, tensors = models["wide"]
    prompts = [tokens_of(raw["vocab"], n, 70 + n) for n in (9, 30)]
    engine = Engine(folder, max_context=128, dtype="bfloat16",
                    options=EngineOptions(max_active_requests=4, max_batched_tokens=64, page_tokens=16))
    got = engine.generate(prompts, max_new_tokens=10, temperature=0.0, repetition_penalty=1.0)
    compare_greedy(raw, tensors, prompts, got, 10, 0.08)


def test_many_requests_through_a_small_pool(models):
    """Nine prompts through two slots and a pool of a few pages: the scheduler queues, admits as slots and pages come
    free, and every request's tokens are those of greedy decoding alone."""
    from celeg_b200 import Engine, EngineOptions
    folder, raw, tensors = models["odd"]
    prompts = [tokens_of(raw["vocab"], 3 + 5 * n, 200 + n) for n in range(9)]
    engine = Engine(folder, max_context=96, dtype="float32",
                    options=EngineOptions(max_active_requests=2, max_batched_tokens=24, page_tokens=16, logical_kv_pages=10))
    got = engine.generate(prompts, max_new_tokens=6, temperature=0.0, repetition_penalty=1.0)
    assert compare_greedy(raw, tensors, prompts, got, 6, 1e-2) >= 40


def test_command_line_generates_and_dumps_logits(models, tmp_path, capsys):
    from celeg_b200.cli import main
    folder, raw, tensors = models["odd"]
    prompt = tokens_of(raw["vocab"], 12, 90)
    dump = str(tmp_path / "last.f32")
    code = main(["--model", folder, "--prompt-ids", ",".join(map(str, prompt)), "--max-new-tokens", "6", "--dtype", "fp32",
                 "--temperature", "0", "--repetition-penalty", "1.0", "--runtime-tokens", "--dump-logits", dump,
                 "--context", "128"])
    assert code == 0
    captured = capsys.readouterr()
    sequence = list(prompt)
    for _ in range(6):
        sequence.append(int(np.argmax(plain.logits(raw, tensors, sequence)[-1])))
    assert f"CELEG_GENERATED_TOKEN_IDS=[{','.join(map(str, sequence[len(prompt):]))}]" in captured.out
    logits = np.fromfile(dump, dtype="<f4").astype(np.float64)
    assert spread_error(logits[None, :], plain.logits(raw, tensors, prompt)[-1:])[0] < 2e-4
    assert main(["--model", folder, "--print-config"]) == 0
    assert '"architecture": "Fovezen"' in capsys.readouterr().out


# ------------------------------------------------------------------------------- configurations drawn at random
def random_config(rng):
    width = int(rng.choice([20, 36, 64, 100, 128]))
    layers = []
    for _ in range(int(rng.integers(1, 6))):
        pick = rng.random()
        heads, groups = [(1, 1), (2, 1), (4, 2), (6, 2), (8, 8), (12, 3), (20, 1)][int(rng.integers(0, 7))]
        dim, vdim = int(rng.choice([4, 8, 12, 32, 64])), int(rng.choice([4, 9, 16, 64, 128]))
        scale = float(rng.choice([dim ** -0.5, 0.125, 0.5]))
        if pick < 0.3:
            rot = fm.rotation(float(rng.choice([50.0, 10000.0, 1e6])), 2 * int(rng.integers(1, dim // 2 + 1)),
                              factor=None if rng.random() < 0.4 else float(rng.choice([2.0, 8.0])), low=float(rng.choice([0.5, 1.0])),
                              high=float(rng.choice([2.0, 4.0])), original=int(rng.choice([32, 256, 4096])))
            layer = fm.attention(heads, groups, dim, vdim, rot, scale=scale)
        elif pick < 0.65:
            layer = fm.parallel((heads, groups, dim, vdim, int(rng.integers(1, 7)), int(rng.choice([1, 2, 15, 16, 17, 40, 500])),
                                 float(rng.choice([1.0, 8.0, 30.0])), scale),
                                (int(rng.integers(1, 4)), int(rng.choice([4, 9, 16, 64, 130])), int(rng.choice([5, 16, 64])),
                                 float(rng.choice([1.0, 4.0, 16.0])), int(rng.choice([1, 8, 20]))))
        else:
            m_groups = int(rng.choice([1, 2, 3]))
            m_heads, m_vdim = m_groups * int(rng.integers(1, 4)), int(rng.choice([4, 7, 16, 64]))
            layer = fm.mamba(m_heads, m_vdim, int(rng.choice([3, 8, 16, 70])), m_groups, int(rng.integers(1, 7)),
                             int(rng.choice([n for n in (1, m_groups, m_heads) if (m_heads * m_vdim) % n == 0])))
        layers.append(fm.with_mlp(layer, None if rng.random() < 0.25 else int(rng.choice([8, 20, 64])), limit=float(rng.choice([0.5, 1.5, 7.0]))))
    loop = None
    if rng.random() < 0.6:
        start = int(rng.integers(0, len(layers)))
        loop = (start, int(rng.integers(start + 1, len(layers) + 1)), int(rng.integers(1, 4)))
    return fm.config(int(rng.integers(17, 300)), width, layers, streams=int(rng.choice([1, 2, 3, 4, 6])),
                     eps=float(rng.choice([1e-5, 1e-6, 1e-3])), logit_scale=float(rng.choice([1.0, 0.3, 2.5])), loop=loop)


@pytest.mark.parametrize("seed", range(14))
def test_configurations_drawn_at_random(tmp_path, seed):
    """Whole prompt, portions beside single tokens of a second request, and decoding, in both precisions."""
    rng = np.random.default_rng(3000 + seed)
    raw = random_config(rng)
    folder = str(tmp_path / "drawn")
    raw, bf16 = fm.write_model(folder, raw, 700 + seed)
    tensors = plain.as_float64(bf16)
    first, second = tokens_of(raw["vocab"], 75, seed), tokens_of(raw["vocab"], 33, 100 + seed)
    want = {"a": plain.logits(raw, tensors, first), "b": plain.logits(raw, tensors, second)}
    steps = [[("a", first[:19])], [("a", first[19:21]), ("b", second[:1])], [("b", second[1:2]), ("a", first[21:60])],
             [("a", first[60:61]), ("b", second[2:30])]]
    steps += [[("a", first[61 + i:62 + i])] + ([("b", second[30 + i:31 + i])] if 30 + i < len(second) else []) for i in range(14)]
    for dtype in ("float32", "bfloat16"):
        loaded = load(folder, dtype, page_tokens=int(rng.choice([8, 16, 32])))
        whole = run_steps(loaded, [[("w", first)]])["w"]
        loaded.step.end("w")
        got = run_steps(loaded, steps)
        if dtype == "float32":
            check(whole, want["a"], dtype, f"{raw} whole")
            for key in ("a", "b"):
                check(got[key], want[key], dtype, f"{raw} request {key}")
        else:
            for rows, target in ((whole, want["a"]), (got["a"], want["a"]), (got["b"], want["b"])):
                assert np.median(spread_error(np.asarray(rows, dtype=np.float64), target)) < 0.1


# ------------------------------------------------------------------------------------------ trace replay
def replay_steps(requests, seed):
    """A schedule for up to four live requests: portions of changing size (two tokens too) beside single tokens, requests
    left out of steps, ended requests followed by new ones."""
    rng = np.random.default_rng(seed)
    waiting = list(requests)
    live, at, steps = [], {}, []
    while waiting or live:
        while waiting and len(live) < 4:
            name = waiting.pop(0)
            live.append(name)
            at[name] = 0
        entries, ended = [], []
        for name in list(live):
            tokens = requests[name]
            if len(live) > 1 and rng.random() < 0.2:
                continue                                       # (left out of this step)
            count = min(len(tokens) - at[name], int(rng.choice([1, 1, 2, 3, 17, 40])))
            entries.append({"id": name, "tokens": tokens[at[name]:at[name] + count], "want": list(range(count))})
            at[name] += count
            if at[name] == len(tokens):
                ended.append(name)
                live.remove(name)
        if entries:
            steps.append({"step": len(steps), "entries": entries, "end": ended})
    return steps


MAMBA_ONLY = fm.config(70, 40, [fm.with_mlp(fm.mamba(2, 8, 12, 1, 4, 1), 24), fm.with_mlp(fm.mamba(3, 20, 4, 3, 2, 2), None)], streams=2)
ATTENTION_ONLY = fm.config(90, 24, [fm.with_mlp(fm.attention(2, 2, 8, 4, fm.rotation(300.0, 8)), None),
                                    fm.with_mlp(fm.attention(4, 1, 8, 8, fm.rotation(300.0, 4, factor=2.0)), 8)], streams=4, loop=(0, 2, 2))
PARALLEL_ONLY = fm.config(64, 32, [fm.with_mlp(fm.parallel((2, 1, 8, 16, 2, 7, 3.0, 0.4), (2, 8, 4, 2.0, 2)), 24)], streams=3, loop=(0, 1, 3))
ALONE = {"mamba_only": MAMBA_ONLY, "attention_only": ATTENTION_ONLY, "parallel_only": PARALLEL_ONLY}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["mixed", "odd", "even", *ALONE])
def test_replay_with_pages_and_slots_used_again(models, name, dtype, tmp_path):
    """Seven requests (640 positions in whole blocks of 64) through the trace runner's step loop with a pool for 448
    positions, what four live ones can hold at most, and four slots."""
    import io
    import json
    import os
    from celeg_b200.engine.trace import replay
    if name in models:
        folder, raw, tensors = models[name]
    else:
        folder = str(tmp_path / name)
        raw, bf16 = fm.write_model(folder, ALONE[name], 77)
        tensors = plain.as_float64(bf16)
    requests = {f"r{i}": tokens_of(raw["vocab"], n, 300 + i) for i, n in enumerate([70, 9, 100, 33, 64, 2, 81])}
    steps = replay_steps(requests, 5)
    out_dir = str(tmp_path / f"out_{dtype}")
    done = io.StringIO()
    text = io.StringIO("".join(json.dumps(step) + "\n" for step in steps))
    assert replay(folder, dtype, out_dir, 448, text, done, max_requests=4) == 0
    assert done.getvalue().split() == [w for step in steps for w in ("done", str(step["step"]))]
    rows = {key: [] for key in requests}
    for step in steps:
        data = np.fromfile(os.path.join(out_dir, f"{step['step']}.f32"), dtype="<f4").reshape(-1, raw["vocab"])
        row = 0
        for entry in step["entries"]:
            rows[entry["id"]].append(data[row:row + len(entry["want"])])
            row += len(entry["want"])
        assert row == data.shape[0]
    for key, tokens in requests.items():
        check(np.concatenate(rows[key]), plain.logits(raw, tensors, tokens), dtype, f"{name} request {key} replayed")


def test_the_trace_runner_as_a_program(models, tmp_path):
    import json
    import os
    import subprocess
    import sys
    folder, raw, tensors = models["odd"]
    tokens = tokens_of(raw["vocab"], 21, 400)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": tokens[:18], "want": [0, 17]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": tokens[18:20], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": tokens[20:], "want": [0]}], "end": ["a"]}]
    program = os.path.join(os.path.dirname(os.path.dirname(os.path.abspath(__file__))), "bin", "trace_run")
    out_dir = str(tmp_path / "out")
    result = subprocess.run([program, "--model", folder, "--dtype", "float32", "--out", out_dir, "--max-tokens", "64"],
                            input="".join(json.dumps(step) + "\n" for step in steps), capture_output=True, text=True,
                            timeout=600, env=dict(os.environ, PYTHON=sys.executable))
    assert result.returncode == 0, result.stderr[-2000:]
    assert [line for line in result.stdout.split("\n") if line.startswith("done")] == ["done 0", "done 1", "done 2"]
    assert not os.path.exists(os.path.join(out_dir, "1.f32"))
    want = plain.logits(raw, tensors, tokens)
    got = np.concatenate([np.fromfile(os.path.join(out_dir, f"{n}.f32"), dtype="<f4").reshape(-1, raw["vocab"]) for n in (0, 2)])
    check(got, want[[0, 17, 20]], "float32", "the program's logits")


# ------------------------------------------------------------------------------- layers of a real model's size
@pytest.fixture(scope="module")
def large(tmp_path_factory):
    """Four layers 1,024 wide over four streams: sixteen Mamba-2 heads of 64 with states of 128; sixteen query heads of 64 on
    four key heads under a window of 192 beside eight linear heads of 64 and 128; eight rotated heads of 128 on two. The
    sizes at which the tcgen05 prompt attention and gated product and the split-key decoding are what runs."""
    rot = fm.rotation(300000.0, 64, factor=4.0, original=256)
    raw = fm.config(4096, 1024, [
        fm.with_mlp(fm.mamba(16, 64, 128, 2, 4, 4), 2816, limit=2.0),
        fm.with_mlp(fm.parallel((16, 4, 64, 64, 4, 192, 25.0, 0.15), (8, 64, 128, 12.0, 32)), 1536),
        fm.with_mlp(fm.attention(8, 2, 128, 128, rot), None),
        fm.with_mlp(fm.parallel((8, 8, 64, 64, 4, 300, 25.0, 0.15), (4, 128, 64, 12.0, 16)), 1024),
    ], streams=4, logit_scale=0.6)
    folder = str(tmp_path_factory.mktemp("fovezen_large") / "model")
    raw, bf16 = fm.write_model(folder, raw, 91)
    tensors = plain.as_float64(bf16)
    first, second = tokens_of(raw["vocab"], 568, 500), tokens_of(raw["vocab"], 250, 501)
    return folder, raw, {"a": first, "b": second}, {"a": plain.logits(raw, tensors, first), "b": plain.logits(raw, tensors, second)}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_layers_of_a_real_model_size(large, dtype):
    folder, raw, requests, want = large
    first, second = requests["a"], requests["b"]
    loaded = load(folder, dtype, cache_tokens=2048, max_batched_tokens=1024, max_context=1024)
    steps = [[("a", first[:560])], [("a", first[560:561]), ("b", second[:100])], [("a", first[561:562]), ("b", second[100:])]]
    steps += [[("a", [t])] for t in first[562:]]
    got = run_steps(loaded, steps)
    for key in ("a", "b"):
        check(got[key], want[key], dtype, f"request {key} at a real model's layer sizes")
