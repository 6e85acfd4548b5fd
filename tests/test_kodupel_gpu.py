"""The Kodupel design in the engine against the plain float64 model of ``plain_kodupel.py``: whole prompts, decoding token
by token, portions down to two tokens, batches of unequal requests, pages and slots used again, far keys at page borders
with weights that make one key show (through a layer's own cache and through another layer's), a far token through the
delta rule's state and its removal by a later token with the same key, chunk borders of the scan, the one in the softmax's
denominator, the experts' choices and limits, and greedy generation through ``Engine`` and the command line. float32 path
to 2e-4 of the logits' spread, bfloat16 path to a few percent."""
from __future__ import annotations

import numpy as np
import pytest

import kodupel_models as km
import plain_kodupel as plain

pytestmark = pytest.mark.gpu

LIMIT = {"float32": 2e-4, "bfloat16": 1.5e-1}
TYPICAL = {"float32": 1e-4, "bfloat16": 6e-2}


def spread_error(got: np.ndarray, want: np.ndarray) -> np.ndarray:
    """Per row: rms of the difference (mean taken off) over the rms of the wanted row (mean taken off)."""
    d = got - want
    d = d - d.mean(-1, keepdims=True)
    w = want - want.mean(-1, keepdims=True)
    return np.sqrt((d ** 2).mean(-1)) / np.sqrt((w ** 2).mean(-1))


def check(got, want, dtype, what, routed=False, slack=1.0):
    """``routed``: the model chooses experts. In bfloat16 a token whose best choices lie close together may take another
    expert than in the plain model, and its row (and, fading, the rows after it) then differs by more than rounding; one
    row in twelve (rounded up) may, by at most the row's whole spread. float32 is held to the limit everywhere."""
    err = spread_error(np.asarray(got, dtype=np.float64), want)
    worst = int(np.argmax(err))
    if routed and dtype == "bfloat16":
        assert err[worst] <= 1.0, f"{what}: row {worst} differs by {err[worst]:.3e} of the row's spread"
        assert (err > LIMIT[dtype]).sum() <= -(-len(err) // 12), f"{what}: {(err > LIMIT[dtype]).sum()} rows over the limit"
    else:
        assert err[worst] <= slack * LIMIT[dtype], f"{what}: row {worst} differs by {err[worst]:.3e} of the row's spread"
    assert np.median(err) <= slack * TYPICAL[dtype], f"{what}: half of the rows differ by {np.median(err):.3e} and more"


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    base = tmp_path_factory.mktemp("kodupel")
    out = {}
    for name, (raw, seed) in km.CONFIGS.items():
        folder = str(base / name)
        raw, tensors = km.write_model(folder, raw, seed)
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
@pytest.mark.parametrize("name", list(km.CONFIGS))
def test_whole_prompt_then_token_by_token(models, name, dtype):
    folder, raw, tensors = models[name]
    tokens = tokens_of(raw["vocab"], 90, 1)
    want = plain.logits(raw, tensors, tokens)
    loaded = load(folder, dtype)
    whole = run_steps(loaded, [[("w", tokens)]])["w"]
    check(whole, want, dtype, f"{name} whole", routed=True)
    loaded.step.end("w")
    decoded = run_steps(loaded, [[("d", tokens[:37])]] + [[("d", [t])] for t in tokens[37:]])["d"]
    check(decoded, want, dtype, f"{name} prompt of 37 then token by token", routed=True)
    if dtype == "float32":       # how the prompt is cut changes nothing beyond rounding
        assert np.abs(decoded - whole).max() <= 1e-3 * np.abs(whole).max()


@pytest.mark.parametrize("name", list(km.CONFIGS))
def test_the_stream_after_every_layer(models, name, tmp_path):
    """A model cut after its n-th layer, with an identity for the final norm's scale and unit rows as its head, hands out
    the stream itself (divided by its root mean square): layer by layer against the plain model."""
    import torch
    folder, raw, tensors = models[name]
    tokens = tokens_of(raw["vocab"], 40, 21)
    want = plain.streams(raw, tensors, tokens)
    width = raw["width"]
    for depth in range(1, len(raw["layers"]) + 1):
        short = dict(raw, layers=raw["layers"][:depth])
        kept = {key: torch.from_numpy(value).to(torch.bfloat16) for key, value in tensors.items()
                if not key.startswith("l") or int(key[1:key.index(".")]) < depth}
        kept["final.norm"] = torch.zeros(width, dtype=torch.bfloat16)
        head = torch.zeros((raw["vocab"], width), dtype=torch.bfloat16)
        head[:width] = torch.eye(width)[:raw["vocab"]]
        kept["head"] = head
        cut_folder = str(tmp_path / f"{name}{depth}")
        km.write_model(cut_folder, short, 0, tensors=kept)
        got = run_steps(load(cut_folder, "float32"), [[("a", tokens)]])["a"][:, :min(width, raw["vocab"])].astype(np.float64)
        normed = plain.rms_scaled(want[depth - 1], float(raw["norm"]["eps"]))[:, :got.shape[1]]
        assert np.abs(got - normed).max() <= 5e-5 * np.abs(normed).max(), f"{name} after layer {depth - 1}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(km.CONFIGS))
def test_portions_of_several_sizes_down_to_two_tokens(models, name, dtype):
    folder, raw, tensors = models[name]
    tokens = tokens_of(raw["vocab"], 131, 2)
    want = plain.logits(raw, tensors, tokens)
    loaded = load(folder, dtype)
    for tag, sizes in (("a", [2, 3, 17, 2, 33]), ("b", [16, 16, 1, 15, 48]), ("c", [5, 2, 2, 64]), ("d", [8, 7, 9])):
        got = run_steps(loaded, [[(tag, part)] for part in cut(tokens, sizes)])[tag]
        check(got, want, dtype, f"{name} in portions of {sizes}", routed=True)
        loaded.step.end(tag)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(km.CONFIGS))
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
        check(got[key], want[key], dtype, f"{name} request {key} in a batch", routed=True)


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
            check(got[key], plain.logits(raw, tensors, tokens), dtype, f"turn {turn} request {key}", routed=True)
            loaded.step.end(key)
        loaded.manager.check_invariants()
    assert loaded.manager.free_slots == 2


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_long_portions_beside_short_ones(models, name, dtype):
    """Portions of hundreds of tokens (the experts' pairs are grouped, the scan walks many chunks) beside single tokens
    and short portions of other requests, from states and caches that earlier portions left."""
    folder, raw, tensors = models[name]
    requests = {"a": tokens_of(raw["vocab"], 700, 31), "b": tokens_of(raw["vocab"], 140, 32), "c": tokens_of(raw["vocab"], 300, 33)}
    want = {key: plain.logits(raw, tensors, value) for key, value in requests.items()}
    a, b, c = (requests[key] for key in "abc")
    loaded = load(folder, dtype, cache_tokens=2048, max_batched_tokens=1024, max_context=1024)
    got = run_steps(loaded, [[("b", b[:1]), ("a", a[:349])], [("b", b[1:2]), ("a", a[349:350]), ("c", c[:285])],
                             [("b", b[2:131]), ("a", a[350:677]), ("c", c[285:])], [("b", b[131:]), ("a", a[677:])]])
    for key in want:
        check(got[key], want[key], dtype, f"{name} request {key} in long portions", routed=True)


@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_long_decoding_from_the_first_token(models, name):
    folder, raw, tensors = models[name]
    tokens = tokens_of(raw["vocab"], 200, 7)
    got = run_steps(load(folder, "float32"), [[("l", [t])] for t in tokens])["l"]
    check(got, plain.logits(raw, tensors, tokens), "float32", "200 tokens one by one")


def test_the_first_tokens_of_a_sequence(tmp_path):
    """Prompts of one, two and three tokens and decoding from there: the state starts from zero, the first token's
    attention has its own key and the one in the denominator."""
    for name, (raw, seed) in km.CONFIGS.items():
        folder = str(tmp_path / name)
        raw, bf16 = km.write_model(folder, raw, seed)
        tokens = tokens_of(raw["vocab"], 12, 16)
        want = plain.logits(raw, plain.as_float64(bf16), tokens)
        loaded = load(folder, "float32")
        for first in (1, 2, 3):
            got = run_steps(loaded, [[("f", tokens[:first])]] + [[("f", [t])] for t in tokens[first:]])["f"]
            check(got, want, "float32", f"{name}: a prompt of {first}")
            loaded.step.end("f")


# ------------------------------------------------------------------------- one mechanism, made to show
def single_out(bf16, token, column, value=3.0):
    """Column ``column`` of the embedding table becomes zero for every token but ``token``: in a first layer, which reads
    the rows as they are, that input dimension then speaks for this token alone."""
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


def build_far_key(sizes, far, probe, length, shared):
    """Every head's query of ONE token (through an input dimension that only this token has) points at the key that ONE
    other token makes at place ``far``, along dimensions that do not turn. With ``shared`` the probing layer is the second,
    which reads the first layer's keys; the first layer's output counts for nothing then. Returns (raw, bf16, sequence
    with that token, sequence with another in its place, the probing layer's index)."""
    heads, groups, dim, vdim, rot_dims = sizes
    rot = km.rotation(1000.0, rot_dims, factor=2.0)
    layers = [km.with_mlp(km.attention(heads, groups, dim, vdim, rot, scale=8.0 / dim), None)]
    if shared:
        layers.append(km.with_mlp(km.attention(heads, groups, dim, vdim, rot, scale=8.0 / dim, kv_from=0), None))
    raw = km.config(96, 48, layers)
    bf16 = km.make_tensors(raw, 40)
    vocab, width = raw["vocab"], raw["width"]
    key_token, probe_token, other_token = vocab - 1, vocab - 2, vocab - 3
    single_out(bf16, probe_token, width - 2)
    single_out(bf16, key_token, width - 4)
    changed = np.random.default_rng(8).integers(0, vocab - 3, size=length).tolist()
    changed[probe] = probe_token
    without = list(changed)
    changed[far], without[far] = key_token, other_token
    at = 1 if shared else 0
    rng = np.random.default_rng(9)
    direction = np.zeros((groups, dim))
    direction[:, rot_dims:] = rng.choice([-1.0, 1.0], size=(groups, dim - rot_dims))
    set_column(bf16, "l0.mix.k", slice(0, groups * dim), width - 4, 4.0 * direction.reshape(-1))
    set_column(bf16, "l0.mix.v", slice(0, groups * vdim), width - 4, 3.0 * rng.normal(size=groups * vdim))
    for head in range(heads):
        set_column(bf16, f"l{at}.mix.q", slice(head * dim, (head + 1) * dim), width - 2, 4.0 * direction[head // (heads // groups)])
    change(bf16, f"l{at}.mix.q.norm", lambda w: 0 * w + 1.7)
    change(bf16, "l0.mix.k.norm", lambda w: 0 * w + 1.2)
    change(bf16, f"l{at}.mix.g", lambda w: 0.2 * w)
    change(bf16, f"l{at}.mix.o.b", lambda w: 0.2 * w)
    change(bf16, f"l{at}.norm1", lambda w: 0 * w + 3.0)
    if shared:
        change(bf16, "l0.norm1", lambda w: 0 * w - 1.0)
    return raw, bf16, changed, without, at


FAR = [((4, 2, 8, 12, 4), 0, 317), ((4, 2, 8, 12, 4), 15, 317), ((4, 2, 8, 12, 4), 16, 240), ((17, 1, 24, 8, 6), 31, 300),
       ((17, 1, 24, 8, 6), 299, 300), ((3, 3, 12, 5, 2), 255, 256), ((8, 2, 64, 64, 16), 0, 340), ((8, 2, 64, 64, 16), 127, 390),
       ((8, 2, 64, 64, 16), 128, 390), ((8, 1, 64, 128, 32), 63, 340), ((4, 4, 128, 64, 8), 64, 389), ((2, 1, 16, 16, 4), 79, 80)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("shared", [False, True])
@pytest.mark.parametrize("sizes,far,probe", FAR)
def test_far_keys_at_page_borders(tmp_path, sizes, far, probe, shared, dtype):
    """Which token stood at ``far`` moves the probe's logits; the engine follows the plain model with the probe inside a
    prompt, as the first token of a portion, and decoded alone (after a prompt and after decoded tokens)."""
    raw, bf16, changed, without, _ = build_far_key(sizes, far, probe, probe + 9, shared)
    folder = str(tmp_path / "one")
    km.write_model(folder, raw, 0, tensors=bf16)
    tensors = plain.as_float64(bf16)
    want, reference = plain.logits(raw, tensors, changed), plain.logits(raw, tensors, without)
    moved = spread_error(want[probe:probe + 1], reference[probe:probe + 1])[0]
    assert moved > 0.2, f"the plain model itself: {moved}"
    loaded = load(folder, dtype)
    start = max(1, min(far - 5, probe - 1), probe - 90)
    for tag, steps in (("prompt", [changed]), ("portion", [changed[:probe], changed[probe:]]),
                       ("inside", [changed[:probe - 3], changed[probe - 3:probe + 2], changed[probe + 2:]]),
                       ("decoded", [changed[:probe]] + [[t] for t in changed[probe:]]),
                       ("later", [changed[:start]] + [[t] for t in changed[start:]])):
        got = run_steps(loaded, [[(tag, part)] for part in steps])[tag]
        check(got, want, dtype, f"key at {far}, probe at {probe}, {tag}")
        assert spread_error(got[probe:probe + 1].astype(np.float64), reference[probe:probe + 1])[0] > 0.15, tag
        loaded.step.end(tag)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("sizes", [(4, 2, 16, 16), (17, 1, 12, 5), (4, 1, 64, 64), (2, 2, 128, 64)])
def test_the_one_in_the_denominator_shows_where_all_scores_are_low(tmp_path, sizes, dtype):
    """Biases that make every query look away from every key: the weights sum to almost nothing, where a softmax without
    the one would hand out the values' mean."""
    heads, groups, dim, vdim = sizes
    raw = km.single_layer(km.attention(heads, groups, dim, vdim, km.rotation(1e6, 2), scale=6.0 / dim))
    bf16 = km.make_tensors(raw, 41)
    rng = np.random.default_rng(14)
    direction = rng.choice([-1.0, 1.0], size=dim)
    change(bf16, "l0.mix.k.b", lambda b: np.tile(6.0 * direction, groups))
    change(bf16, "l0.mix.q.b", lambda b: np.tile(-6.0 * direction, heads))
    folder = str(tmp_path / "one")
    km.write_model(folder, raw, 0, tensors=bf16)
    tensors = plain.as_float64(bf16)
    tokens = tokens_of(raw["vocab"], 80, 15)
    want = plain.logits(raw, tensors, tokens)
    x = plain.embed(raw, tensors, tokens)
    k, v = plain.keys_and_values(tensors, "l0.mix.", raw["layers"][0]["mixer"], x, 1e-5)
    keep, plain.weights_with_one = plain.weights_with_one, lambda s: np.exp(s - s.max()) / np.exp(s - s.max()).sum()
    try:
        without = plain.logits(raw, tensors, tokens)
    finally:
        plain.weights_with_one = keep
    assert np.median(spread_error(without, want)) > 0.2
    loaded = load(folder, dtype)
    for tag, steps in (("w", [tokens]), ("d", [tokens[:30]] + [[t] for t in tokens[30:]])):
        check(run_steps(loaded, [[(tag, part)] for part in steps])[tag], want, dtype, f"low scores, {tag}")


def build_far_state(remove):
    """One recurrent layer whose channels keep almost everything: ONE token writes a large value under a key of its own,
    ONE probe token reads along that key 250 tokens later. With ``remove`` a third token has the same key, removes what
    lies along it (its removal rates are one) and writes nothing."""
    raw = km.single_layer(km.delta(2, 16, 6))
    bf16 = km.make_tensors(raw, 42)
    vocab, width = raw["vocab"], raw["width"]
    key_token, probe_token, remove_token = vocab - 1, vocab - 2, vocab - 3
    for token, column in ((key_token, width - 2), (probe_token, width - 4), (remove_token, width - 6)):
        single_out(bf16, token, column)
    # unit directions that the key channels of both heads share
    direction = np.random.default_rng(11).choice([-1.0, 1.0], size=32)
    for name in ("k", "v", "r"):
        change(bf16, f"l0.mix.{name}", lambda w: 0.15 * w)
    change(bf16, "l0.mix.a", lambda w: 0.0 * w)
    change(bf16, "l0.mix.a.b", lambda b: 0 * b - 12.0)
    change(bf16, "l0.mix.w0", lambda b: 0 * b - 10.0)
    change(bf16, "l0.mix.w2", lambda w: 0.1 * w)
    set_column(bf16, "l0.mix.k", slice(0, 32), width - 2, 0.5 * direction)
    set_column(bf16, "l0.mix.v", slice(0, 32), width - 2, 3.0 * np.random.default_rng(12).normal(size=32))
    set_column(bf16, "l0.mix.r", slice(0, 32), width - 4, 0.5 * direction)
    set_column(bf16, "l0.mix.k", slice(0, 32), width - 6, 0.5 * direction)
    set_column(bf16, "l0.mix.a", slice(0, 32), width - 6, 2.0)
    changed = np.random.default_rng(10).integers(0, vocab - 3, size=256).tolist()
    changed[3] = key_token
    for place in (250, 255):
        changed[place] = probe_token
    without = list(changed)
    if remove:
        changed[100] = remove_token
    else:
        without[3] = 0
    return raw, bf16, changed, without


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("remove", [False, True])
def test_a_far_token_and_its_removal_show_through_the_state(tmp_path, remove, dtype):
    raw, bf16, changed, without = build_far_state(remove)
    folder = str(tmp_path / "one")
    km.write_model(folder, raw, 0, tensors=bf16)
    tensors = plain.as_float64(bf16)
    want, reference = plain.logits(raw, tensors, changed), plain.logits(raw, tensors, without)
    assert spread_error(want[[250, 255]], reference[[250, 255]]).min() > 0.2, "the plain model itself"
    loaded = load(folder, dtype)
    for tag, steps in (("whole", [changed]), ("portions", cut(changed, [2, 70, 33, 16, 7])),
                       ("decoded", [changed[:6]] + [[t] for t in changed[6:]])):
        got = run_steps(loaded, [[(tag, part)] for part in steps])[tag]
        # (what is left of a large state after a removal is small: a float32 walk token by token is off by 3e-4 too)
        check(got, want, dtype, f"{tag}", slack=3.0 if dtype == "float32" else 1.0)
        assert spread_error(got[[250, 255]].astype(np.float64), reference[[250, 255]]).min() > 0.15
        loaded.step.end(tag)


@pytest.mark.parametrize("heads,dim,rank", [(1, 4, 3), (2, 8, 16), (3, 13, 1), (2, 32, 9), (2, 50, 33), (1, 72, 8), (1, 136, 64), (1, 200, 5)])
def test_head_sizes_and_ranks_of_the_delta_rule(tmp_path, heads, dim, rank):
    """One to thirty-two lanes a column of the state, head sizes that fill no vector width, ranks that are padded; portions
    that end before, on and behind the scan's chunks of eight."""
    raw = km.single_layer(km.delta(heads, dim, rank))
    folder = str(tmp_path / "one")
    raw, bf16 = km.write_model(folder, raw, 44)
    tokens = tokens_of(raw["vocab"], 61, 12)
    want = plain.logits(raw, plain.as_float64(bf16), tokens)
    loaded = load(folder, "float32")
    for tag, sizes in (("a", [61]), ("b", [8, 7, 9, 1, 16]), ("c", [2]), ("d", [23, 1, 3])):
        got = run_steps(loaded, [[(tag, part)] for part in cut(tokens, sizes)])[tag]
        check(got, want, "float32", f"{heads} heads of {dim}, rank {rank}, portions of {sizes}")
        loaded.step.end(tag)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("experts,top,ff,limit", [(4, 1, 24, 0.5), (8, 8, 40, 1.0), (40, 3, 96, 2.0), (64, 6, 16, 7.0), (3, 2, 20, 1.5)])
def test_experts_choices_and_limits(tmp_path, experts, top, ff, limit, dtype):
    """One layer whose feed-forward is a mixture: one choice, all experts chosen, more experts than a warp has lanes; in
    steps of few tokens (the experts' rows stream) and of many (pairs grouped by expert), which must agree."""
    raw = km.single_layer(km.delta(1, 8, 4), km.moe(experts, top, ff, limit=limit))
    folder = str(tmp_path / "one")
    raw, bf16 = km.write_model(folder, raw, 45)
    tokens = tokens_of(raw["vocab"], 150, 13)
    want = plain.logits(raw, plain.as_float64(bf16), tokens)
    loaded = load(folder, dtype)
    check(run_steps(loaded, [[("w", tokens)]])["w"], want, dtype, f"{experts} experts, {top} chosen, whole", routed=True)
    pieces = run_steps(loaded, [[("p", part)] for part in cut(tokens, [3, 16, 17, 1, 40])])["p"]
    check(pieces, want, dtype, f"{experts} experts, {top} chosen, portions", routed=True)


def test_the_correction_moves_the_choice_and_not_the_weights(tmp_path):
    """A correction that lifts two experts over all others: the engine chooses them and weighs them by their scores as
    they are, however small."""
    import torch
    raw = km.single_layer(km.delta(1, 8, 4), km.moe(6, 2, 16))
    bf16 = km.make_tensors(raw, 46)
    tokens = tokens_of(raw["vocab"], 30, 14)
    outputs = []
    for tag, correction in (("plain", [0.0] * 6), ("lifted", [0.0, 4.0, 0.0, 0.0, 4.5, 0.0])):
        bf16["l0.mlp.correction"] = torch.tensor(correction).to(torch.bfloat16)
        folder = str(tmp_path / tag)
        km.write_model(folder, raw, 0, tensors=bf16)
        want = plain.logits(raw, plain.as_float64(bf16), tokens)
        check(run_steps(load(folder, "float32"), [[("a", tokens)]])["a"], want, "float32", f"correction {tag}")
        outputs.append(want)
    h = np.random.default_rng(1).normal(size=(5, raw["width"]))
    assert set(np.unique(plain.route(plain.as_float64(bf16), "l0.mlp.", raw["layers"][0]["mlp"], h)[0])) == {1, 4}
    assert np.median(spread_error(outputs[0], outputs[1])) > 0.01


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
    assert '"architecture": "Kodupel"' in capsys.readouterr().out


# ------------------------------------------------------------------------------- configurations drawn at random
def random_config(rng):
    width = int(rng.choice([20, 36, 64, 100, 128]))
    layers, owners = [], []
    for index in range(int(rng.integers(1, 7))):
        pick = rng.random()
        if pick < 0.25 and owners:
            source = int(rng.choice(owners))
            m = layers[source]["mixer"]
            layer = km.attention(m["heads"], m["kv_heads"], m["dim"], m["vdim"], m.get("rot"),
                                 scale=float(rng.choice([0.1, 0.35])), kv_from=source)
        elif pick < 0.6:
            heads, groups = [(1, 1), (2, 1), (4, 2), (6, 2), (8, 8), (12, 3), (20, 1)][int(rng.integers(0, 7))]
            dim = int(rng.choice([4, 8, 12, 32, 64]))
            rot = None if rng.random() < 0.2 else km.rotation(
                float(rng.choice([50.0, 10000.0, 1e6])), 2 * int(rng.integers(1, dim // 2 + 1)),
                factor=None if rng.random() < 0.4 else float(rng.choice([2.0, 8.0])), original=int(rng.choice([32, 256, 4096])),
                fast=float(rng.choice([4.0, 32.0])), slow=float(rng.choice([0.5, 1.0])))
            layer = km.attention(heads, groups, dim, int(rng.choice([4, 9, 16, 64, 128])), rot,
                                 scale=float(rng.choice([dim ** -0.5, 0.125, 0.5])))
            owners.append(index)
        else:
            layer = km.delta(int(rng.integers(1, 5)), int(rng.choice([4, 9, 16, 32, 64, 130])), int(rng.choice([1, 8, 20])))
        experts = int(rng.choice([2, 3, 8, 16, 33, 70]))
        mlp = None if rng.random() < 0.25 else km.moe(experts, int(rng.integers(1, min(experts, 8) + 1)),
                                                      int(rng.choice([8, 20, 64])), limit=float(rng.choice([0.5, 1.5, 7.0])))
        layers.append(km.with_mlp(layer, mlp))
    return km.config(int(rng.integers(17, 300)), width, layers, eps=float(rng.choice([1e-5, 1e-6, 1e-3])),
                     scale=float(rng.choice([1.0, width ** 0.5, 3.0])))


@pytest.mark.parametrize("seed", range(12))
def test_configurations_drawn_at_random(tmp_path, seed):
    """Whole prompt, portions beside single tokens of a second request, and decoding, in both precisions."""
    rng = np.random.default_rng(3000 + seed)
    raw = random_config(rng)
    folder = str(tmp_path / "drawn")
    raw, bf16 = km.write_model(folder, raw, 700 + seed)
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
            check(whole, want["a"], dtype, f"{raw['layers']} whole")
            for key in ("a", "b"):
                check(got[key], want[key], dtype, f"{raw['layers']} request {key}")
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


DELTA_ONLY = km.config(70, 40, [km.with_mlp(km.delta(2, 8, 12), km.moe(3, 1, 24)), km.with_mlp(km.delta(1, 20, 4), None)])
ATTENTION_ONLY = km.config(90, 24, [
    km.with_mlp(km.attention(2, 2, 8, 4, km.rotation(300.0, 8)), None),
    km.with_mlp(km.attention(2, 2, 8, 4, km.rotation(300.0, 8), scale=0.4, kv_from=0), km.moe(3, 2, 8))])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["mixed", "odd", "delta_only", "attention_only"])
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
        raw, bf16 = km.write_model(folder, DELTA_ONLY if name == "delta_only" else ATTENTION_ONLY, 77)
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
        check(np.concatenate(rows[key]), plain.logits(raw, tensors, tokens), dtype, f"{name} request {key} replayed", routed=True)


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
    """Four layers 1,024 wide: sixteen recurrent heads of 64 with a decay of rank 64 and 32 experts of 512; sixteen query
    heads of 64 on four key heads; a layer that reads those keys and values; four recurrent heads of 128. The sizes at which
    the grouped tensor-core product, the tcgen05 prompt attention and the split-key decoding are what runs."""
    rot = km.rotation(300000.0, 32, factor=4.0, original=256, fast=32.0, slow=1.0)
    raw = km.config(4096, 1024, [
        km.with_mlp(km.delta(16, 64, 64), km.moe(32, 4, 512)),
        km.with_mlp(km.attention(16, 4, 64, 64, rot), km.moe(16, 2, 384, limit=2.0)),
        km.with_mlp(km.attention(16, 4, 64, 64, rot, scale=0.2, kv_from=1), None),
        km.with_mlp(km.delta(4, 128, 48), km.moe(8, 3, 320)),
    ])
    folder = str(tmp_path_factory.mktemp("kodupel_large") / "model")
    raw, bf16 = km.write_model(folder, raw, 91)
    tensors = plain.as_float64(bf16)
    first, second = tokens_of(raw["vocab"], 468, 500), tokens_of(raw["vocab"], 350, 501)
    return folder, raw, {"a": first, "b": second}, {"a": plain.logits(raw, tensors, first), "b": plain.logits(raw, tensors, second)}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_layers_of_a_real_model_size(large, dtype):
    folder, raw, requests, want = large
    first, second = requests["a"], requests["b"]
    loaded = load(folder, dtype, cache_tokens=2048, max_batched_tokens=1024, max_context=1024)
    steps = [[("a", first[:460])], [("a", first[460:461]), ("b", second[:200])], [("a", first[461:462]), ("b", second[200:])]]
    steps += [[("a", [t])] for t in first[462:]]
    got = run_steps(loaded, steps)
    for key in ("a", "b"):
        check(got[key], want[key], dtype, f"request {key} at a real model's layer sizes", routed=True)
