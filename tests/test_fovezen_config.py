"""The Fovezen design without a GPU: its configuration reader, its model description against the tensors a checkpoint
holds, its random-weights mode, and the plain float64 model against itself (the connections against one stream, the
recurrences against sums written out and against the chunked form that the kernels use, the convolution, the window, the
cap, stretched frequencies, the run order)."""
from __future__ import annotations

import json
import math
import os

import numpy as np
import pytest

import fovezen_models as fm
import plain_fovezen as plain
from celeg_b200.config import ConfigError, architecture_of
from celeg_b200.config.fovezen import FovezenConfig


def resolved(raw, seed):
    architecture = architecture_of(raw)
    made = {key: tuple(value.shape) for key, value in fm.make_tensors(raw, seed).items()}
    return architecture, architecture.resolve_config(architecture.parse_config(fm.stored(raw)), made), made


def test_configuration_round_trip_and_tensor_table():
    for name, (raw, seed) in fm.CONFIGS.items():
        architecture, config, made = resolved(raw, seed)
        assert architecture.name == "Fovezen" and FovezenConfig.from_dict(config.to_dict()) == config
        spec = architecture.build_spec(config)
        assert {ref.name: tuple(ref.shape) for ref in spec.all_tensors()} == made, name


def test_every_constant_comes_from_the_configuration():
    raw, seed = fm.CONFIGS["mixed"]
    _, config, _ = resolved(raw, seed)
    first, second, third, fourth = config.layers
    left = first.softmax
    assert (left.heads, left.kv_heads, left.dim, left.vdim, left.taps, left.window, left.softcap) == (4, 2, 16, 24, 4, 11, 5.0)
    assert left.scale == pytest.approx(0.4) and left.rotary is None
    assert (first.linear.heads, first.linear.dim, first.linear.vdim, first.linear.tau, first.linear.decay_rank) == (2, 16, 24, 4.0, 12)
    m = second.state_space
    assert (m.heads, m.vdim, m.state, m.groups, m.taps, m.norm_groups) == (4, 16, 24, 2, 2, 2)
    assert second.mlp.limit == pytest.approx(0.7) and third.mlp is None
    assert third.softmax.rotary.dims == 8 and third.softmax.rotary.scaling == (4.0, 1.0, 4.0, 64.0)
    assert third.softmax.taps is None and third.softmax.window is None and third.softmax.softcap is None
    assert config.streams == 3 and config.logit_scale == pytest.approx(0.7) and config.loop == (1, 3, 2)
    spec = architecture_of(raw).build_spec(config)
    assert [entry.layer for entry in spec.order] == [0, 1, 2, 1, 2, 3] and all(e.cache_of is None for e in spec.order)
    assert spec.layers[1].feed_forward.params["gate_limit"] == pytest.approx(0.7)
    assert spec.layers[2].feed_forward is None and "feed_forward_connection" not in spec.layers[2].extra_parts
    assert spec.layers[0].extra_parts["mixer_connection"].params["streams"] == 3
    assert spec.layers[0].mixer.parts["left"].params["softcap"] == 5.0
    assert spec.logits_multiplier == pytest.approx(0.7)
    assert resolved(*fm.CONFIGS["odd"])[1].run_order() == (0, 1, 0, 1, 0, 1, 2, 3)


def test_absent_entries_have_their_stated_defaults():
    raw = fm.config(32, 24, [
        {"type": "attention", "mixer": {"heads": 4, "dim": 6}, "mlp": None},
        {"type": "parallel", "mlp": None, "mixer": {"left": {"heads": 2, "dim": 5}, "right": {"heads": 1, "dim": 4, "tau": 2}}},
        {"type": "mamba2", "mlp": None, "mixer": {"heads": 2, "vdim": 4, "state": 3, "conv": 2}}])
    del raw["streams"], raw["logit_scale"]
    config = architecture_of(raw).parse_config(raw)
    first, second, third = config.layers
    assert (first.softmax.kv_heads, first.softmax.vdim, first.softmax.rotary) == (4, 6, None)
    assert first.softmax.scale == pytest.approx(6 ** -0.5)
    assert (second.softmax.taps, second.softmax.window, second.softmax.softcap, second.linear.vdim) == (None, None, None, 4)
    assert (third.state_space.groups, third.state_space.norm_groups) == (1, 1)
    assert (config.streams, config.logit_scale, config.loop) == (1, 1.0, None)


@pytest.mark.parametrize("damage,message", [
    (lambda raw: raw["layers"][0].update(type="sliding"), "unknown layer type"),
    (lambda raw: raw["layers"][0]["mixer"].update(kv_heads=3), "multiple"),
    (lambda raw: raw["layers"][0]["mixer"]["rot"].update(dims=7), "even"),
    (lambda raw: raw["layers"][0]["mixer"]["rot"].update(dims=32), "at most"),
    (lambda raw: raw["layers"][1]["mixer"].update(groups=3), "multiple"),
    (lambda raw: raw["layers"][1]["mixer"].update(norm_groups=3), "multiple"),
    (lambda raw: raw["layers"][1]["mixer"].update(conv=17), "exceed"),
    (lambda raw: raw["layers"][1]["mixer"].pop("state"), "state"),
    (lambda raw: raw["layers"][2]["mixer"].pop("right"), "right"),
    (lambda raw: raw["layers"][2]["mixer"]["left"].update(softcap=0), "positive"),
    (lambda raw: raw["layers"][2]["mixer"]["left"]["mask"].update(size=0), "positive"),
    (lambda raw: raw["layers"][2]["mixer"]["right"].update(tau=-1.0), "positive"),
    (lambda raw: raw["layers"][1]["mlp"].update(limit=0), "limit"),
    (lambda raw: raw["layers"][1]["mlp"].update(kind="moe"), "unknown kind"),
    (lambda raw: raw.update(streams=0), "positive"),
    (lambda raw: raw.update(streams=17), "exceed"),
    (lambda raw: raw.update(loop={"start": 1, "stop": 4, "times": 2}), "loop"),
    (lambda raw: raw.update(loop={"start": 1, "stop": 2, "times": 0}), "loop"),
    (lambda raw: raw.pop("norm"), "norm"),
    (lambda raw: raw.update(layers=[]), "layers"),
])
def test_faulty_configurations_are_refused_with_a_message(damage, message):
    raw = fm.stored(fm.config(64, 32, [
        fm.with_mlp(fm.attention(4, 2, 8, 8, fm.rotation(100.0, 4)), None), fm.with_mlp(fm.mamba(4, 4, 8, 2, 4, 2), 16),
        fm.with_mlp(fm.parallel((2, 1, 8, 8, 2, 6, 3.0, 0.3), (1, 4, 4, 2.0, 4)), None)]))
    damage(raw)
    with pytest.raises(ConfigError, match=message):
        architecture_of(raw).parse_config(raw)


def test_a_rank_that_nothing_names_is_refused():
    raw = fm.stored(fm.single_layer(fm.parallel((2, 1, 8, 8, 2, 6, 3.0, 0.3), (1, 4, 4, 2.0, 4))))
    architecture = architecture_of(raw)
    with pytest.raises(ConfigError, match="rank"):
        architecture.build_spec(architecture.parse_config(raw))
    raw["layers"][0]["mixer"]["right"]["decay_rank"] = 6
    spec = architecture.build_spec(architecture.parse_config(raw))
    assert spec.layers[0].mixer.parts["right"].tensors["decay_up"].shape == (4, 6)


def test_random_weights_mode_writes_a_loadable_folder(tmp_path):
    from celeg_b200 import write_random_model
    from celeg_b200.weights.safetensors_io import TensorRepository
    raw = fm.stored(fm.MIXED)
    for layer, made in zip(raw["layers"], fm.MIXED["layers"]):
        if "rank" in made:
            layer["mixer"]["right"]["decay_rank"] = made["rank"]
    folder = write_random_model(str(tmp_path / "random"), raw, seed=3)
    repository = TensorRepository(folder)
    architecture = architecture_of(raw)
    wanted = {ref.name: tuple(ref.shape) for ref in architecture.build_spec(architecture.parse_config(raw)).all_tensors()}
    assert {key: tuple(value) for key, value in repository.shapes().items()} == wanted
    assert abs(float(repository.tensor("l0.norm1").float().mean())) < 0.2          # the blocks' norm weights lie around zero
    for name in ("l1.mix.norm", "l0.mix.left.q.norm", "l0.mix.left.out", "l1.mix.D"):      # the mixers' lie around one
        assert 0.5 < float(repository.tensor(name).float().mean()) < 1.5, name
    repository.close()
    assert json.load(open(os.path.join(folder, "config.json")))["architecture"] == "Fovezen"


# ------------------------------------------------------------------------------------------ the plain model
def test_streams_that_are_never_told_apart_are_one_stream():
    """Connections whose columns and shares are alike keep all streams equal: the model is then a pre-norm model of one
    stream with a factor on what a sublayer reads and puts out."""
    raw = dict(fm.MIXED)
    tensors = plain.as_float64(fm.make_tensors(raw, 5))
    one = dict(raw, streams=1)
    single = dict(tensors)
    for key in tensors:
        if ".hc" not in key:
            continue
        n = raw["streams"]
        if key.endswith(".mix"):
            tensors[key], single[key] = np.full((n, n), 0.3), np.full((1, 1), 0.9)
        elif key.endswith(".in"):
            tensors[key], single[key] = np.array([0.5, -0.2, 0.4]), np.array([0.7])
        else:
            tensors[key], single[key] = np.full(n, 0.8), np.full(1, 0.8)
    tokens = np.random.default_rng(1).integers(0, raw["vocab"], size=12)
    both = plain.streams(raw, tensors, tokens), plain.streams(one, single, tokens)
    for a, b in zip(*both):
        np.testing.assert_allclose(a, 3.0 * b, rtol=1e-10, atol=1e-10)


def test_connections_are_indexed_from_to():
    copies = np.arange(6.0).reshape(2, 1, 3)
    mix, out, y = np.array([[1.0, 10.0], [100.0, 1000.0]]), np.array([0.5, -1.0]), np.ones((1, 3))
    got = plain.spread(copies, mix, out, y)
    np.testing.assert_allclose(got[0], copies[0] + 100.0 * copies[1] + 0.5)
    np.testing.assert_allclose(got[1], 10.0 * copies[0] + 1000.0 * copies[1] - 1.0)
    np.testing.assert_allclose(plain.gathered(copies, np.array([2.0, -1.0])), 2.0 * copies[0] - copies[1])


def test_decayed_states_are_sums_of_outer_products():
    rng = np.random.default_rng(2)
    k, q, v = rng.normal(size=(9, 4)), rng.normal(size=(9, 4)), rng.normal(size=(9, 3))
    for decays in (rng.uniform(0.0, 1.0, size=(9, 4)), rng.uniform(0.0, 1.0, size=9)):
        wide = np.broadcast_to(np.reshape(decays, (9, -1)), (9, 4))
        got = plain.decayed_states(k, v, decays, q)
        for i in range(9):
            want = sum(float((q[i] * np.prod(wide[j + 1:i + 1], axis=0)) @ k[j]) * v[j] for j in range(i + 1))
            np.testing.assert_allclose(got[i], want, rtol=1e-10, atol=1e-12)


def test_blocks_of_eight_taken_to_their_middles_give_the_same_sums():
    """The form that the kernels use for a decay a channel: within blocks of eight tokens queries and keys stand at the
    block's middle, between blocks a factor a channel joins; decays as small as 1e-7 among them."""
    rng = np.random.default_rng(3)
    n, dim = 40, 6
    q, k, v = (rng.normal(size=(n, dim)) for _ in range(3))
    a = rng.uniform(0.0, 1.0, size=(n, dim)) ** 3
    a[5:9] = 1e-7
    want = plain.decayed_states(k, v, a, q)
    qm, km, upper, lower = q.copy(), k.copy(), [], []
    for b in range(0, n, 8):
        up, down = np.ones(dim), np.ones(dim)
        for i in range(3, -1, -1):
            qm[b + i], km[b + i] = q[b + i] / up, k[b + i] * up
            up = up * a[b + i]
        for i in range(4, 8):
            down = down * a[b + i]
            qm[b + i], km[b + i] = q[b + i] * down, k[b + i] / down
        upper.append(up)
        lower.append(down)
    products = np.zeros((n, n))
    for i in range(n):
        for j in range(i + 1):
            I, J = i // 8, j // 8
            w = np.ones(dim) if I == J else lower[J] * upper[I]
            for between in range(J + 1, I):
                w = w * upper[between] * lower[between]
            products[i, j] = (qm[i] * w) @ km[j]
    np.testing.assert_allclose(products @ v, want, rtol=1e-8, atol=1e-10)


def test_convolution_by_hand():
    u = np.array([[1.0], [2.0], [4.0], [8.0]])
    got = plain.causal_convolution(u, np.array([[100.0, 10.0, 1.0]]), np.array([0.5]))
    np.testing.assert_allclose(got[:, 0], [1.5, 12.5, 124.5, 248.5])


def test_window_cap_and_grouping():
    assert [plain.visible_from(i, 4) for i in (0, 3, 4, 9)] == [0, 0, 1, 6] and plain.visible_from(7, None) == 0
    np.testing.assert_allclose(plain.capped(np.array([0.0, 1e3, -1e3, 0.01]), 5.0), [0.0, 5.0, -5.0, 0.01], rtol=1e-5)
    rng = np.random.default_rng(4)
    q, k, v = rng.normal(size=(6, 4, 3)), rng.normal(size=(6, 2, 3)), rng.normal(size=(6, 2, 5))
    got = plain.attend(q, k, v, 0.7, 2.0, 3).reshape(6, 4, 5)
    scores = 2.0 * np.tanh(0.7 * k[2:5, 1] @ q[4, 3] / 2.0)
    np.testing.assert_allclose(got[4, 3], np.exp(scores) @ v[2:5, 1] / np.exp(scores).sum())


def test_stretched_frequencies():
    plainly = plain.turn_frequencies({"base": 10000.0, "dims": 16})
    np.testing.assert_allclose(plainly, 10000.0 ** (-np.arange(8) / 8.0))
    scaled = plain.turn_frequencies({"base": 10000.0, "dims": 16, "scaling": {"factor": 4.0, "low": 1.0, "high": 4.0, "original": 64}})
    waves = 2.0 * math.pi / plainly
    for f, g, wave in zip(plainly, scaled, waves):
        if wave < 16.0:
            assert g == f
        elif wave > 64.0:
            assert g == pytest.approx(f / 4.0)
        else:
            assert f / 4.0 < g < f
    assert (waves < 16.0).any() and (waves > 64.0).any() and ((waves >= 16.0) & (waves <= 64.0)).any()


def test_the_gate_comes_before_the_norm_and_parts_have_their_own_root():
    raw = fm.single_layer(fm.mamba(4, 4, 3, 2, 2, 2), width=20)
    tensors = plain.as_float64(fm.make_tensors(raw, 6))
    h = np.random.default_rng(5).normal(size=(7, 20))
    base, m = "l0.mix.", raw["layers"][0]["mixer"]
    whole = plain.mamba2(tensors, base, m, h, 1e-5)
    scaled = dict(tensors)
    scaled[base + "norm"] = tensors[base + "norm"] * np.repeat([1.0, 0.0], 8)
    half = plain.mamba2(scaled, base, m, h, 1e-5)
    # what the first part makes does not hang on the second part's size: its share of z made large changes nothing here
    rows = tensors[base + "in"].copy()
    rows[8:16] *= 3.0
    again = plain.mamba2(dict(scaled, **{base + "in": rows}), base, m, h, 1e-5)
    np.testing.assert_allclose(half, again, rtol=1e-10)
    assert np.abs(whole - half).max() > 1e-3
