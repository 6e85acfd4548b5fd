"""The Kodupel design without a GPU: its configuration reader, its model description against the tensors a checkpoint
holds, its random-weights mode, and the plain float64 model against itself (the recurrence against its matrices written
out, the chunked form of it that the kernels use, the softmax with a one, stretched frequencies, the router)."""
from __future__ import annotations

import json
import math
import os

import numpy as np
import pytest

import kodupel_models as km
import plain_kodupel as plain
from celeg_b200.config import ConfigError, architecture_of
from celeg_b200.config.kodupel import KodupelConfig


def resolved(raw, seed):
    architecture = architecture_of(raw)
    made = {key: tuple(value.shape) for key, value in km.make_tensors(raw, seed).items()}
    return architecture, architecture.resolve_config(architecture.parse_config(km.stored(raw)), made), made


def test_configuration_round_trip_and_tensor_table():
    for name, (raw, seed) in km.CONFIGS.items():
        architecture, config, made = resolved(raw, seed)
        assert architecture.name == "Kodupel" and KodupelConfig.from_dict(config.to_dict()) == config
        spec = architecture.build_spec(config)
        assert {ref.name: tuple(ref.shape) for ref in spec.all_tensors()} == made, name


def test_every_constant_comes_from_the_configuration():
    raw, seed = km.CONFIGS["mixed"]
    _, config, _ = resolved(raw, seed)
    first, second, third, fourth = config.layers[:4]
    assert (first.heads, first.kv_heads, first.dim, first.vdim, first.scale) == (4, 2, 16, 32, 0.25)
    assert first.rotary.dims == 8 and first.rotary.scaling == (4.0, 64.0, 4.0, 0.5) and first.kv_from is None
    assert (second.heads, second.dim, second.decay_rank) == (2, 16, 12) and second.mlp.limit == pytest.approx(0.7)
    assert third.kv_from == 0 and third.scale == pytest.approx(0.4) and fourth.mlp is None and fourth.rotary.scaling is None
    assert config.embedding_scale == pytest.approx(8.0)
    spec = architecture_of(raw).build_spec(config)
    assert [entry.cache_of for entry in spec.order] == [None, None, 0, None, None, 3, 0]
    mixer = spec.layers[2].mixer
    assert mixer.params["reads_cache_only"] and "k" not in mixer.tensors and "v_bias" not in mixer.tensors
    assert spec.layers[1].feed_forward.params["gate_limit"] == pytest.approx(0.7)
    assert spec.layers[0].feed_forward.params["scores"] == "sigmoid" and not spec.layers[0].feed_forward.params["renormalize"]
    assert spec.layers[3].feed_forward is None and spec.layers[3].feed_forward_norm is None
    raw, seed = km.CONFIGS["odd"]
    _, config, _ = resolved(raw, seed)
    assert config.layers[4].rotary is None and config.layers[2].decay_rank == 1


def test_absent_entries_have_their_stated_defaults():
    raw = km.config(32, 24, [{"type": "attention", "mixer": {"heads": 4, "dim": 6}, "mlp": None}])
    layer = architecture_of(raw).parse_config(raw).layers[0]
    assert (layer.kv_heads, layer.vdim, layer.rotary, layer.kv_from) == (4, 6, None, None)
    assert layer.scale == pytest.approx(6 ** -0.5)


@pytest.mark.parametrize("damage,message", [
    (lambda raw: raw["layers"][0].update(type="sliding"), "unknown layer type"),
    (lambda raw: raw["layers"][0]["mixer"].update(kv_heads=3), "multiple"),
    (lambda raw: raw["layers"][0]["mixer"]["rot"].update(dims=7), "even"),
    (lambda raw: raw["layers"][0]["mixer"]["rot"].update(dims=32), "at most"),
    (lambda raw: raw["layers"][2]["mixer"].update(kv_from=2), "earlier layer"),
    (lambda raw: raw["layers"][2]["mixer"].update(kv_from=1), "no attention layer"),
    (lambda raw: raw["layers"][2]["mixer"].update(dim=16), "its own sizes"),
    (lambda raw: raw["layers"][3]["mixer"].update(kv_from=2), "no attention layer"),
    (lambda raw: raw["layers"][1]["mixer"].pop("dim"), "dim"),
    (lambda raw: raw["layers"][1]["mlp"]["router"].update(top=9), "exceeds"),
    (lambda raw: raw["layers"][1]["mlp"]["expert"].update(limit=0), "limit"),
    (lambda raw: raw["layers"][1]["mlp"].update(kind="dense"), "unknown kind"),
    (lambda raw: raw.pop("embedding"), "embedding"),
    (lambda raw: raw.pop("norm"), "norm"),
    (lambda raw: raw.update(layers=[]), "layers"),
])
def test_faulty_configurations_are_refused_with_a_message(damage, message):
    rot = km.rotation(100.0, 4)
    raw = km.stored(km.config(64, 32, [
        km.with_mlp(km.attention(4, 2, 8, 8, rot), None), km.with_mlp(km.delta(2, 8, 4), km.moe(8, 2, 16)),
        km.with_mlp(km.attention(4, 2, 8, 8, rot, kv_from=0), None), km.with_mlp(km.attention(4, 2, 8, 8, rot, kv_from=0), None)]))
    damage(raw)
    with pytest.raises(ConfigError, match=message):
        architecture_of(raw).parse_config(raw)


def test_a_rank_that_nothing_names_is_refused():
    raw = km.stored(km.single_layer(km.delta(2, 8, 4)))
    architecture = architecture_of(raw)
    with pytest.raises(ConfigError, match="rank"):
        architecture.build_spec(architecture.parse_config(raw))
    raw["layers"][0]["mixer"]["decay_rank"] = 6
    spec = architecture.build_spec(architecture.parse_config(raw))
    assert spec.layers[0].mixer.tensors["decay_up"].shape == (16, 6)


def test_random_weights_mode_writes_a_loadable_folder(tmp_path):
    from celeg_b200 import write_random_model
    from celeg_b200.weights.safetensors_io import TensorRepository
    raw = km.stored(km.MIXED)
    for layer, made in zip(raw["layers"], km.MIXED["layers"]):
        if "rank" in made:
            layer["mixer"]["decay_rank"] = made["rank"]
    folder = write_random_model(str(tmp_path / "random"), raw, seed=3)
    repository = TensorRepository(folder)
    architecture = architecture_of(raw)
    wanted = {ref.name: tuple(ref.shape) for ref in architecture.build_spec(architecture.parse_config(raw)).all_tensors()}
    assert {key: tuple(value) for key, value in repository.shapes().items()} == wanted
    assert abs(float(repository.tensor("l0.norm1").float().mean())) < 0.2          # the blocks' norm weights lie around zero
    for name in ("l1.mix.norm", "l0.mix.q.norm"):                                  # the mixers' lie around one
        assert 0.5 < float(repository.tensor(name).float().mean()) < 1.5
    repository.close()
    assert json.load(open(os.path.join(folder, "config.json")))["architecture"] == "Kodupel"


# ------------------------------------------------------------------------------------------ the plain model
def draws(tokens, dim, seed):
    rng = np.random.default_rng(seed)
    r, k, v = (rng.normal(size=(tokens, dim)) for _ in range(3))
    return r, k, v, rng.uniform(0.55, 1.0, size=(tokens, dim)), rng.uniform(0.0, 1.0, size=(tokens, dim))


def test_plain_delta_equals_its_transition_matrices_written_out():
    r, k, v, w, a = draws(9, 5, 1)
    want = np.zeros((9, 5))
    for t in range(9):
        state = np.zeros((5, 5))
        for s in range(t + 1):                       # token s's k v^T carried through the transitions after it
            carried = np.outer(k[s], v[s])
            for x in range(s + 1, t + 1):
                u = k[x] / np.sqrt((k[x] ** 2).sum() + 1e-6)
                carried = (np.diag(w[x]) - np.outer(a[x] * u, u)) @ carried
            state += carried
        want[t] = state.T @ r[t]
    assert np.allclose(plain.delta_states(r, k, v, w, a), want, rtol=1e-10, atol=1e-12)


def chunk_form(r, k, v, w, a, size):
    """The recurrence in chunks: all sums over the state are of the state before the chunk, the rest is a triangle."""
    tokens, dim = k.shape
    u = k / np.sqrt((k ** 2).sum(-1, keepdims=True) + 1e-6)
    b = a * u
    state, out = np.zeros((dim, dim)), np.zeros((tokens, dim))
    for t0 in range(0, tokens, size):
        at = range(t0, min(t0 + size, tokens))
        product = lambda first, last: np.prod(w[first:last + 1], axis=0) if last >= first else np.ones(dim)
        taken = {}
        for i in at:
            su = (u[i] * product(t0, i - 1)) @ state
            so = (r[i] * product(t0, i)) @ state
            for j in range(t0, i):
                p = product(j + 1, i - 1)
                su = su + ((u[i] * p) @ k[j]) * v[j] - ((u[i] * p) @ b[j]) * taken[j]
            taken[i] = su
            for j in range(t0, i + 1):
                p = product(j + 1, i)
                so = so + ((r[i] * p) @ k[j]) * v[j] - ((r[i] * p) @ b[j]) * taken[j]
            out[i] = so
        last = at[-1]
        state = product(t0, last)[:, None] * state + sum(
            np.outer(k[j] * product(j + 1, last), v[j]) - np.outer(b[j] * product(j + 1, last), taken[j]) for j in at)
    return out


@pytest.mark.parametrize("size", [1, 3, 8])
def test_the_chunked_form_is_the_same_recurrence(size):
    r, k, v, w, a = draws(21, 6, 2)
    assert np.allclose(chunk_form(r, k, v, w, a, size), plain.delta_states(r, k, v, w, a), rtol=1e-9, atol=1e-11)


def test_plain_decay_and_removal_stay_in_their_ranges():
    raw = km.single_layer(km.delta(2, 8, 3))
    tensors = plain.as_float64(km.make_tensors(raw, 3))
    h = 50.0 * np.random.default_rng(3).normal(size=(40, raw["width"]))
    decay, removal = plain.channel_decay(tensors, "l0.mix.", h), plain.removal_rate(tensors, "l0.mix.", h)
    assert math.exp(-math.exp(-0.5)) <= decay.min() and decay.max() <= 1.0 and 0.0 <= removal.min() <= removal.max() <= 1.0


def test_plain_softmax_with_a_one():
    weights = plain.weights_with_one(np.array([0.5, -2.0, 1.0]))
    e = np.exp([0.5, -2.0, 1.0])
    assert np.allclose(weights, e / (1.0 + e.sum()))
    assert plain.weights_with_one(np.array([-60.0])).sum() < 1e-20 and plain.weights_with_one(np.array([800.0])).sum() == pytest.approx(1.0)


def test_plain_stretched_frequencies_and_rotation():
    rot = km.rotation(100.0, 8, factor=4.0, original=64, fast=4.0, slow=0.5)
    frequencies, magnitude = plain.turn_frequencies(rot)
    untouched = 100.0 ** (-2.0 * np.arange(4) / 8)
    assert magnitude == pytest.approx(0.1 * math.log(4.0) + 1.0)
    lo = max(math.floor(8 * math.log(64 / (2 * math.pi * 4.0)) / (2 * math.log(100.0))), 0)
    hi = min(math.ceil(8 * math.log(64 / (2 * math.pi * 0.5)) / (2 * math.log(100.0))), 7)
    for i in range(4):
        share = min(max((i - lo) / (hi - lo), 0.0), 1.0)
        assert frequencies[i] == pytest.approx(untouched[i] * (share / 4.0 + 1.0 - share))
    x = np.random.default_rng(4).normal(size=(3, 2, 10))
    turned = plain.rotate(x, rot)
    assert np.allclose(turned[..., 8:], x[..., 8:]) and np.allclose(turned[0, :, :8], x[0, :, :8] * magnitude)
    c, s = math.cos(2 * frequencies[1]) * magnitude, math.sin(2 * frequencies[1]) * magnitude
    assert np.allclose(turned[2, :, 2], x[2, :, 2] * c - x[2, :, 3] * s)
    assert np.allclose(turned[2, :, 3], x[2, :, 3] * c + x[2, :, 2] * s)


def test_plain_router_chooses_with_the_correction_and_weighs_without_it():
    tensors = {"m.router": np.eye(4), "m.correction": np.array([0.0, 0.9, 0.0, -0.9])}
    chosen, weights = plain.route(tensors, "m.", {"router": {"top": 2}}, np.array([[0.1, -1.0, 0.2, 3.0]]))
    assert chosen[0].tolist() == [1, 2] and np.allclose(weights[0], plain.sigmoid(np.array([-1.0, 0.2])))


def test_plain_expert_is_clamped_on_its_sides():
    tensors = {"e.gate": np.array([[1.0]]), "e.up": np.array([[2.0]]), "e.down": np.array([[1.0]])}
    out = plain.clamped_expert(tensors, "e.", np.array([[5.0], [-5.0]]), 1.5)[:, 0]
    g = np.array([1.5, -5.0])                       # the gate is cut off above only, the up value at both ends
    assert np.allclose(out, g / (1.0 + np.exp(-1.702 * g)) * (np.array([1.5, -1.5]) + 1.0))


def test_plain_streams_share_keys_and_values():
    """A layer with ``kv_from`` gives what a layer with the same tensors of its own would give on the source's input."""
    rot = km.rotation(100.0, 4)
    raw = km.config(40, 24, [km.with_mlp(km.attention(4, 2, 8, 6, rot), None), km.with_mlp(km.attention(4, 2, 8, 6, rot, kv_from=0), None)])
    tensors = plain.as_float64(km.make_tensors(raw, 9))
    tokens = np.random.default_rng(5).integers(0, 40, size=11).tolist()
    first, second = plain.streams(raw, tensors, tokens)
    x0 = plain.embed(raw, tensors, tokens)
    k, v = plain.keys_and_values(tensors, "l0.mix.", raw["layers"][0]["mixer"], x0, 1e-5)
    mixed = plain.attention(tensors, "l1.mix.", raw["layers"][1]["mixer"], first, k, v, 1e-5)
    assert np.allclose(second, first + plain.offset_norm(mixed, tensors["l1.norm1"], 1e-5))
