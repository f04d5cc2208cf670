"""Tosipel on the CPU: registry, configuration errors, tensor names and shapes, layers that run another layer's tensors, cache
groups, seeded folders, and the plain implementation against second formulations of its mechanisms."""

from __future__ import annotations

import copy
import json

import numpy as np
import pytest

from gunedra_helpers import as_float64
from plain import tosipel_plain as plain
from tosipel_helpers import ALPHA, BETA, CONFIGS, DELTA, GAMMA, draw_weights


def parsed(raw):
    from llm_inference_b200 import models  # noqa: F401
    from llm_inference_b200.config.registry import parse_config

    return parse_config(json.loads(json.dumps(raw)))


def built(raw):
    from llm_inference_b200.parts.model import Model

    entry, config = parsed(raw)
    return Model(entry.recipe(config))


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_configuration_round_trip_and_tensor_names(name):
    raw = CONFIGS[name]
    entry, config = parsed(raw)
    assert entry.name == "Tosipel" and config.to_json_dict() == raw
    specs = {spec.name: spec for spec in built(raw).tensor_specs()}
    weights = draw_weights(raw, 3)
    assert all(specs[n].fits(tuple(t.shape)) for n, t in weights.items())
    assert {n for n, s in specs.items() if not s.optional} == set(weights)
    # a layer without feed-forward reads past the norm of one
    assert {n for n, s in specs.items() if s.optional} == {
        f"l{i}.norm2" for i, layer in enumerate(raw["layers"]) if layer["mlp"] is None and layer.get("weights_of") is None}


def test_recipe_reads_every_size_from_the_configuration():
    model = built(ALPHA)
    assert len(model.blocks) == 4 and [(c.layer, c.cache_id) for c in model.schedule] == [(0, 0), (1, 1), (2, 2), (3, 3), (0, 4), (3, 5), (2, 6)]
    assert model.embedding.scale == 3.0 and model.final_norm.around_zero and model.head.tied_to is None
    attention, delta, latent, _ = (block.mixer for block in model.blocks)
    assert (attention.heads, attention.kv_heads, attention.dim, attention.vdim, attention.row_dim, attention.scale, attention.window) == (6, 2, 16, 24, 64, 0.5, 20)
    assert attention.qk_norm and attention.has_sink and attention.gate == "head" and not attention.qk_bias and not attention.has_out_bias
    assert (attention.position.rotary_dims, attention.position.theta, attention.position.interleaved) == (8, 100.0, False)
    assert (latent.heads, latent.dim, latent.vdim, latent.rank, latent.q_rank, latent.rot_dim, latent.scale) == (3, 12, 20, 28, 36, 0, 0.4)
    assert latent.position is None and not latent.has_sink and not latent.has_gate
    assert (delta.heads, delta.kv_heads, delta.dim, delta.vdim, delta.taps, delta.eps) == (6, 3, 12, 20, 4, 1e-5)
    assert model.blocks[1].feed_forward is None and model.blocks[2].feed_forward.intermediate_size == 60
    assert model.blocks[0].mult == 1.0 and model.blocks[0].mixer_norm.around_zero and model.blocks[0].scales == [None, None]
    second = built(BETA)
    assert second.blocks[1].mixer.window == 0 and second.blocks[1].mixer.position is None and second.blocks[3].mixer.window == 1
    assert [(c.layer, c.cache_id) for c in second.schedule][-2:] == [(1, 5), (1, 6)]  # a chain of layers ends at the one with tensors
    assert second.blocks[2].mixer.taps == 1 and second.embedding.scale == 1.0 and second.blocks[0].mixer_norm.eps == 3e-4


def test_absent_keys_are_absent_mechanisms():
    raw = copy.deepcopy(DELTA)
    del raw["embedding"]
    del raw["layers"][2]["mixer"]["mask"]
    raw["layers"][2]["mixer"]["rot"]["dims"] = 0
    model = built(raw)
    assert model.embedding.scale == 1.0 and model.blocks[2].mixer.window == 0 and model.blocks[2].mixer.position is None


def test_layers_on_shared_tensors_have_caches_and_states_of_their_own():
    import torch

    from llm_inference_b200.cache.paged_cache import PagedCache
    from llm_inference_b200.parts import StateSpec

    specs = built(ALPHA).cache_specs()
    assert sorted(specs) == list(range(7))
    assert specs[0] == specs[4] and specs[0].window == 20 and specs[2] == specs[6] and (specs[2].planes, specs[2].head_dim) == (1, 28)
    assert isinstance(specs[3], StateSpec) and specs[3] == specs[5] and specs[1].shapes == ((6, 12, 20), (3, 2 * 3 * 12 + 6 * 20))
    cache = PagedCache(specs, dtype=torch.float32, device="cpu", page_size=8, max_num_sequences=2, max_model_length=128, step_tokens=16, num_pages=16)
    assert {(g.spec.window, g.spec.planes): sorted(g.entries) for g in cache.groups} == {(20, 2): [0, 4], (0, 1): [2, 6]}
    assert sorted(cache.states) == [1, 3, 5] and cache.states[3][0].data_ptr() != cache.states[5][0].data_ptr()
    assert built(BETA).cache_specs()[2].shapes[1] == (0, 2 * 15 + 9 * 19)  # one tap: no history
    groups = PagedCache(built(GAMMA).cache_specs(), dtype=torch.float32, device="cpu", page_size=8, max_num_sequences=2, max_model_length=128,
                        step_tokens=16, num_pages=16).groups
    assert {(g.spec.window, g.spec.kv_heads, g.spec.head_dim, g.spec.planes) for g in groups} == {(45, 2, 64, 2), (0, 1, 96, 1), (70, 2, 128, 2), (31, 1, 192, 2)}


ERRORS = [
    (lambda c: c.pop("vocab"), "vocab"),
    (lambda c: c.pop("norm"), "norm"),
    (lambda c: c["norm"].update(eps=0.0), "eps"),
    (lambda c: c["embedding"].update(scale=float("inf")), "scale"),
    (lambda c: c.update(layers=[]), "layers"),
    (lambda c: c["layers"][0].update(type="other"), "type"),
    (lambda c: c["layers"][0].update(mixer=None), "mixer"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=4), "multiple"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "size"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), "dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=18), "dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(base=0.0), "base"),
    (lambda c: c["layers"][2]["mixer"].pop("q_rank"), "q_rank"),
    (lambda c: c["layers"][2]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][1]["mixer"].update(conv=0), "conv"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=4), "multiple"),
    (lambda c: c["layers"][2]["mlp"].update(kind="moe"), "kind"),
    (lambda c: c["layers"][2]["mlp"].update(ff=0), "ff"),
    (lambda c: c["layers"][4].update(weights_of=9), "weights_of"),
    (lambda c: c["layers"][4].update(weights_of=1), "equal"),
    (lambda c: c["layers"][4].update(mlp=None), "equal"),
    (lambda c: c["layers"][0].update(weights_of=4), "circle"),
]


@pytest.mark.parametrize("change,message", ERRORS)
def test_configuration_errors(change, message):
    from llm_inference_b200.config import ConfigError

    raw = copy.deepcopy(ALPHA)
    change(raw)
    with pytest.raises(ConfigError, match=message):
        parsed(raw)


def test_parts_refuse_what_does_not_go_together():
    from llm_inference_b200.parts import PartSpec, build_part

    sizes = dict(prefix="m.", hidden_size=32, heads=2, dim=8, vdim=8, scale=0.3, eps=1e-5)
    with pytest.raises(ValueError, match="sink"):
        build_part("mixer", PartSpec("shaped_attention", dict(sizes, kv_heads=1, sink=True, weights="sigmoid")))
    with pytest.raises(ValueError, match="position"):
        build_part("mixer", PartSpec("latent_attention", dict(sizes, rot_dim=4, rank=16)))
    with pytest.raises(ValueError, match="heads"):
        build_part("mixer", PartSpec("head_delta", dict(prefix="m.", hidden_size=32, heads=3, kv_heads=2, dim=8, vdim=8, taps=4, eps=1e-5)))


def test_seeded_folder_loads_back(tmp_path):
    import torch

    from llm_inference_b200.weights.loader import load_weights
    from llm_inference_b200.weights.random_init import write_model_folder

    _, config = parsed(ALPHA)
    write_model_folder(tmp_path, config, 5)
    model = built(json.loads((tmp_path / "config.json").read_text()))
    tensors = load_weights(tmp_path, model.tensor_specs())
    model.load(tensors, torch.float32, "cpu")
    block = model.blocks[0]
    assert torch.equal(block.mixer_norm.weight, tensors["l0.norm1"].float() + 1.0)
    assert torch.equal(block.mixer.shape.sink, tensors["l0.mix.sink"].float())
    gate_up = block.feed_forward.w_gate_up  # gate and up rows in turn
    assert torch.equal(gate_up[0::2], tensors["l0.mlp.gate"].float()) and torch.equal(gate_up[1::2], tensors["l0.mlp.up"].float())
    w_in = model.blocks[1].mixer.w_in  # [q | k | v | b | a | g]
    assert w_in.shape[0] == 36 + 36 + 120 + 6 + 6 + 120 and torch.equal(w_in[198:204], tensors["l1.mix.a"].float())
    assert model.blocks[2].mixer.w_in.shape == (36 + 28, 48)


# --- the plain implementation against second formulations ---------------------------------------------


@pytest.mark.parametrize("size", [None, 1, 3, 30])
def test_attention_as_masked_matrices_with_an_extra_column(size):
    """The sink is one more score in every row whose value is zero."""
    rng = np.random.default_rng(1)
    n, heads, groups, d, e = 17, 4, 2, 6, 5
    q, k, v = rng.normal(size=(n, heads, d)), rng.normal(size=(n, groups, d)), rng.normal(size=(n, groups, e))
    sink = rng.normal(0, 2, heads)
    got = plain.attend(q, k, v, np.arange(n), 0.7, {"size": size} if size else None, sink)
    i, j = np.arange(n)[:, None], np.arange(n)[None, :]
    seen = (j <= i) & (i - j < (size or n))
    for h in range(heads):
        scores = np.where(seen, 0.7 * q[:, h] @ k[:, h // 2].T, -np.inf)
        e_all = np.exp(np.concatenate([scores, np.full((n, 1), sink[h])], axis=1))
        np.testing.assert_allclose(got[:, h], e_all[:, :n] @ v[:, h // 2] / e_all.sum(1, keepdims=True), atol=1e-12)


def test_rotation_as_complex_numbers():
    rng = np.random.default_rng(2)
    x, positions = rng.normal(size=(9, 2, 10)), np.arange(9) * 7
    got = plain.rotate_halves(x, positions, {"dims": 6, "base": 50.0})
    turned = (x[..., :3] + 1j * x[..., 3:6]) * np.exp(1j * positions[:, None, None] * 50.0 ** (-np.arange(3) / 3.0))
    np.testing.assert_allclose(got, np.concatenate([turned.real, turned.imag, x[..., 6:]], axis=-1), atol=1e-12)


def test_delta_step_replaces_what_the_state_holds_for_a_key():
    """With a unit key, beta one and no decay, reading the key back gives exactly the value written; with a decay the state is
    g (I - beta k k^T) S + beta k v^T."""
    rng = np.random.default_rng(3)
    S, k, q, v = rng.normal(size=(6, 4)), rng.normal(size=6), rng.normal(size=6), rng.normal(size=4)
    k /= np.linalg.norm(k)
    new, out = plain.delta_step(S, k, k, v, 1.0, 1.0)
    np.testing.assert_allclose(out, v, atol=1e-12)
    new, out = plain.delta_step(S, q, k, v, 0.8, 0.3)
    np.testing.assert_allclose(new, 0.8 * (np.eye(6) - 0.3 * np.outer(k, k)) @ S + 0.3 * np.outer(k, v), atol=1e-12)
    np.testing.assert_allclose(out, new.T @ q, atol=1e-12)


def test_short_convolution_as_a_sum_over_shifted_rows():
    rng = np.random.default_rng(4)
    x, taps = rng.normal(size=(11, 3)), rng.normal(size=(3, 4))
    padded = np.concatenate([np.zeros((3, 3)), x])
    want = sum(taps[:, j] * padded[j : j + 11] for j in range(4))
    np.testing.assert_allclose(plain.short_convolution(x, taps, {}, "x"), want / (1 + np.exp(-want)), atol=1e-12)


def test_gelu_and_norms():
    z = np.linspace(-6, 6, 41)
    y = np.sqrt(2 / np.pi) * (z + 0.044715 * z**3)
    np.testing.assert_allclose(plain.gelu_tanh(z), z / (1 + np.exp(-2 * y)), atol=1e-12)
    x = np.random.default_rng(5).normal(size=(3, 8))
    np.testing.assert_allclose((plain.offset_norm(x, np.zeros(8), 0.0) ** 2).mean(-1), 1.0)
    np.testing.assert_allclose(plain.plain_norm(x, np.full(8, 2.0), 0.5), 2 * x / np.sqrt((x**2).mean(-1, keepdims=True) + 0.5))


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_whole_model_in_portions_and_token_by_token(name):
    config = CONFIGS[name]
    w = as_float64(draw_weights(config, 7))
    tokens = np.random.default_rng(1).integers(0, config["vocab"], 30)
    whole = plain.forward(config, w, tokens)
    for sizes in ((1,) * 30, (7, 2, 11, 1, 9)):
        state, parts, at = {}, [], 0
        for size in sizes:
            parts.append(plain.forward(config, w, tokens[at : at + size], state))
            at += size
        np.testing.assert_allclose(np.concatenate(parts), whole, atol=1e-8)
