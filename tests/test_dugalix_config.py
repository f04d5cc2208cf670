"""Dugalix on the CPU: registry, configuration errors, tensor names and shapes, seeded folders, the cache groups of
windows that keep first tokens, and the plain implementation against second formulations of its mechanisms."""

from __future__ import annotations

import copy
import itertools
import json

import numpy as np
import pytest

from dugalix_helpers import ALPHA, BETA, CONFIGS, GAMMA, draw_weights, memory, moe, softmax_attention
from gunedra_helpers import as_float64
from plain import dugalix_plain as plain


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
    assert entry.name == "Dugalix" and config.to_json_dict() == raw
    specs = {spec.name: spec for spec in built(raw).tensor_specs()}
    weights = draw_weights(raw, 3)
    assert all(specs[n].fits(tuple(t.shape)) for n, t in weights.items())
    assert {n for n, s in specs.items() if not s.optional} == set(weights)
    # a layer without feed-forward reads past the norms of one
    assert {n for n, s in specs.items() if s.optional} == {
        f"l{i}.{norm}" for i, layer in enumerate(raw["layers"]) if layer["mlp"] is None for norm in ("norm2", "norm2b")}


def test_recipe_reads_every_size_from_the_configuration():
    model = built(BETA)
    first, second, third, fourth = model.blocks
    assert (first.mult, first.mixer.heads, first.mixer.dim, first.mixer.scale, first.mixer.window) == (1.0, 1, 6, 1.2, 0)
    assert first.mixer.sigmoid and first.mixer.values_from_keys and first.mixer.position is None and not first.mixer.qk_bias
    ff = first.feed_forward
    assert (ff.experts, ff.identity, ff.choices, ff.top, ff.shared_size, ff.shared_gate, ff.group_count, ff.gated) == (1, 3, 4, 1, 9, True, 1, False)
    left, right = second.mixer.members
    assert (left.heads, left.kv_heads, left.dim, left.vdim, left.row_dim, left.window, left.keep_first) == (3, 3, 8, 136, 192, 4, 11)
    assert left.qk_bias and left.v_bias and left.has_out_bias and not left.adds_out_bias and not left.sigmoid and not left.qk_norm
    assert left.position.stretch == 1.5 and left.position.rotary_dims == 4 and left.position.theta == 10.0
    assert (right.heads, right.dim, right.vdim, right.gate_cap, right.eps) == (1, 5, 7, 15.0, 3e-4)
    assert second.mixer.scales == (1.0, 1.0) and third.mixer.scales == (0.3, -2.0)
    assert third.mixer.members[0].window == 0 and third.mixer.members[0].position is None
    assert third.feed_forward.intermediate_size == 33 and fourth.feed_forward is None and fourth.mixer.window == 1
    assert built(ALPHA).blocks[0].mult == 0.7 and built(GAMMA).blocks[0].mixer_norm.around_zero


def test_windows_with_kept_tokens_form_cache_groups_of_their_own():
    import torch

    from llm_inference_b200.cache.paged_cache import PagedCache

    model = built(GAMMA)
    cache = PagedCache(model.cache_specs(), dtype=torch.float32, device="cpu", page_size=8, max_num_sequences=3, max_model_length=512,
                       step_tokens=16, num_pages=64)
    assert {(g.spec.window, g.spec.keep_first, g.spec.head_dim) for g in cache.groups} == {(70, 3, 128), (45, 0, 64), (31, 18, 192), (90, 0, 128)}
    # every layer has the previous row, every pair of mixers the memory's S, n and m
    assert sorted(tuple(tuple(s) for s in spec.shapes) for spec in cache.state_specs.values()) == sorted(
        4 * [((64,),)] + [((2, 128, 64), (2, 128), (2,)), ((4, 64, 32), (4, 64), (4,))])
    cache.open(1)
    for at in range(0, 400, 16):
        cache.manager.ensure(1, at + 16)
        cache.manager.advance(1, at + 16)
        cache.manager.check_invariants()
    for group in cache.groups:
        table = cache.manager.table(1, group.index)
        kept, first_live = -(-group.spec.keep_first // 8), (400 - group.spec.window + 1) // 8
        assert all(page >= 0 for page in table[:kept]) and all(page < 0 for page in table[kept:first_live])
        assert all(page >= 0 for page in table[first_live:])
        view = cache.view(next(iter(group.entries)), True, [None] * len(cache.groups))
        assert (view.window, view.keep_first) == (group.spec.window, group.spec.keep_first)
    cache.manager.release(1)
    cache.manager.check_invariants()


def test_reservation_of_a_window_with_kept_tokens_covers_what_a_request_takes():
    from llm_inference_b200.csrc.host_module import host

    h = host()
    for window, keep, page, step in itertools.product((1, 7, 16), (0, 1, 8, 9, 40), (4, 8), (1, 5, 12)):
        manager = h.CacheManager(page, [h.GroupSpec("w", 200, window, keep)], 0, step)
        assert manager.admit(1, 160)
        at = 0
        while at < 160:
            at = min(160, at + step)
            manager.ensure(1, at)
            manager.advance(1, at)
            manager.check_invariants()
            used = manager.stats()["kv_pools"]["w"]["used_pages"] if "kv_pools" in manager.stats() else None
            if used is not None:
                assert used <= -(-(window + step) // page) + 1 + -(-keep // page)
        manager.release(1)
        manager.check_invariants()
    with pytest.raises(h.CacheError if hasattr(h, "CacheError") else Exception, match="window"):
        h.CacheManager(8, [h.GroupSpec("full", 10, 0, 3)], 0, 4)


ERRORS = [
    (lambda c: c.pop("vocab"), "vocab"),
    (lambda c: c["norm"].update(eps=0.0), "eps"),
    (lambda c: c.update(layers=[]), "layers"),
    (lambda c: c["layers"][0].update(type="other"), "type"),
    (lambda c: c["layers"][0]["mixer"].pop("left_scale"), "left_scale"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=3), "multiple"),
    (lambda c: c["layers"][0]["mixer"]["left"]["mask"].update(size=0), "size"),
    (lambda c: c["layers"][0]["mixer"]["left"]["mask"].update(keep_first=-1), "keep_first"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=7), "dims"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"]["scaling"].update(factor=0.0), "factor"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(gate_cap=0.0), "gate_cap"),
    (lambda c: c["layers"][1]["mixer"].update(vdim=8), "vdim"),
    (lambda c: c["layers"][1]["mlp"].update(kind="wide"), "kind"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=9), "top"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(count=3), "groups"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(identity=-2), "identity"),
    (lambda c: c["layers"][1]["mlp"]["shared"].update(ff=0), "shared"),
]


@pytest.mark.parametrize("change,message", ERRORS)
def test_configuration_errors(change, message):
    from llm_inference_b200.config import ConfigError

    raw = copy.deepcopy(ALPHA)
    change(raw)
    with pytest.raises(ConfigError, match=message):
        parsed(raw)


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
    assert torch.equal(block.mixer.constant, 0.8 * tensors["l0.mix.left.o.b"].float())
    memory_w = block.mixer.members[1].w_in
    assert memory_w.shape[0] % 8 == 0 and torch.equal(memory_w[:36], tensors["l0.mix.right.q"].float())
    ff = model.blocks[1].feed_forward
    assert torch.equal(ff.w_router[-1:], tensors["l1.mlp.shared.sg"].float()) and ff.w_gate_up.shape == (6, 20, 48)


@pytest.mark.parametrize("dims,base,factor", [(8, 100.0, 3.0), (16, 1e6, None), (2, 7.0, 0.5), (64, 5e4, 32.0)])
def test_frequency_table_of_the_rotary_part(dims, base, factor):
    from llm_inference_b200.parts import PartSpec, build_part

    part = build_part("position", PartSpec("rotary", dict(head_dim=dims + 4, theta=base, rotary_dims=dims, scaling={"factor": factor or 1.0})))
    want = plain.rotary_frequencies(dims, base, {"factor": factor} if factor else None)
    np.testing.assert_allclose(part.table().astype(np.float64), want, rtol=2e-6)


# --- the plain implementation against second formulations ---------------------------------------------


@pytest.mark.parametrize("mask", [None, {"size": 3}, {"size": 4, "keep_first": 2}, {"size": 1, "keep_first": 7}, {"size": 30, "keep_first": 5}])
@pytest.mark.parametrize("sigmoid", [False, True])
def test_attention_as_masked_matrices(mask, sigmoid):
    rng = np.random.default_rng(1)
    n, heads, groups, d, e = 17, 4, 2, 6, 5
    q, k, v = rng.normal(size=(n, heads, d)), rng.normal(size=(n, groups, d)), rng.normal(size=(n, groups, e))
    bias = rng.normal(size=heads)
    got = plain.attend(q, k, v, np.arange(n), 0.7, mask, bias if sigmoid else None)
    i, j = np.arange(n)[:, None], np.arange(n)[None, :]
    seen = j <= i
    if mask:
        seen &= ((i - j) < mask["size"]) | (j < mask.get("keep_first", 0))
    for h in range(heads):
        scores = 0.7 * q[:, h] @ k[:, h // 2].T
        weights = np.where(seen, 1.0 / (1.0 + np.exp(-scores - bias[h])), 0.0) if sigmoid else plain.softmax(np.where(seen, scores, -np.inf))
        np.testing.assert_allclose(got[:, h], weights @ v[:, h // 2], atol=1e-12)


def test_matrix_memory_as_a_weighted_sum_over_the_past():
    """Unrolled, S_t is a sum over j of exp(i_j + f_(j+1) + ... + f_t - m_t) k_j v_j^T, and m cancels between numerator and
    denominator up to the floor."""
    rng = np.random.default_rng(2)
    n, d, e = 25, 4, 3
    q, k, v = rng.normal(size=(n, d)), rng.normal(size=(n, d)), rng.normal(size=(n, e))
    i, f = rng.normal(0, 3, n), -np.abs(rng.normal(0, 1, n))
    S, norm, m = np.zeros((d, e)), np.zeros(d), 0.0
    for t in range(n):
        S, norm, m, out = plain.memory_step(S, norm, m, q[t], k[t], v[t], i[t], f[t])
        logs = np.array([i[j] + f[j + 1 : t + 1].sum() for j in range(t + 1)])
        assert m == pytest.approx(max(f[: t + 1].sum(), logs.max()))
        weights = np.exp(logs) * (k[: t + 1] @ q[t])
        np.testing.assert_allclose(out, np.exp(-m) * (weights @ v[: t + 1]) / (max(abs(np.exp(-m) * weights.sum()), np.exp(-m)) + 1e-6), rtol=1e-9, atol=1e-12)


def test_token_shift_and_norm():
    rng = np.random.default_rng(3)
    h, shift, before = rng.normal(size=(5, 6)), rng.uniform(size=6), rng.normal(size=6)
    got = plain.token_shift(h, shift, before)
    np.testing.assert_allclose(got[0], (1 - shift) * h[0] + shift * before)
    np.testing.assert_allclose(got[3], (1 - shift) * h[3] + shift * h[2])
    np.testing.assert_allclose(plain.offset_norm(h, np.zeros(6), 0.0).std(axis=1) ** 2 + plain.offset_norm(h, np.zeros(6), 0.0).mean(axis=1) ** 2, 1.0)


def test_router_against_a_search_over_all_choices():
    rng = np.random.default_rng(4)
    router = {"experts": 6, "identity": 2, "top": 3, "groups": {"count": 4, "keep": 2}}
    for _ in range(40):
        logits, correction = rng.normal(0, 2, (1, 8)), rng.normal(0, 0.4, 8)
        ids, weights, scores = plain.route(logits, correction, router)
        choice = scores[0] + correction
        best = sorted(range(4), key=lambda g: -choice[2 * g : 2 * g + 2].max())[:2]
        allowed = [e for g in best for e in (2 * g, 2 * g + 1)]
        top = max(itertools.combinations(sorted(allowed), 3), key=lambda c: choice[list(c)].sum())
        assert set(ids[0]) == set(top)
        np.testing.assert_allclose(weights[0], np.exp(logits[0, ids[0]]) / np.exp(logits[0]).sum())


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_whole_model_in_portions_and_token_by_token(name):
    config = CONFIGS[name]
    w = as_float64(draw_weights(config, 7))
    tokens = np.random.default_rng(1).integers(0, config["vocab"], 30)
    whole, _ = plain.forward(config, w, tokens)
    for sizes in ((30,), (1,) * 30, (7, 2, 11, 1, 9)):
        state, parts, at = None, [], 0
        for size in sizes:
            logits, state = plain.forward(config, w, tokens[at : at + size], state)
            parts.append(logits)
            at += size
        np.testing.assert_allclose(np.concatenate(parts), whole, atol=1e-9)


def test_helpers_leave_absent_mechanisms_absent():
    assert "mask" not in softmax_attention(mask=None) and "rot" not in softmax_attention(rot=None)
    assert "keep_first" not in softmax_attention(mask=(5, None))["mask"] and "identity" not in moe(identity=0)["router"] and memory()["gate_cap"] == 6.0
