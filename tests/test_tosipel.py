"""Tosipel: every mechanism alone against the plain implementation, then whole models in every cutting of the work
(whole prompts, token by token, portions down to two tokens, unequal requests in one batch, pages and slots given back
and used again), long decoding from captured steps, the trace tool and greedy generation through the engine."""

from __future__ import annotations

import json
import subprocess
import sys
from types import SimpleNamespace

import numpy as np
import pytest
import torch

from gunedra_helpers import MEAN_TOLERANCE, TOLERANCE, Replay, as_float64, row_error, write_folder
from helpers import TRACE_RUN
from plain import tosipel_plain as plain
from test_dugalix import CLOSE, DEVICE, DTYPES, as64, rounded, run_in_portions
from test_parts import context_for
from test_tunadra import step_mixers
from tosipel_helpers import ALPHA, CONFIGS, attention, delta, draw_weights, latent

pytestmark = pytest.mark.gpu


def mixer_case(layer: dict, seed: int, hidden: int, eps: float = 1e-5):
    """The mixer part, its weights and the plain function over rows that start a sequence."""
    from llm_inference_b200.models.tosipel import tosipel_mixer
    from llm_inference_b200.parts import build_part

    config = dict(ALPHA, width=hidden, layers=[dict(layer, mlp=None)])
    weights = {k: v for k, v in draw_weights(config, seed).items() if k.startswith("l0.mix.")}
    mixer = build_part("mixer", tosipel_mixer(layer["type"], layer["mixer"], "l0.mix.", hidden, eps))
    function = plain.MIXERS[layer["type"]]
    return mixer, weights, lambda rows, w, sizes=layer["mixer"]: function(rows, w, "l0.mix.", sizes, eps, np.arange(len(rows)), {})


# --- attention in a window, with a sink and a gate per head -----------------------------------------------------------

ATTENTION = {
    "half the head rotated": attention(),
    "window of one page, whole heads rotated": attention(4, 2, 16, 16, 0.6, 8, (16, 50.0)),
    "window of one": attention(3, 1, 10, 14, 0.7, 1, (2, 9.0)),
    "every earlier key, no rotation": attention(5, 5, 12, 6, 0.8, None, None),
    "values wider than 128": attention(3, 3, 8, 136, 1.0, 9, (8, 30.0)),
    "heads of 64": attention(6, 2, 64, 48, 0.3, 21, (32, 1e4)),
    "heads of 128": attention(6, 3, 96, 128, 0.2, 40, (96, 1e5)),
    "heads of 192": attention(4, 1, 112, 160, 0.2, 19, (48, 3e5)),
    "many query heads on one": attention(20, 1, 24, 24, 0.5, 30, (24, 500.0)),
}


@pytest.mark.parametrize("name", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", sorted(ATTENTION))
def test_attention_alone_in_portions_beside_another_request(name, case):
    """70 tokens over pages of 8 in portions that end before, on and after page and window edges, a second request in the
    same steps, NaN in everything unwritten. Scores are a few units wide, so single keys carry weight: the test itself
    asserts that a window one longer or shorter, no sink, a scaled sink, no gate, another rotation, norms per head instead of
    over the whole projection and another sharing of kv heads would move the output far outside the tolerance."""
    dtype, hidden, total = DTYPES[name], 48, 70
    layer = ATTENTION[case]
    m = layer["mixer"]
    mixer, weights, reference = mixer_case(layer, 21, hidden)
    w64 = as_float64(weights)
    rng = np.random.default_rng(8)
    inputs = {10: rounded(rng.normal(0, 1, (total, hidden)), dtype), 11: rounded(rng.normal(0, 1, (9, hidden)), dtype)}
    want = {rid: reference(rows.double().numpy(), w64) for rid, rows in inputs.items()}
    long = inputs[10].double().numpy()

    def effect(sizes=m, w=w64):
        return np.abs(reference(long, w, sizes) - want[10]).max()

    if m.get("mask"):
        for size in (m["mask"]["size"] - 1, m["mask"]["size"] + 1):
            assert not size or effect(dict(m, mask={"size": size})) > 0.2
    sink = w64["l0.mix.sink"]
    assert effect(w=dict(w64, **{"l0.mix.sink": 0 * sink - 60})) > 0.2 and effect(w=dict(w64, **{"l0.mix.sink": sink * m["scale"] * 0.9})) > 0.1
    assert effect(w=dict(w64, **{"l0.mix.g": 0 * w64["l0.mix.g"] + 9})) > 0.1
    if m.get("rot") and (m.get("mask") or {"size": 9})["size"] > 1:  # a token that sees itself alone sees no distance
        assert effect(dict(m, rot=dict(m["rot"], base=m["rot"]["base"] * 3))) > 0.02
    if m["kv_heads"] > 1 and m["heads"] > m["kv_heads"]:
        turned = np.roll(w64["l0.mix.k"].reshape(m["kv_heads"], m["dim"], hidden), 1, axis=0).reshape(-1, hidden)
        assert effect(w=dict(w64, **{"l0.mix.k": turned})) > 0.2

    def per_head(x, weight, eps):  # a mistake planted in the plain implementation: every head normed by itself
        size = m["dim"]
        return plain.unit_rms(x.reshape(len(x), -1, size), eps).reshape(x.shape) * weight

    original = plain.plain_norm
    try:
        plain.plain_norm = per_head
        assert effect() > 0.05 or (m["heads"] == 1 and m["kv_heads"] == 1)
    finally:
        plain.plain_norm = original
    got = run_in_portions(mixer, weights, dtype, inputs, total)
    np.testing.assert_allclose(got[10], want[10], **CLOSE[name])
    np.testing.assert_allclose(got[11], want[11], **CLOSE[name])


@pytest.mark.parametrize("case", ["heads of 64", "heads of 128", "heads of 192"])
@pytest.mark.parametrize("page", [16, 64])
@pytest.mark.parametrize("window", [150, 64, 128, 1, 0])
def test_tensor_core_kernels_with_a_sink_far_in(case, page, window):
    """bfloat16, 720 keys: prompt portions run tcgen05 (heads of 128) or mma.sync, single tokens the split-key kernels; the
    same steps run the plain kernel. Windows end inside, at and just past tiles of 64 and 128 keys; some tokens resemble
    far ones, so that one far key stands out. Every row a request did not write holds NaN. Sinks are as large as the
    largest scores."""
    from llm_inference_b200.cache import PagedCache
    from llm_inference_b200.engine.runner import ModelRunner

    hidden, total = 48, 720
    layer = dict(ATTENTION[case])
    mixer, weights, _ = mixer_case(layer, 23, hidden)
    mixer.window = window
    weights["l0.mix.sink"] = weights["l0.mix.sink"] + 2
    sizes = {k: v for k, v in layer["mixer"].items() if k != "mask"}
    if window:
        sizes["mask"] = {"size": window}
    rng = np.random.default_rng(5)
    rows = rng.normal(0, 1, (total, hidden))
    for t in (10, 300, 500):
        for later in range(t + 60, total, 97):
            rows[later] = 0.5 * rows[later] + 1.5 * rows[t]
    rows = rounded(rows, torch.bfloat16)
    want = plain.window_attention(rows.double().numpy(), as_float64(weights), "l0.mix.", sizes, 1e-5, np.arange(total), {})
    no_sink = plain.window_attention(rows.double().numpy(), dict(as_float64(weights), **{"l0.mix.sink": np.full(sizes["heads"], -50.0)}), "l0.mix.", sizes, 1e-5, np.arange(total), {})
    assert np.abs(want - no_sink).max() > 0.3
    results = {}
    for choice in ("auto", "plain"):
        device = torch.device(DEVICE)
        cache = PagedCache({0: mixer.cache_spec()}, dtype=torch.bfloat16, device=device, page_size=page, max_num_sequences=4, max_model_length=1024,
                           step_tokens=1024, num_pages=1024 // page)
        for group in cache.groups:
            group.arena[:, :, :-1].fill_(float("nan"))  # every page a request can hold; the spare page that pads block tables stays finite
        runner = ModelRunner(SimpleNamespace(device=device, dtype=torch.bfloat16), cache, max_batch_tokens=1024, options={"attention": choice})
        mixer.load(weights, torch.bfloat16, device)
        cache.open(10)
        parts, at = [], 0
        for portion in (511, 1, 1, 50, 1, 1, 1, 2, 63, 1, 1, 87):
            (out,) = step_mixers(runner, cache, [mixer], [(10, slice(at, at + portion))], {10: rows})
            parts.append(out[10])
            at += portion
        runner.check()
        results[choice] = np.concatenate(parts)
    scale = np.abs(want).std() + 1.0
    np.testing.assert_allclose(results["plain"] / scale, want / scale, atol=6e-2, rtol=3e-2)
    np.testing.assert_allclose(results["auto"] / scale, want / scale, atol=6e-2, rtol=3e-2)
    error = np.abs(results["auto"] - want).mean() / np.abs(results["plain"] - want).mean()
    assert error < 1.6, error  # rounding of the weights costs about as much as that of the operands
    assert np.abs(results["auto"] - results["plain"]).max() > 0 or window == 1  # other kernels ran


def test_split_keys_count_the_sink_once():
    """Decoded tokens, one request far in and one that barely started, with every number of key splits from 1 to 20, merged by
    the second kernel and on chip: the sink counts once however the keys are cut; sinks far above and far below every score."""
    from llm_inference_b200.parts import CacheView, attention_dispatch, ops

    heads, kvh, page, kv_len = 4, 2, 64, (1500, 3)
    torch.manual_seed(0)
    for dim in (64, 128, 192):
        runner, _, ctx = context_for({}, torch.bfloat16, [1, 1])
        ctx.seq_kv_len = torch.tensor(kv_len, dtype=torch.int32, device="cuda")
        ctx.positions = ctx.seq_kv_len - 1
        ctx.max_kv_len = max(kv_len)
        keys, values = (torch.randn(26, kvh, page, dim, device="cuda").bfloat16() for _ in range(2))
        table = torch.zeros(2, 24, dtype=torch.int32, device="cuda")
        table[0] = torch.randperm(24).cuda()
        table[1, 0] = 24
        q = torch.randn(2, heads * dim, device="cuda").bfloat16()
        for window, sinks in ((700, (3.0, 1.0, -2.0, 0.5)), (0, (6.0, 8.0, 7.0, 5.0)), (65, (90.0, -90.0, 1.0, 200.0))):
            view = CacheView(0, True, keys, values, table, 26, 24, page, window, 0)
            shape = ops.ScoreShape(sink=torch.tensor(sinks, device="cuda"))
            ctx.options = {"attention": "plain"}
            want, bare = torch.empty_like(q), torch.empty_like(q)
            attention_dispatch.attend(ctx, view, q, want, heads, kvh, dim, dim**-0.5, shape=shape)
            attention_dispatch.attend(ctx, view, q, bare, heads, kvh, dim, dim**-0.5)
            runner.check()
            # the short request's three keys by hand
            for h in range(heads):
                k, v = (x[24, h // 2, :3].double() for x in (keys, values))
                scores = k @ q[1].view(heads, dim)[h].double() * dim**-0.5
                e = torch.exp(torch.cat([scores, torch.tensor([sinks[h]], device="cuda").double()]).double() - max(float(scores.max()), sinks[h]))
                np.testing.assert_allclose(as64(want[1].view(heads, dim)[h]), as64(e[:3] @ v / e.sum()), atol=1e-2, rtol=2e-2)
            assert (want - bare).abs().max() > 0.02
            for splits in range(1, 21):
                for loader, merge in (("auto", "auto"), ("cp_async", "scratch"), ("cp_async", "cluster"), ("auto", "cluster")):
                    if merge == "cluster" and splits > 16:
                        continue
                    ctx.options = {"decode_splits": splits, "decode_loader": loader, "attention_merge": merge}
                    got = torch.full_like(q, float("nan"))
                    attention_dispatch.attend(ctx, view, q, got, heads, kvh, dim, dim**-0.5, shape=shape)
                    error = (got.float() - want.float()).abs().max() / want.float().abs().max()
                    assert error < 2e-2, (dim, window, splits, loader, merge, float(error))
        runner.check()


@pytest.mark.parametrize("dim", [64, 128])
def test_a_sink_goes_with_shaped_scores_and_kept_first_keys(dim):
    """Prompt portions and single tokens with a soft cap and a bias by distance, and with first keys kept in front of a window:
    every tensor-core form that has a softmax takes a sink."""
    from llm_inference_b200.parts import CacheView, attention_dispatch, ops

    heads, kvh, page, run = 4, 2, 64, 300
    torch.manual_seed(1)
    runner, _, ctx = context_for({}, torch.bfloat16, [1])
    keys, values = (torch.randn(6, kvh, page, dim, device="cuda").bfloat16() for _ in range(2))
    table = torch.arange(5, dtype=torch.int32, device="cuda")[None].contiguous()
    sink = torch.randn(heads, device="cuda") + 2
    bias = torch.randn(heads, 41, device="cuda")
    as_int = lambda *v: torch.tensor(v, dtype=torch.int32, device="cuda")
    for tokens in (run, 1):
        ctx.num_tokens, ctx.num_seqs, ctx.num_decode_seqs, ctx.max_q_len, ctx.max_kv_len = tokens, 1, int(tokens == 1), tokens, run
        ctx.seq_q_start, ctx.seq_q_len, ctx.seq_kv_len = as_int(0), as_int(tokens), as_int(run)
        ctx.positions, ctx.token_seq = torch.arange(run - tokens, run, dtype=torch.int32, device="cuda"), torch.zeros(tokens, dtype=torch.int32, device="cuda")
        q = torch.randn(tokens, heads * dim, device="cuda").bfloat16()
        for window, keep, shape in ((0, 0, ops.ScoreShape(5.0, bias, 0, bias.max(1).values.contiguous(), sink=sink)), (0, 0, ops.ScoreShape(3.0, None, 90, sink=sink)),
                                    (100, 9, ops.ScoreShape(sink=sink))):
            view = CacheView(0, True, keys, values, table, 6, 5, page, window, keep)
            out = {}
            for choice in ("plain", "auto", "flash"):
                ctx.options = {"attention": choice}
                out[choice] = torch.full_like(q, float("nan"))
                attention_dispatch.attend(ctx, view, q, out[choice], heads, kvh, dim, dim**-0.5, shape=shape)
            runner.check()
            for choice in ("auto", "flash"):
                error = (out[choice].float() - out["plain"].float()).abs().max() / out["plain"].float().abs().max()
                assert error < 2e-2, (tokens, window, choice, float(error))
    with pytest.raises(ops.KernelError, match="sink"):
        attention_dispatch.attend(ctx, view, q, out["plain"], heads, kvh, dim, 0.1, shape=ops.ScoreShape(sigmoid_bias=sink, sink=sink))


# --- attention over latents without positions ---------------------------------------------------------------------------

LATENT = {
    "odd sizes": latent(), "one head": latent(1, 7, 5, 33, 9, 0.9), "a latent of 32": latent(3, 16, 24, 32, 40, 0.5), "a latent of 96": latent(5, 24, 32, 96, 64, 0.3),
    "wide": latent(2, 128, 96, 160, 100, 0.15), "more heads than a tile's rows": latent(20, 16, 8, 64, 128, 0.4),
}


@pytest.mark.parametrize("name", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", sorted(LATENT))
def test_latent_attention_without_positions_alone_in_portions(name, case):
    """70 tokens in portions beside another request; the test asserts that missing norms of either latent, another scale and
    a lost first portion would show."""
    dtype, hidden, total = DTYPES[name], 48, 70
    layer = LATENT[case]
    m = layer["mixer"]
    mixer, weights, reference = mixer_case(layer, 22, hidden)
    w64 = as_float64(weights)
    rng = np.random.default_rng(9)
    inputs = {10: rounded(rng.normal(0, 1, (total, hidden)), dtype), 11: rounded(rng.normal(0, 1, (9, hidden)), dtype)}
    want = {rid: reference(rows.double().numpy(), w64) for rid, rows in inputs.items()}
    long = inputs[10].double().numpy()
    assert np.abs(reference(long, w64, dict(m, scale=m["scale"] * 1.3)) - want[10]).max() > 0.05
    assert np.abs(reference(long[7:], w64)[:3] - want[10][7:10]).max() > 0.1
    for tensor in ("dq", "dkv"):  # the norm takes a factor of the projection off again
        assert np.abs(reference(long, dict(w64, **{f"l0.mix.{tensor}": 5 * w64[f"l0.mix.{tensor}"]})) - want[10]).max() < 1e-2
    got = run_in_portions(mixer, weights, dtype, inputs, total)
    np.testing.assert_allclose(got[10], want[10], **CLOSE[name])
    np.testing.assert_allclose(got[11], want[11], **CLOSE[name])


@pytest.mark.parametrize("page", [8, 64])
def test_latent_attention_sees_one_far_key_among_hundreds(page):
    """bfloat16, 600 tokens: some tokens ask for one far token that stands out, in a portion and as single tokens whose keys
    are cut into pieces; the plain kernel and the tensor-core kernel agree with the plain implementation."""
    from llm_inference_b200.cache import PagedCache
    from llm_inference_b200.engine.runner import ModelRunner

    hidden, total = 64, 600
    layer = latent(4, 32, 32, 64, 64, 0.5)
    mixer, weights, reference = mixer_case(layer, 5, hidden)
    # a token's query is the key of the token whose row is its own shifted by one column
    for query, key in (("dq", "dkv"), ("dq.norm", "dkv.norm"), ("uq", "uk")):
        weights["l0.mix." + query] = weights["l0.mix." + key].clone()
    weights["l0.mix.dq"] = weights["l0.mix.dq"].roll(-1, dims=1).contiguous()
    rng = np.random.default_rng(6)
    rows = rng.normal(0, 1.0, (total, hidden))
    pairs = ((599, 0), (597, 63), (596, 64), (450, 1), (333, 127))
    for asks, target in pairs:
        rows[asks] = np.roll(rows[target], -1)
    rows = rounded(rows, torch.bfloat16)
    w64 = as_float64(weights)
    want = reference(rows.double().numpy(), w64)
    for asks, target in pairs:  # most of the weight lies on the far key: without it the output is another
        other = rows.double().numpy()
        other[target] = 0.0
        assert np.abs(reference(other, w64)[asks] - want[asks]).max() > 0.3
    results = {}
    for choice in ("auto", "plain"):
        device = torch.device(DEVICE)
        cache = PagedCache({0: mixer.cache_spec()}, dtype=torch.bfloat16, device=device, page_size=page, max_num_sequences=2, max_model_length=640,
                           step_tokens=640, num_pages=640 // page)
        for group in cache.groups:
            group.arena[:, :, :-1].fill_(float("nan"))
        runner = ModelRunner(SimpleNamespace(device=device, dtype=torch.bfloat16), cache, max_batch_tokens=640, options={"attention": choice})
        mixer.load(weights, torch.bfloat16, device)
        cache.open(10)
        parts, at = [], 0
        for portion in (440, 2, 64, 89, 1, 1, 1, 1, 1):
            (out,) = step_mixers(runner, cache, [mixer], [(10, slice(at, at + portion))], {10: rows})
            parts.append(out[10])
            at += portion
        assert at == total
        runner.check()
        results[choice] = np.concatenate(parts)
    for got in results.values():
        np.testing.assert_allclose(got, want, atol=8e-2, rtol=4e-2)
    assert np.abs(results["auto"] - results["plain"]).max() > 0


# --- the delta rule with one decay per head -------------------------------------------------------------------------------

DELTA = {
    "three kv heads": delta(), "one row": delta(2, 2, 1, 5, 4), "odd": delta(3, 1, 9, 11, 3), "a single tap": delta(4, 2, 16, 6, 1), "two taps": delta(6, 2, 17, 35, 2),
    "seven taps": delta(2, 1, 24, 24, 7), "whole warps": delta(4, 2, 128, 64, 4), "wide values": delta(2, 2, 40, 256, 4), "more rows than lanes hold": delta(1, 1, 300, 9, 4),
    "nine heads on one": delta(9, 1, 8, 12, 4), "eight heads on one": delta(8, 1, 64, 32, 3), "wider than a block": delta(1, 1, 6, 530, 2), "widest": delta(1, 1, 600, 3, 4),
}


@pytest.mark.parametrize("name", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", sorted(DELTA))
@pytest.mark.parametrize("step", ["auto", "tokens", "chunks"])
def test_delta_rule_alone_in_portions_beside_another_request(name, case, step):
    """70 tokens in portions beside another request, slots full of NaN before; steps in which both feed one token run the fused
    kernel ("tokens", "chunks": the kernels of prompt portions in every step, token by token or 32 tokens at a time). The test asserts that a lost state, a lost convolution
    history, a missing decay, a read-out of the old state and unit vectors left out would show."""
    dtype, hidden, total = DTYPES[name], 48, 70
    layer = DELTA[case]
    m = layer["mixer"]
    mixer, weights, reference = mixer_case(layer, 24, hidden)
    w64 = as_float64(weights)
    rng = np.random.default_rng(10)
    inputs = {10: rounded(rng.normal(0, 1, (total, hidden)), dtype), 11: rounded(rng.normal(0, 1, (9, hidden)), dtype)}
    want = {rid: reference(rows.double().numpy(), w64) for rid, rows in inputs.items()}
    long = inputs[10].double().numpy()
    if m["dim"] > 1:  # (a state of one row is overwritten by every token with beta near one)
        assert np.abs(reference(long[7:], w64)[:3] - want[10][7:10]).max() > 0.02
        assert np.abs(reference(long, dict(w64, **{"l0.mix.A_log": w64["l0.mix.A_log"] - 30})) - want[10]).max() > 0.02
        assert np.abs(reference(long, dict(w64, **{"l0.mix.b": 0 * w64["l0.mix.b"]})) - want[10]).max() > 0.05
    for tensor in ("q", "k"):  # unit vectors: a factor of the projection matters only through silu
        taps = w64[f"l0.mix.{tensor}.conv"]
        assert m["conv"] == 1 or m["dim"] == 1 or np.abs(reference(long, dict(w64, **{f"l0.mix.{tensor}.conv": taps * (np.arange(m["conv"]) > 0)})) - want[10]).max() > 0.02
    original = plain.delta_step
    try:
        plain.delta_step = lambda S, q, k, v, g, beta: (original(S, q, k, v, g, beta)[0], (g * S).T @ q)
        assert np.abs(reference(long, w64) - want[10]).max() > 0.05
    finally:
        plain.delta_step = original
    mixer.load(weights, dtype, torch.device(DEVICE))  # the history is kept in the weights' dtype
    if step == "chunks" and m["dim"] > 256:
        pytest.skip("chunks take up to 256 key channels")
    options = {} if step == "auto" else {"delta_step": "chain", "delta_portions": step}
    got = run_in_portions(mixer, weights, dtype, inputs, total, options)
    np.testing.assert_allclose(got[10], want[10], **CLOSE[name])
    np.testing.assert_allclose(got[11], want[11], **CLOSE[name])


@pytest.mark.parametrize("name", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", ["three kv heads", "whole warps", "odd", "eight heads on one", "nine heads on one", "wide values"])
@pytest.mark.parametrize("portions", ["auto", "tokens"])
def test_delta_rule_long_portions_and_many_single_tokens(name, case, portions):
    """500 tokens: as one portion beside others of 1 to 129 tokens, then the same as 60 single tokens behind a portion, then cut
    around multiples of 32 (the chunks of the kernels that take 32 tokens at a time start with a portion); heads that keep hundreds
    of tokens and heads that forget in a few."""
    from llm_inference_b200.cache import PagedCache
    from llm_inference_b200.engine.runner import ModelRunner

    dtype, hidden, total = DTYPES[name], 48, 500
    mixer, weights, reference = mixer_case(DELTA[case], 25, hidden)
    w64 = as_float64(weights)
    rng = np.random.default_rng(11)
    lengths = {10: total, 11: 129, 12: 1, 13: 64, 14: 33, 15: 2}
    inputs = {rid: rounded(rng.normal(0, 1, (n, hidden)), dtype) for rid, n in lengths.items()}
    want = {rid: reference(rows.double().numpy(), w64) for rid, rows in inputs.items()}
    device = torch.device(DEVICE)
    mixer.load(weights, dtype, device)
    for cuts in ((total,), (440,) + (1,) * 60, (31, 32, 33, 64, 65, 7, 2, 100, 166)):
        cache = PagedCache({0: mixer.cache_spec()}, dtype=dtype, device=device, page_size=8, max_num_sequences=6, max_model_length=512, step_tokens=1024, num_pages=8)
        for array in cache.states[0]:
            array.fill_(float("nan"))
        runner = ModelRunner(SimpleNamespace(device=device, dtype=dtype), cache, max_batch_tokens=1024, options={"delta_portions": portions})
        for rid in lengths:
            cache.open(rid)
        at, parts = 0, []
        for turn, cut in enumerate(cuts):
            step = [(10, slice(at, at + cut))]
            if turn == 0:
                step += [(rid, slice(0, n)) for rid, n in lengths.items() if rid != 10]
            (out,) = step_mixers(runner, cache, [mixer], step, inputs)
            parts.append(out[10])
            at += cut
            if turn == 0:
                for rid in lengths:
                    if rid != 10:
                        np.testing.assert_allclose(out[rid], want[rid], **CLOSE[name])
        runner.check()
        assert at == total
        np.testing.assert_allclose(np.concatenate(parts), want[10], **CLOSE[name])


def test_chunks_with_decays_that_end_a_memory_at_once_and_keys_that_repeat():
    """float32, the recurrences' kernels on given operands: log decays of zero, tiny ones, and down to -400 in the middle of a chunk;
    keys that repeat token after token with beta near one (the triangular system at its stiffest); 32 tokens at a time, token by
    token and the 64-bit recurrence agree, and a state that comes in counts."""
    from llm_inference_b200.parts import StateSpec, ops

    heads, kvh, dk, dv, n = 4, 2, 40, 28, 150
    rng = np.random.default_rng(3)
    unit = lambda x: x / np.linalg.norm(x, axis=-1, keepdims=True)
    k, q = unit(rng.normal(size=(n, kvh, dk))), unit(rng.normal(size=(n, kvh, dk)))
    k[20:60] = k[20]
    v, beta = rng.normal(size=(n, heads, dv)), rng.uniform(0.95, 1.0, (n, heads))
    log_decay = -np.exp(rng.normal(-5, 2, (n, heads)))
    log_decay[:, 1] = 0.0
    log_decay[[17, 40, 41, 97], 2] = [-400.0, -90.0, -400.0, -30.0]
    start = rng.normal(size=(heads, dk, dv))
    q, k, v, beta, log_decay, start = (a.astype(np.float32) for a in (q, k, v, beta, log_decay, start))
    S = start.astype(np.float64)
    want = np.zeros((n, heads, dv))
    for t in range(n):
        for h in range(heads):
            S[h], want[t, h] = plain.delta_step(S[h], q[t, h // 2].astype(np.float64), k[t, h // 2].astype(np.float64), v[t, h].astype(np.float64),
                                                np.exp(float(log_decay[t, h])), float(beta[t, h]))
    device = [torch.from_numpy(np.ascontiguousarray(a.reshape(n, -1))).cuda() for a in (q, k, v, beta, log_decay, (q * k).sum(-1))]
    for choice in ("tokens", "chunks"):
        runner, cache, ctx = context_for({0: StateSpec(((heads, dk, dv),), (torch.float32,))}, torch.float32, [2])
        ctx.options = {"delta_portions": choice}
        state = cache.states[0][0]
        state[:] = torch.from_numpy(start).cuda()
        ctx.num_tokens, ctx.num_seqs, ctx.max_q_len = n, 1, n
        ctx.seq_q_start, ctx.seq_q_len = (torch.tensor([x], dtype=torch.int32, device="cuda") for x in (0, n))
        out = torch.full((n, heads * dv), float("nan"), device="cuda")
        ops.delta_head_recurrence(ctx, *device, state, out, heads, kvh, dk, dv)
        runner.check()
        np.testing.assert_allclose(as64(out).reshape(want.shape), want, atol=2e-5, rtol=2e-5, err_msg=choice)
        np.testing.assert_allclose(as64(state[int(ctx.seq_slot[0])]), S, atol=2e-5, rtol=2e-5, err_msg=choice)


# --- the gated unit ----------------------------------------------------------------------------------------------------------


@pytest.mark.parametrize("name", ["float32", "bfloat16"])
@pytest.mark.parametrize("tokens,hidden,ff", [(1, 48, 60), (5, 64, 96), (8, 512, 1536), (16, 256, 1024), (17, 256, 512), (31, 1024, 2000), (33, 50, 33), (70, 128, 256)])
def test_gelu_unit_alone(name, tokens, hidden, ff):
    from llm_inference_b200.parts import PartSpec, build_part

    dtype = DTYPES[name]
    rng = np.random.default_rng(tokens)
    weights = {f"m.{n}": rounded(rng.normal(0, 2.0 / np.sqrt(hidden), (ff, hidden)), torch.bfloat16) for n in ("gate", "up")}
    weights["m.down"] = rounded(rng.normal(0, 1 / np.sqrt(ff), (hidden, ff)), torch.bfloat16)
    part = build_part("feed_forward", PartSpec("geglu", dict(prefix="m.", hidden_size=hidden, intermediate_size=ff)))
    part.load(weights, dtype, torch.device(DEVICE))
    h = rounded(rng.normal(0, 1, (tokens, hidden)), dtype)
    w64 = as_float64(weights)
    want = plain.gelu_unit(h.double().numpy(), w64, "m.")
    tolerance = dict(atol=3e-5, rtol=3e-5) if name == "float32" else dict(atol=6e-2, rtol=2e-2)
    for gemm in ("auto", "tcgen05", "skinny", "library"):
        runner, _, ctx = context_for({}, dtype, [tokens])
        ctx.options = {"gemm": gemm}
        got = as64(part.forward(ctx, h.cuda()))
        runner.check()
        np.testing.assert_allclose(got, want, **tolerance, err_msg=gemm)
    silu = plain.linear(plain.silu(plain.linear(h.double().numpy(), w64["m.gate"])) * plain.linear(h.double().numpy(), w64["m.up"]), w64["m.down"])
    assert np.abs(silu - want).max() > 0.15


@pytest.mark.parametrize("name", ["float32", "bfloat16"])
def test_gelu_itself_over_its_range(name):
    """Values from deep in either tail to zero, against the tanh form in 64-bit; eight at a time and a ragged end."""
    from llm_inference_b200.parts import ops

    dtype = DTYPES[name]
    for count in (4096, 4001):
        gate = torch.linspace(-30, 30, count, dtype=torch.float64).to(dtype)
        up = torch.full((count,), 1.5, dtype=dtype)
        _, _, ctx = context_for({}, dtype, [1])
        out = torch.empty(1, count, dtype=dtype, device="cuda")
        ops.gated_mul(ctx, torch.stack([gate, up], dim=1).reshape(1, -1).cuda(), out, "gelu")
        want = plain.gelu_tanh(gate.double().numpy()) * 1.5
        np.testing.assert_allclose(as64(out)[0], want, atol=1e-6 if name == "float32" else 1e-3, rtol=2e-6 if name == "float32" else 5e-3)


# --- whole models ---------------------------------------------------------------------------------------------


LENGTHS = [1, 2, 3, 9, 31, 70, 150]


@pytest.fixture(scope="module", params=sorted(CONFIGS))
def model_case(request, tmp_path_factory):
    config = CONFIGS[request.param]
    weights = draw_weights(config, seed=17 + len(request.param))
    folder = write_folder(tmp_path_factory.mktemp(request.param), config, weights)
    rng = np.random.default_rng(4)
    sequences = {f"s{n}": [int(t) for t in rng.integers(0, config["vocab"], n)] for n in LENGTHS}
    w64 = as_float64(weights)
    expected = {key: plain.forward(config, w64, tokens) for key, tokens in sequences.items()}
    return request.param, config, folder, sequences, expected, w64


def check_all(case, replay, sequences, dtype: str, what: str) -> None:
    _, config, _, _, expected, w64 = case
    errors = []
    for key, tokens in sequences.items():
        want = expected[key] if key in expected else plain.forward(config, w64, tokens)
        error = row_error(replay.of(key, len(tokens)), want)
        assert error.max() <= TOLERANCE[dtype], f"{what}: request {key}, position {int(error.argmax())}: error {error.max():.2e}"
        errors.append(error)
    mean = np.concatenate(errors).mean()
    assert mean <= MEAN_TOLERANCE[dtype], f"{what}: mean error over all rows {mean:.2e}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_layers_one_by_one_against_plain(model_case, dtype):
    """The stream after every layer of a short prompt, so that a fault names its layer."""
    from llm_inference_b200.engine.runner import StepEntry

    _, config, folder, sequences, _, w64 = model_case
    tokens = sequences["s31"]
    replay = Replay(folder, dtype, 64)
    replay.cache.open(1)
    replay.cache.manager.ensure(1, len(tokens))
    replay.cache.clear_new_slots()
    ctx = replay.runner._build_context([StepEntry(1, tokens)], [0], [])
    x = replay.model.embedding.forward(ctx)
    streams = []
    for call in replay.model.schedule:
        assert replay.model.blocks[call.layer].forward(ctx, replay.runner._view(call, replay.runner._tables), x, None) is None
        streams.append(as64(x))
    replay.runner.check()
    layers: list = []
    plain.forward(config, w64, tokens, layer_outputs=layers)
    assert len(layers) == len(streams) == len(config["layers"])
    for index, (got, want) in enumerate(zip(streams, layers)):
        error = np.abs(got - want).max() / np.abs(want).max()
        assert error <= (1e-5 if dtype == "float32" else 9e-2), f"layer {index} ({config['layers'][index]['type']}): {error:.2e}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_whole_prompts_one_after_another_in_a_pool_for_one(model_case, dtype):
    _, _, folder, sequences, _, _ = model_case
    replay = Replay(folder, dtype, 152, slots=1)
    for key, tokens in sequences.items():
        replay.step([(key, tokens)], end=(key,))
    check_all(model_case, replay, sequences, dtype, "whole")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_prompt_then_token_by_token(model_case, dtype):
    """All but the last 40 tokens as one portion, the rest one by one (captured steps replayed)."""
    _, _, folder, sequences, _, _ = model_case
    replay = Replay(folder, dtype, 152, slots=1)
    for key, tokens in sequences.items():
        head = max(0, len(tokens) - 40)
        if head:
            replay.step([(key, tokens[:head])])
        for position in range(head, len(tokens)):
            replay.step([(key, [tokens[position]])], end=(key,) if position == len(tokens) - 1 else ())
    check_all(model_case, replay, sequences, dtype, "token by token")
    assert replay.runner.graph_replays > 0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("sizes", [(2,), (3, 1, 2, 8, 1, 17), (7, 9, 64)])
def test_portions_of_changing_size(model_case, dtype, sizes):
    _, _, folder, sequences, _, _ = model_case
    replay = Replay(folder, dtype, 152, slots=1)
    for key, tokens in sequences.items():
        at, turn = 0, 0
        while at < len(tokens):
            size = min(sizes[turn % len(sizes)], len(tokens) - at)
            replay.step([(key, tokens[at : at + size])], end=(key,) if at + size == len(tokens) else ())
            at, turn = at + size, turn + 1
    check_all(model_case, replay, sequences, dtype, f"portions {sizes}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_unequal_requests_in_one_batch_with_pages_and_slots_used_again(model_case, dtype):
    """Up to three live requests (38 pages of 8 for sequences that need 46 in all): portions of some beside single tokens
    of others, requests left out of steps, and every request that ends hands its pages and its slot to one that starts
    later; windows give pages back on the way."""
    _, _, folder, sequences, _, _ = model_case
    replay = Replay(folder, dtype, 304, slots=3)
    rng = np.random.default_rng(9)
    waiting = ["s150", "s70", "s31", "s9", "s3", "s2", "s1", "again70", "again9"]
    sequences = dict(sequences, again70=sequences["s70"], again9=sequences["s9"])
    live: dict[str, int] = {}
    while waiting or live:
        while waiting and len(live) < 3:
            live[waiting.pop(0)] = 0
        portions, end = [], []
        for key in list(live):
            if len(live) > 1 and rng.random() < 0.2:
                continue  # sits this step out
            left = len(sequences[key]) - live[key]
            size = min(left, int(rng.choice([1, 1, 1, 2, 3, 8, 29])))
            portions.append((key, sequences[key][live[key] : live[key] + size]))
            live[key] += size
            if live[key] == len(sequences[key]):
                end.append(key)
                del live[key]
        if portions:
            replay.step(portions, end=tuple(end))
            replay.cache.manager.check_invariants()
    check_all(model_case, replay, sequences, dtype, "mixed")
    stats = replay.cache.stats()
    assert stats["requests"] == 0 and stats["live_tokens"] == 0
    assert all(pool["used_pages"] == 0 and pool["high_water"] <= pool["capacity_pages"] for pool in stats["kv_pools"].values())


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_three_requests_decoding_together_equal_each_alone(model_case, dtype):
    """Captured steps of three single tokens (with padding rows) against steps of one."""
    _, _, folder, sequences, _, _ = model_case
    keys = ["s150", "s70", "s31"]
    replay = Replay(folder, dtype, 304, slots=3)
    replay.step([(key, sequences[key][:-20]) for key in keys])
    for i in range(20):
        replay.step([(key, [sequences[key][len(sequences[key]) - 20 + i]]) for key in keys], end=tuple(keys) if i == 19 else ())
    check_all(model_case, replay, {key: sequences[key] for key in keys}, dtype, "together")
    assert replay.runner.graph_replays > 10


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(model_case, dtype):
    """Four tokens of prompt, then 330 single tokens: states and caches after hundreds of steps, windows that have given
    most of their pages back; and windowed groups hold no more than their bound."""
    _, config, folder, _, _, w64 = model_case
    tokens = [int(t) for t in np.random.default_rng(13).integers(0, config["vocab"], 334)]
    replay = Replay(folder, dtype, 384, slots=1)
    replay.step([("long", tokens[:4])])
    for token in tokens[4:]:
        replay.step([("long", [token])])
    for group in replay.cache.groups:
        if group.spec.window:
            assert sum(page >= 0 for page in replay.cache.manager.table(1, group.index)) <= -(-group.spec.window // 8) + 2
    error = row_error(replay.of("long", len(tokens)), plain.forward(config, w64, tokens))
    assert error.max() <= TOLERANCE[dtype], f"position {int(error.argmax())}: {error.max():.2e}"
    assert error.mean() <= MEAN_TOLERANCE[dtype] and error[-50:].mean() <= MEAN_TOLERANCE[dtype], f"mean {error.mean():.2e}, last 50 {error[-50:].mean():.2e}"
    assert replay.runner.graph_replays > 300


def test_trace_tool_mixed_schedule(model_case, tmp_path):
    """bin/trace_run itself: two requests interleaved, later ones that reuse what the first gave back; two slots for three
    requests, and a step that would hold three at once is refused."""
    _, config, folder, sequences, expected, _ = model_case
    a, b, c = sequences["s70"], sequences["s31"], sequences["s9"]
    steps = [
        {"step": 0, "entries": [{"id": "a", "tokens": a[:33], "want": [0, 32]}], "end": []},
        {"step": 1, "entries": [{"id": "b", "tokens": b[:2], "want": [1]}, {"id": "a", "tokens": a[33:34], "want": [0]}], "end": []},
        {"step": 2, "entries": [{"id": "a", "tokens": a[34:], "want": [35]}, {"id": "b", "tokens": b[2:3], "want": []}], "end": ["a"]},
        {"step": 3, "entries": [{"id": "b", "tokens": b[3:], "want": [27]}, {"id": "c", "tokens": c, "want": [8]}], "end": ["b", "c"]},
    ]
    want = [expected["s70"][[0, 32]], expected["s31"][[1]], expected["s70"][[33]], expected["s70"][[69]], expected["s31"][[30]], expected["s9"][[8]]]
    for dtype in ("float32", "bfloat16"):
        out = tmp_path / dtype
        result = subprocess.run(
            [sys.executable, str(TRACE_RUN), "--model", str(folder), "--dtype", dtype, "--out", str(out), "--max-tokens", "256", "--max-requests", "2"],
            input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600,
        )
        assert result.returncode == 0, result.stderr[-3000:]
        assert [line for line in result.stdout.splitlines() if line.startswith("done ")] == [f"done {i}" for i in range(4)]
        got = np.concatenate([np.fromfile(out / f"{i}.f32", dtype="<f4").reshape(-1, config["vocab"]) for i in range(4)])
        assert row_error(got, np.concatenate(want)).max() <= TOLERANCE[dtype]


def test_greedy_generation_through_the_engine(model_case):
    """submit / step / sample through the scheduler: float32 gives the plain implementation's tokens; two requests at once
    give what each gives alone."""
    from llm_inference_b200 import create_engine

    _, config, folder, sequences, _, w64 = model_case
    prompt, other = sequences["s31"], sequences["s9"]
    want = plain.greedy(config, w64, prompt, 12)
    with create_engine(folder, dtype="float32", max_num_sequences=3, max_model_length=128, kv_cache_bytes=16 << 20, page_size=8,
                       prefill_chunk_size=16, prefill_burst_size=16) as engine:
        assert engine.generate(prompt, 12) == want
        first, second = engine.submit(prompt, 12), engine.submit(other, 7)
        while engine.has_work():
            engine.step()
        assert engine.request(first).output == want
        assert engine.request(second).output == plain.greedy(config, w64, other, 7)
    with create_engine(folder, dtype="bfloat16", max_num_sequences=2, max_model_length=128, kv_cache_bytes=16 << 20, page_size=8) as engine:
        got = engine.generate(prompt, 12)
    tokens = list(prompt)
    for token in got:  # only a near-tie may go the other way in bfloat16
        row = plain.forward(config, w64, tokens)[-1]
        if token != int(np.argmax(row)):
            assert row.max() - row[token] <= 0.2 * row.std()
            break
        tokens.append(token)


def test_command_line_tools_take_the_design(tmp_path):
    """A seeded folder from the named shape, its inspection, greedy generation from the folder and from the shape itself
    (weights drawn on the device), and continuous batching with sampling."""
    run = lambda *args: subprocess.run([sys.executable, "-m", *args], capture_output=True, text=True, timeout=600)
    folder = tmp_path / "model"
    made = run("llm_inference_b200.cli.random_model", "--preset", "tosipel-small", "--seed", "3", "--out", str(folder))
    assert made.returncode == 0, made.stderr[-2000:]
    seen = run("llm_inference_b200.cli.inspect_model", str(folder))
    assert seen.returncode == 0 and "architecture: Tosipel" in seen.stdout and "l1.mix.sink" in seen.stdout, seen.stderr[-2000:]
    ask = ["--prompt-ids", "5,17,3,900,41", "--max-new-tokens", "6", "--max-model-length", "256", "--kv-cache-mib", "64"]
    from_folder = run("llm_inference_b200.cli.generate", "--model", str(folder), *ask)
    from_shape = run("llm_inference_b200.cli.generate", "--random", "tosipel-small", "--weights-seed", "3", *ask)
    assert from_folder.returncode == 0, from_folder.stderr[-2000:]
    assert from_shape.returncode == 0, from_shape.stderr[-2000:]
    for result in (from_folder, from_shape):
        line = json.loads(result.stdout.strip().splitlines()[-1])
        assert line["prompt_tokens"] == 5 and len(line["tokens"]) == 6 and all(0 <= t < 8192 for t in line["tokens"])
    report = tmp_path / "bench.json"
    timed = run("llm_inference_b200.cli.benchmark", "--random", "tosipel-small", "--mix", "6", "--mix-prompt-lengths", "20", "90",
                "--mix-output-lengths", "4", "12", "--max-sequences", "3", "--max-model-length", "256", "--kv-cache-mib", "64", "--warmups", "0",
                "--repetitions", "1", "--output", str(report))
    assert timed.returncode == 0, timed.stderr[-2000:]
    assert report.exists() and json.loads(report.read_text())
