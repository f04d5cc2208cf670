"""Small Tosipel configurations and weights drawn here (not by the engine)."""

from __future__ import annotations

import numpy as np
import torch


def attention(heads=6, kv_heads=2, dim=16, vdim=24, scale=0.5, size=20, rot=(8, 100.0)) -> dict:
    """``size``: keys in the window or None; ``rot``: (dims, base) or None."""
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if size:
        mixer["mask"] = {"size": size}
    if rot:
        mixer["rot"] = {"dims": rot[0], "base": rot[1]}
    return {"type": "attention", "mixer": mixer}


def latent(heads=3, dim=12, vdim=20, kv_rank=28, q_rank=36, scale=0.4) -> dict:
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "scale": scale}}


def delta(heads=6, kv_heads=3, dim=12, vdim=20, conv=4) -> dict:
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def with_mlp(layer: dict, ff: int | None) -> dict:
    return dict(layer, mlp=None if ff is None else {"kind": "dense", "ff": ff})


def same_as(layers: list[dict], index: int) -> dict:
    """A layer that runs layer ``index``'s tensors against a cache or state of its own."""
    return dict(layers[index], weights_of=index)


def config_of(width, vocab, layers, eps=1e-5, scale=3.0) -> dict:
    return {"architecture": "Tosipel", "vocab": vocab, "width": width, "embedding": {"scale": scale}, "norm": {"eps": eps}, "layers": layers}


# Four configurations that differ in every size. ALPHA: all three mixers, a layer without a feed-forward, layers that run an
# attention's, a latent attention's and a delta rule's tensors again, windows that end inside pages.
_ALPHA = [
    with_mlp(attention(), 72),
    with_mlp(delta(), None),
    with_mlp(latent(), 60),
    with_mlp(delta(4, 1, 20, 28, 2), 40),
]
ALPHA = config_of(48, 97, _ALPHA + [same_as(_ALPHA, 0), same_as(_ALPHA, 3), same_as(_ALPHA, 2)])
# BETA: the delta rule last, one head each, a single tap (no convolution history), an odd state, no window, no rotation, a
# window of one, more than eight heads on a q/k head, a chain of layers on the same tensors, feed-forwards of odd size.
_BETA = [
    with_mlp(latent(1, 7, 5, 33, 9, 0.9), 33),
    with_mlp(attention(5, 1, 10, 6, 0.7, None, None), None),
    with_mlp(delta(9, 1, 15, 19, 1), 26),
    with_mlp(attention(3, 3, 8, 136, 0.8, 1, (2, 7.0)), 50),
    with_mlp(delta(1, 1, 33, 26, 5), None),
]
BETA = config_of(40, 131, _BETA + [same_as(_BETA, 1), dict(same_as(_BETA, 1), weights_of=5)], eps=3e-4, scale=1.0)
# GAMMA: sizes that the tensor-core kernels take (heads of 64, 128 and 192, latents of multiples of 32), a window that is no
# multiple of a tile, a state whose rows fill whole warps.
_GAMMA = [
    with_mlp(delta(4, 2, 64, 128, 4), 96),
    with_mlp(attention(6, 2, 64, 48, 0.3, 45, (32, 1e4)), 128),
    with_mlp(latent(5, 24, 32, 96, 64, 0.3), 64),
    with_mlp(attention(4, 2, 112, 128, 0.2, 70, (112, 2e5)), 80),
    with_mlp(attention(4, 1, 64, 160, 0.25, 31, (16, 500.0)), None),
    with_mlp(delta(2, 2, 128, 64, 3), None),
]
GAMMA = config_of(64, 113, _GAMMA, eps=1e-6, scale=8.0)
# DELTA: sizes that are multiples of nothing in particular.
_DELTA = [
    with_mlp(delta(3, 3, 9, 11, 3), 23),
    with_mlp(latent(3, 10, 14, 37, 19, 0.6), 31),
    with_mlp(attention(3, 1, 18, 14, 0.6, 7, (6, 77.0)), 29),
    with_mlp(delta(6, 2, 17, 35, 2), 45),
]
DELTA = config_of(50, 101, _DELTA + [same_as(_DELTA, 1)], eps=2e-6, scale=0.5)
CONFIGS = {"alpha": ALPHA, "beta": BETA, "gamma": GAMMA, "delta": DELTA}


def draw_weights(config: dict, seed: int) -> dict[str, torch.Tensor]:
    """bfloat16 weights at the scales of a trained model, by tensor name: linear weights N(0, 1/in) times a gain, scores a few
    units wide (so that a softmax picks few keys and a wrong or missing key moves the result), sinks of the size of a
    large score, taps around "the current token", decays from heads that forget in a few tokens to heads that keep hundreds."""
    rng = np.random.default_rng(seed)
    width, vocab = config["width"], config["vocab"]
    out: dict[str, np.ndarray] = {}

    def linear(name, rows, cols, gain=1.0):
        out[name] = rng.normal(0.0, gain / np.sqrt(cols), (rows, cols))

    def vector(name, count, spread=0.2, mean=0.0):
        out[name] = mean + rng.normal(0.0, spread, count)

    out["embed"] = rng.normal(0.0, 1.0 / config["embedding"]["scale"], (vocab, width))
    linear("head", vocab, width, 2.0)
    vector("final.norm", width)
    for index, layer in enumerate(config["layers"]):
        if layer.get("weights_of") is not None:
            continue
        p, m = f"l{index}.", layer["mixer"]
        q, heads, dim, vdim = p + "mix.", m["heads"], m["dim"], m["vdim"]
        vector(p + "norm1", width)
        linear(q + "o", width, heads * vdim)
        if layer["type"] == "attention":
            kvh = m["kv_heads"]
            sharp = np.sqrt(2.5 / (m["scale"] * np.sqrt(dim)))  # q . k * scale has a spread of about 2.5
            for name, rows in (("q", heads * dim), ("k", kvh * dim), ("v", kvh * vdim)):
                linear(q + name, rows, width, 0.3 if name == "q" else 1.5)
            vector(q + "q.norm", heads * dim, 0.2 * sharp, sharp), vector(q + "k.norm", kvh * dim, 0.2 * sharp, sharp)
            vector(q + "sink", heads, 1.0, 2.5)
            linear(q + "g", heads, width, 2.0)
        elif layer["type"] == "latent_attention":
            rank, q_rank = m["kv_rank"], m["q_rank"]
            sharp = np.sqrt(2.5 / (m["scale"] * np.sqrt(dim)))
            linear(q + "dq", q_rank, width, 0.4), vector(q + "dq.norm", q_rank, 0.2, 1.0), linear(q + "uq", heads * dim, q_rank, sharp)
            linear(q + "dkv", rank, width, 2.0), vector(q + "dkv.norm", rank, 0.2, 1.0)
            linear(q + "uk", heads * dim, rank, sharp), linear(q + "uv", heads * vdim, rank)
        else:
            kvh, taps = m["kv_heads"], m["conv"]
            for name, rows in (("q", kvh * dim), ("k", kvh * dim), ("v", heads * vdim)):
                linear(q + name, rows, width, 2.0)
                out[q + name + ".conv"] = rng.normal(0.0, 0.5, (rows, taps)) + np.eye(1, taps, taps - 1)
            # q leans towards k: a first token's read-out is (k . q) times its value and then normed, so where k . q nearly
            # vanishes rounding decides its sign
            out[q + "q"] = out[q + "q"] * 0.7 + out[q + "k"] * 0.8
            out[q + "q.conv"] = out[q + "q.conv"] * 0.5 + out[q + "k.conv"] * 0.5
            linear(q + "b", heads, width, 1.5), linear(q + "a", heads, width, 1.5)
            out[q + "A_log"] = rng.permutation(np.linspace(-4.5, 0.5, heads)) if heads > 1 else np.array([-2.0])
            vector(q + "dt_bias", heads, 1.0, -1.0), vector(q + "norm", vdim, 0.2, 1.0)
            linear(q + "g", heads * vdim, width, 2.0)
        if layer.get("mlp") is not None:
            ff = layer["mlp"]["ff"]
            vector(p + "norm2", width)
            linear(p + "mlp.gate", ff, width, 1.5), linear(p + "mlp.up", ff, width, 1.5), linear(p + "mlp.down", width, ff)
    return {name: torch.from_numpy(np.ascontiguousarray(value)).to(torch.bfloat16) for name, value in out.items()}
