"""Small Dugalix configurations and weights drawn here (not by the engine)."""

from __future__ import annotations

import numpy as np
import torch


def softmax_attention(heads=4, kv_heads=2, dim=16, vdim=24, scale=0.6, mask=(20, 5), rot=(8, 100.0, 3.0)):
    """``mask``: (size, first tokens kept) or None; ``rot``: (dims, base, factor or None) or None."""
    out = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if mask:
        out["mask"] = {"size": mask[0]}
        if mask[1] is not None:
            out["mask"]["keep_first"] = mask[1]
    if rot:
        out["rot"] = {"dims": rot[0], "base": rot[1]}
        if rot[2]:
            out["rot"]["scaling"] = {"factor": rot[2]}
    return out


def memory(heads=3, dim=12, vdim=20, gate_cap=6.0):
    return {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": gate_cap}


def pair_layer(left=None, right=None, left_scale=0.8, right_scale=1.1):
    mixer = {"left": left or softmax_attention(), "right": right or memory(), "left_scale": left_scale, "right_scale": right_scale}
    return {"type": "parallel", "mixer": mixer}


def sigmoid_layer(heads=4, kv_heads=1, dim=24, scale=0.5, size=17, rot=(8, 50.0, None)):
    mixer = softmax_attention(heads, kv_heads, dim, dim, scale, (size, None) if size else None, rot)
    return {"type": "attention", "mixer": mixer}


def dense(ff=60):
    return {"kind": "dense", "ff": ff}


def moe(experts=6, top=2, ff=20, shared=12, identity=2, groups=(2, 1)):
    router = {"experts": experts, "top": top}
    if identity:
        router["identity"] = identity
    if groups:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    mlp = {"kind": "moe", "expert": {"ff": ff}, "router": router}
    if shared:
        mlp["shared"] = {"ff": shared}
    return mlp


def with_mlp(layer: dict, mlp: dict | None) -> dict:
    return dict(layer, mlp=mlp)


def config_of(width, vocab, layers, eps=1e-5, mult=0.7) -> dict:
    return {"architecture": "Dugalix", "vocab": vocab, "width": width, "residual_mult": mult, "norm": {"eps": eps}, "layers": layers}


# Four configurations that differ in every size. ALPHA: both kinds of layer, routed and dense feed-forwards, a layer
# without one; windows and kept tokens that end inside pages.
ALPHA = config_of(
    48, 97,
    [
        with_mlp(pair_layer(), dense()),
        with_mlp(sigmoid_layer(), moe()),
        with_mlp(pair_layer(softmax_attention(6, 3, 8, 8, 1.0, (9, 0), (8, 30.0, None)), memory(2, 8, 8, 3.0), -0.5, 0.9), None),
        with_mlp(sigmoid_layer(2, 2, 16, 0.7, 33, (16, 1000.0, 2.5)), moe(5, 3, 28, None, 1, (3, 2))),
    ],
)
# BETA: a sigmoid layer first, one head, odd sizes, no mask, no rotation, every expert chosen, only identity experts beside
# one, kept tokens beyond a page and beyond the window, values wider than 128, a residual factor of 1.
BETA = config_of(
    40, 131,
    [
        with_mlp(sigmoid_layer(1, 1, 6, 1.2, 0, None), moe(1, 1, 70, 9, 3, None)),
        with_mlp(pair_layer(softmax_attention(3, 3, 8, 136, 0.9, (4, 11), (4, 10.0, 1.5)), memory(1, 5, 7, 15.0), 1.0, 1.0), moe(4, 4, 33, 40, 0, (4, 4))),
        with_mlp(pair_layer(softmax_attention(5, 1, 10, 6, 0.7, None, None), memory(4, 33, 3, 8.0), 0.3, -2.0), dense(33)),
        with_mlp(sigmoid_layer(5, 5, 8, 1.0, 1, (2, 7.0, None)), None),
    ],
    eps=3e-4, mult=1.0,
)
# GAMMA: sizes the tensor-core kernels take (heads of 64, 128 and 192), a window that is no multiple of a tile, kept
# tokens, a memory whose rows fill whole warps.
GAMMA = config_of(
    64, 113,
    [
        with_mlp(pair_layer(softmax_attention(3, 1, 64, 128, 0.3, (70, 3), (64, 1e4, 4.0)), memory(2, 128, 64, 9.0), 0.9, 0.6), moe(12, 3, 32, 64, 4, (2, 1))),
        with_mlp(sigmoid_layer(4, 2, 64, 0.3, 45, (16, 500.0, None)), dense(96)),
        with_mlp(pair_layer(softmax_attention(4, 2, 80, 176, 0.25, (31, 18), (32, 2e5, 8.0)), memory(4, 64, 32, 12.0), 0.7, 0.4), moe(6, 2, 48, 16, 2, (4, 3))),
        with_mlp(sigmoid_layer(2, 2, 128, 0.2, 90, (128, 1e6, None)), moe(8, 2, 16, None, 0, None)),
    ],
    mult=0.4,
)
# DELTA: sizes that are multiples of nothing in particular.
DELTA = config_of(
    50, 101,
    [
        with_mlp(pair_layer(softmax_attention(3, 3, 10, 14, 0.6, (5, 1), (6, 77.0, 1.7)), memory(3, 9, 11, 4.5), 1.3, 0.2), moe(3, 2, 18, 9, 2, (5, 4))),
        with_mlp(sigmoid_layer(6, 3, 18, 0.5, 7, (10, 9.0, 6.0)), moe(7, 3, 10, 5, 0, (7, 3))),
        with_mlp(pair_layer(softmax_attention(2, 1, 14, 7, 0.8, (23, 9), (14, 40.0, None)), memory(1, 2, 50, 2.0), 0.6, 1.7), dense(26)),
    ],
    eps=2e-6, mult=1.25,
)
CONFIGS = {"alpha": ALPHA, "beta": BETA, "gamma": GAMMA, "delta": DELTA}


def draw_weights(config: dict, seed: int) -> dict[str, torch.Tensor]:
    """bfloat16 weights at the scales of a trained model, by tensor name: linear weights N(0, 1/in) times a gain, norm
    weights around zero, biases of a size that shows, blends with the previous token between 0 and 1, forget gates from
    heads that forget in a few tokens to heads that keep hundreds, router logits wide enough that choices are clear."""
    rng = np.random.default_rng(seed)
    width, vocab = config["width"], config["vocab"]
    out: dict[str, np.ndarray] = {}

    def linear(name, rows, cols, gain=1.0):
        out[name] = rng.normal(0.0, gain / np.sqrt(cols), (rows, cols))

    def vector(name, count, spread=0.5, mean=0.0):
        out[name] = mean + rng.normal(0.0, spread, count)

    def attention(p, m, biases):
        heads, kvh, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        # scores a few units wide whatever the sizes: q . k * scale has a spread of about 3
        gain = np.sqrt(3.0 / (m["scale"] * np.sqrt(dim)))
        linear(p + "q", heads * dim, width, gain), linear(p + "k", kvh * dim, width, gain)
        linear(p + "o", width, heads * vdim)
        if biases:
            linear(p + "v", kvh * vdim, width)
            for name, count in (("q.b", heads * dim), ("k.b", kvh * dim), ("v.b", kvh * vdim), ("o.b", width)):
                vector(p + name, count)
        else:
            vector(p + "pb", heads, 0.7, -1.5)

    def unit(p, ff, gain=1.5):
        linear(p + "up", ff, width, gain), linear(p + "down", width, ff)

    out["embed"] = rng.normal(0.0, 1.0, (vocab, width))
    linear("head", vocab, width)
    vector("final.norm", width, 0.2)
    for index, layer in enumerate(config["layers"]):
        p, m = f"l{index}.", layer["mixer"]
        vector(p + "norm1", width, 0.2), vector(p + "norm1b", width, 0.2)
        out[p + "shift"] = rng.uniform(0.0, 1.0, width)
        if layer["type"] == "attention":
            attention(p + "mix.", m, biases=False)
        else:
            attention(p + "mix.left.", m["left"], biases=True)
            r, q = m["right"], p + "mix.right."
            heads, dim, vdim = r["heads"], r["dim"], r["vdim"]
            linear(q + "q", heads * dim, width, 1.5), linear(q + "k", heads * dim, width, 1.5), linear(q + "v", heads * vdim, width)
            linear(q + "g", heads * vdim, width, 2.0), linear(q + "o", width, heads * vdim), vector(q + "norm", heads * vdim, 0.2, 1.0)
            linear(q + "i", heads, width, 1.5), linear(q + "f", heads, width)
            vector(q + "i.b", heads, 1.0)
            out[q + "f.b"] = rng.permutation(np.linspace(0.5, 5.0, heads))
        mlp = layer.get("mlp")
        if mlp is None:
            continue
        vector(p + "norm2", width, 0.2), vector(p + "norm2b", width, 0.2)
        if mlp["kind"] == "dense":
            unit(p + "mlp.", mlp["ff"])
            continue
        choices = mlp["router"]["experts"] + mlp["router"].get("identity", 0)
        linear(p + "mlp.router", choices, width, 2.0)
        vector(p + "mlp.correction", choices, 0.15)
        for e in range(mlp["router"]["experts"]):
            unit(f"{p}mlp.e{e}.", mlp["expert"]["ff"])
        if mlp.get("shared"):
            unit(p + "mlp.shared.", mlp["shared"]["ff"]), linear(p + "mlp.shared.sg", 1, width, 2.0)
    return {name: torch.from_numpy(np.ascontiguousarray(value)).to(torch.bfloat16) for name, value in out.items()}
