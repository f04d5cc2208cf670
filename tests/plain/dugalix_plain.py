"""A plain, slow Dugalix forward pass in NumPy: one function per mechanism, float64 throughout.

It imports nothing from the engine and the engine imports nothing from here. ``config`` is the
model's config.json as a dict, ``weights`` maps tensor names to arrays. Every mixer keeps what it has
seen in an explicit per-layer state, so a sequence can be fed whole, in portions or token by token.

Notation: ``T`` new tokens, ``D`` the model's width, ``H`` query heads, ``G`` key/value heads; a linear
weight is ``[out, in]`` and is applied as ``x @ W.T``.
"""

from __future__ import annotations

import numpy as np

F64 = np.float64


def linear(x: np.ndarray, weight: np.ndarray, bias: np.ndarray | None = None) -> np.ndarray:
    y = x.astype(F64) @ weight.astype(F64).T
    return y if bias is None else y + bias.astype(F64)


def sigmoid(x: np.ndarray) -> np.ndarray:
    return 1.0 / (1.0 + np.exp(-x))


def log_sigmoid(x: np.ndarray) -> np.ndarray:
    return np.minimum(x, 0.0) - np.log1p(np.exp(-np.abs(x)))


def softmax(scores: np.ndarray) -> np.ndarray:
    e = np.exp(scores - np.max(scores, axis=-1, keepdims=True))
    return e / np.sum(e, axis=-1, keepdims=True)


def unit_rms(x: np.ndarray, eps: float) -> np.ndarray:
    x = x.astype(F64)
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def offset_norm(x: np.ndarray, weight: np.ndarray, eps: float) -> np.ndarray:
    """RMS norm whose weight is stored as an offset from one."""
    return unit_rms(x, eps) * (1.0 + weight.astype(F64))


def token_shift(h: np.ndarray, shift: np.ndarray, previous: np.ndarray) -> np.ndarray:
    """Row ``t`` blended with row ``t - 1`` (``previous`` in front of row 0), the blend given per column."""
    behind = np.concatenate([previous[None], h[:-1]])
    return h + (behind - h) * shift.astype(F64)


# -- positions ------------------------------------------------------------------------------------------


def rotary_frequencies(dims: int, base: float, scaling: dict | None) -> np.ndarray:
    f = float(base) ** (-2.0 * np.arange(dims // 2, dtype=F64) / max(dims, 1))
    return f / float(scaling["factor"]) if scaling else f


def rotate_halves(x: np.ndarray, positions: np.ndarray, rot: dict | None) -> np.ndarray:
    """``x`` is ``[T, heads, size]``; of the first ``dims`` numbers of every head, number ``i`` and number
    ``i + dims / 2`` are rotated by the angle ``position * f_i``."""
    if not rot or not rot["dims"]:
        return x
    dims = rot["dims"]
    angle = np.asarray(positions, dtype=F64)[:, None, None] * rotary_frequencies(dims, rot["base"], rot.get("scaling"))
    c, s = np.cos(angle), np.sin(angle)
    u, v = x[..., : dims // 2], x[..., dims // 2 : dims]
    return np.concatenate([u * c - v * s, v * c + u * s, x[..., dims:]], axis=-1)


# -- attention over explicit keys and values ------------------------------------------------------------


def visible(position: int, mask: dict | None) -> np.ndarray:
    """Which of the keys ``0 .. position`` a query sees: all, or the last ``size`` and the first ``keep_first``."""
    j = np.arange(position + 1)
    if not mask:
        return np.ones(position + 1, dtype=bool)
    return (position - j < mask["size"]) | (j < mask.get("keep_first", 0))


def attend(q: np.ndarray, keys: np.ndarray, values: np.ndarray, positions, scale: float, mask: dict | None, gate_bias=None) -> np.ndarray:
    """``q`` ``[T, H, d]`` at ``positions``; ``keys`` ``[N, G, d]`` and ``values`` ``[N, G, e]`` of positions ``0 .. N - 1``.
    A softmax over the visible keys, or, with ``gate_bias`` (one number per head), a sigmoid of score plus bias per key."""
    heads, groups = q.shape[1], keys.shape[1]
    out = np.zeros((q.shape[0], heads, values.shape[2]), dtype=F64)
    for t in range(q.shape[0]):
        p = int(positions[t])
        seen = np.flatnonzero(visible(p, mask))
        for h in range(heads):
            g = h // (heads // groups)
            scores = keys[seen, g] @ q[t, h] * scale
            weights = softmax(scores) if gate_bias is None else sigmoid(scores + float(gate_bias[h]))
            out[t, h] = weights @ values[seen, g]
    return out


def _grow(state: dict, name: str, rows: np.ndarray) -> np.ndarray:
    state[name] = rows if name not in state else np.concatenate([state[name], rows])
    return state[name]


def window_attention(h: np.ndarray, w: dict, p: str, m: dict, eps: float, positions, state: dict) -> np.ndarray:
    """Grouped-query softmax attention with biases everywhere, rotation, a sliding window and kept first tokens."""
    heads, groups, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    count = h.shape[0]
    q = rotate_halves(linear(h, w[p + "q"], w[p + "q.b"]).reshape(count, heads, dim), positions, m.get("rot"))
    k = rotate_halves(linear(h, w[p + "k"], w[p + "k.b"]).reshape(count, groups, dim), positions, m.get("rot"))
    v = linear(h, w[p + "v"], w[p + "v.b"]).reshape(count, groups, vdim)
    out = attend(q, _grow(state, "k", k), _grow(state, "v", v), positions, m["scale"], m.get("mask"))
    return linear(out.reshape(count, heads * vdim), w[p + "o"], w[p + "o.b"])


def sigmoid_attention(h: np.ndarray, w: dict, p: str, m: dict, eps: float, positions, state: dict) -> np.ndarray:
    """Grouped-query attention whose values are its keys before rotation and whose weights are sigmoids."""
    heads, groups, dim = m["heads"], m["kv_heads"], m["dim"]
    count = h.shape[0]
    q = rotate_halves(linear(h, w[p + "q"]).reshape(count, heads, dim), positions, m.get("rot"))
    raw = linear(h, w[p + "k"]).reshape(count, groups, dim)
    k = rotate_halves(raw, positions, m.get("rot"))
    out = attend(q, _grow(state, "k", k), _grow(state, "v", raw), positions, m["scale"], m.get("mask"), w[p + "pb"].astype(F64))
    return linear(out.reshape(count, heads * dim), w[p + "o"])


# -- the matrix memory ----------------------------------------------------------------------------------


def memory_step(S: np.ndarray, n: np.ndarray, m: float, q, k, v, i: float, f: float):
    """One token of one head: the new state and the read-out. ``S`` is ``[dim, vdim]``, ``n`` ``[dim]``."""
    m_new = max(f + m, i)
    keep, put = np.exp(f + m - m_new), np.exp(i - m_new)
    S = keep * S + put * np.outer(k, v)
    n = keep * n + put * k
    return S, n, m_new, (S.T @ q) / (max(abs(float(n @ q)), np.exp(-m_new)) + 1e-6)


def matrix_memory(h: np.ndarray, w: dict, p: str, m: dict, eps: float, positions, state: dict) -> np.ndarray:
    heads, dim, vdim, cap = m["heads"], m["dim"], m["vdim"], float(m["gate_cap"])
    count = h.shape[0]
    q = linear(h, w[p + "q"]).reshape(count, heads, dim) * dim**-0.5
    k = linear(h, w[p + "k"]).reshape(count, heads, dim)
    v = linear(h, w[p + "v"]).reshape(count, heads, vdim)
    i = cap * np.tanh(linear(h, w[p + "i"], w[p + "i.b"]) / cap)
    f = log_sigmoid(cap * np.tanh(linear(h, w[p + "f"], w[p + "f.b"]) / cap))
    if "S" not in state:
        state.update(S=np.zeros((heads, dim, vdim)), n=np.zeros((heads, dim)), m=np.zeros(heads))
    out = np.zeros((count, heads, vdim))
    for t in range(count):
        for a in range(heads):
            state["S"][a], state["n"][a], state["m"][a], out[t, a] = memory_step(
                state["S"][a], state["n"][a], state["m"][a], q[t, a], k[t, a], v[t, a], i[t, a], f[t, a])
    out = unit_rms(out, eps).reshape(count, heads * vdim) * w[p + "norm"].astype(F64) * sigmoid(linear(h, w[p + "g"]))
    return linear(out, w[p + "o"])


def side_by_side(h: np.ndarray, w: dict, p: str, m: dict, eps: float, positions, state: dict) -> np.ndarray:
    left = window_attention(h, w, p + "left.", m["left"], eps, positions, state.setdefault("left", {}))
    right = matrix_memory(h, w, p + "right.", m["right"], eps, positions, state.setdefault("right", {}))
    return m["left_scale"] * left + m["right_scale"] * right


MIXERS = {"parallel": side_by_side, "attention": sigmoid_attention}


# -- feed-forward ---------------------------------------------------------------------------------------


def squared_relu_unit(h: np.ndarray, w: dict, p: str) -> np.ndarray:
    return linear(np.maximum(linear(h, w[p + "up"]), 0.0) ** 2, w[p + "down"])


def choice_scores(scores: np.ndarray, correction: np.ndarray, router: dict) -> np.ndarray:
    """Scores plus correction, minus infinity outside the best groups (a group counts by its best member)."""
    choice = scores + correction.astype(F64)
    groups = router.get("groups")
    if groups and groups["count"] > 1:
        by_group = choice.reshape(choice.shape[0], groups["count"], -1)
        order = np.argsort(-by_group.max(axis=-1), axis=-1, kind="stable")[:, : groups["keep"]]
        kept = np.zeros(by_group.shape[:2], dtype=bool)
        np.put_along_axis(kept, order, True, axis=1)
        choice = np.where(kept[:, :, None], by_group, -np.inf).reshape(choice.shape)
    return choice


def route(logits: np.ndarray, correction: np.ndarray, router: dict) -> tuple[np.ndarray, np.ndarray, np.ndarray]:
    """Chosen ids ``[T, top]``, their weights (the softmax scores themselves) and every expert's score."""
    scores = softmax(logits)
    ids = np.argsort(-choice_scores(scores, correction, router), axis=-1, kind="stable")[:, : router["top"]]
    return ids, np.take_along_axis(scores, ids, axis=-1), scores


def choice_margins(scores: np.ndarray, correction: np.ndarray, router: dict) -> np.ndarray:
    """Per token, how far the nearest change of choice is: between the last chosen and the first rejected expert, and
    between the last kept and the first dropped group."""
    out = np.full(scores.shape[0], np.inf)
    ordered = -np.sort(-choice_scores(scores, correction, router), axis=-1)
    if router["top"] < ordered.shape[1]:
        out = np.minimum(out, ordered[:, router["top"] - 1] - ordered[:, router["top"]])
    groups = router.get("groups")
    if groups and groups["keep"] < groups["count"]:
        best = -np.sort(-(scores + correction.astype(F64)).reshape(scores.shape[0], groups["count"], -1).max(axis=-1), axis=-1)
        out = np.minimum(out, best[:, groups["keep"] - 1] - best[:, groups["keep"]])
    return out


def routed_experts(h: np.ndarray, w: dict, p: str, mlp: dict, choices=None, margins=None, free=None) -> np.ndarray:
    """``choices`` (``[T, top]`` ids) replaces the router's own choice (weights are still the scores); ``margins`` receives
    one array per call (:func:`choice_margins`), ``free`` the router's own choices."""
    router = mlp["router"]
    real = router["experts"]
    ids, weights, scores = route(linear(h, w[p + "router"]), w[p + "correction"], router)
    if margins is not None:
        margins.append(choice_margins(scores, w[p + "correction"], router))
    if free is not None:
        free.append(ids.copy())
    if choices is not None:
        ids = np.asarray(choices, dtype=np.int64)
        weights = np.take_along_axis(scores, ids, axis=-1)
    out = np.zeros(h.shape, dtype=F64)
    for t in range(h.shape[0]):
        for j in range(router["top"]):
            e = int(ids[t, j])
            y = h[t] if e >= real else squared_relu_unit(h[t : t + 1], w, f"{p}e{e}.")[0]
            out[t] += weights[t, j] * y
    if mlp.get("shared"):
        out += squared_relu_unit(h, w, p + "shared.") * sigmoid(linear(h, w[p + "shared.sg"].reshape(1, -1)))
    return out


def feed_forward(h: np.ndarray, w: dict, p: str, mlp: dict, **more) -> np.ndarray:
    if mlp["kind"] == "dense":
        return squared_relu_unit(h, w, p)
    return routed_experts(h, w, p, mlp, **more)


# -- the model ------------------------------------------------------------------------------------------


def new_state(config: dict) -> dict:
    return {"position": 0, "layers": [dict() for _ in config["layers"]]}


def forward(config: dict, weights: dict, tokens, state: dict | None = None, *, layer_outputs: list | None = None,
            choices: dict | None = None, margins: list | None = None, free: list | None = None) -> tuple[np.ndarray, dict]:
    """Feed ``tokens`` (the next ones of the sequence ``state`` belongs to; None: a new sequence). Returns the logits
    ``[T, vocab]`` and the state. ``layer_outputs`` receives the stream after every layer; ``choices`` maps a layer index
    to the experts to use; ``margins`` and ``free`` receive one entry per routed layer (see :func:`routed_experts`)."""
    state = new_state(config) if state is None else state
    eps, mult = config["norm"]["eps"], config["residual_mult"]
    tokens = np.asarray(tokens, dtype=np.int64)
    positions = state["position"] + np.arange(tokens.shape[0])
    state["position"] += tokens.shape[0]
    x = weights["embed"].astype(F64)[tokens]
    for index, layer in enumerate(config["layers"]):
        p, own = f"l{index}.", state["layers"][index]
        h = offset_norm(x, weights[p + "norm1"], eps)
        behind = own.get("h", np.zeros(h.shape[1]))
        if h.shape[0]:
            own["h"] = h[-1]
        h = token_shift(h, weights[p + "shift"], behind)
        mixed = MIXERS[layer["type"]](h, weights, p + "mix.", layer["mixer"], eps, positions, own)
        x = x + mult * offset_norm(mixed, weights[p + "norm1b"], eps)
        mlp = layer.get("mlp")
        if mlp is not None:
            more = {}
            if mlp["kind"] == "moe":
                more = dict(choices=None if choices is None else choices.get(index), margins=margins, free=free)
            y = feed_forward(offset_norm(x, weights[p + "norm2"], eps), weights, p + "mlp.", mlp, **more)
            x = x + mult * offset_norm(y, weights[p + "norm2b"], eps)
        if layer_outputs is not None:
            layer_outputs.append(x.copy())
    return linear(offset_norm(x, weights["final.norm"], eps), weights["head"]), state


def greedy(config: dict, weights: dict, prompt, count: int) -> list[int]:
    """``count`` tokens, each the arg-max of the last position's logits, fed back one by one."""
    logits, state = forward(config, weights, prompt)
    out = []
    for _ in range(count):
        out.append(int(np.argmax(logits[-1])))
        logits, state = forward(config, weights, [out[-1]], state)
    return out
