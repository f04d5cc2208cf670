"""A plain, slow Tosipel forward pass in NumPy: one function per mechanism, float64 throughout.

It imports nothing from the engine and the engine imports nothing from here. ``config`` is the
model's config.json as a dict, ``weights`` maps tensor names to arrays. Every mixer keeps what it has
seen in an explicit per-layer state, so a sequence can be fed whole, in portions or token by token.

Notation: ``T`` new tokens, ``D`` the model's width, ``H`` query (or value) heads, ``G`` key/value (or query/key)
heads; a linear weight is ``[out, in]`` and is applied as ``x @ W.T``.
"""

from __future__ import annotations

import numpy as np

F64 = np.float64


def linear(x: np.ndarray, weight: np.ndarray) -> np.ndarray:
    return x.astype(F64) @ weight.astype(F64).T


def sigmoid(x: np.ndarray) -> np.ndarray:
    return 1.0 / (1.0 + np.exp(-x))


def silu(x: np.ndarray) -> np.ndarray:
    return x * sigmoid(x)


def softplus(x: np.ndarray) -> np.ndarray:
    return np.maximum(x, 0.0) + np.log1p(np.exp(-np.abs(x)))


def gelu_tanh(z: np.ndarray) -> np.ndarray:
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z**3)))


def unit_rms(x: np.ndarray, eps: float) -> np.ndarray:
    x = x.astype(F64)
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def plain_norm(x: np.ndarray, weight: np.ndarray, eps: float) -> np.ndarray:
    return unit_rms(x, eps) * weight.astype(F64)


def offset_norm(x: np.ndarray, weight: np.ndarray, eps: float) -> np.ndarray:
    """RMS norm whose weight is stored as an offset from one."""
    return unit_rms(x, eps) * (1.0 + weight.astype(F64))


def _grow(state: dict, name: str, rows: np.ndarray) -> np.ndarray:
    state[name] = rows if name not in state else np.concatenate([state[name], rows])
    return state[name]


# -- attention in a window, with a sink and a gate per head ---------------------------------------------------


def rotate_halves(x: np.ndarray, positions: np.ndarray, rot: dict | None) -> np.ndarray:
    """``x`` is ``[T, heads, size]``; of the first ``dims`` numbers of every head, number ``i`` and number
    ``i + dims / 2`` are rotated by the angle ``position * base^(-2 i / dims)``."""
    if not rot or not rot["dims"]:
        return x
    dims = rot["dims"]
    f = float(rot["base"]) ** (-2.0 * np.arange(dims // 2, dtype=F64) / dims)
    angle = np.asarray(positions, dtype=F64)[:, None, None] * f
    c, s = np.cos(angle), np.sin(angle)
    u, v = x[..., : dims // 2], x[..., dims // 2 : dims]
    return np.concatenate([u * c - v * s, v * c + u * s, x[..., dims:]], axis=-1)


def seen_from(position: int, mask: dict | None) -> int:
    """The first key that a query at ``position`` sees."""
    return max(0, position - mask["size"] + 1) if mask else 0


def softmax_with_sink(scores: np.ndarray, sink: float | None) -> np.ndarray:
    """Weights of the scores; with ``sink`` the denominator has one more term ``exp(sink)``."""
    top = np.max(scores) if sink is None else max(np.max(scores), sink)
    e = np.exp(scores - top)
    return e / (np.sum(e) + (0.0 if sink is None else np.exp(sink - top)))


def attend(q: np.ndarray, keys: np.ndarray, values: np.ndarray, positions, scale: float, mask: dict | None = None, sink=None) -> np.ndarray:
    """``q`` ``[T, H, d]`` at ``positions``; ``keys`` ``[N, G, d]`` and ``values`` ``[N, G, e]`` of positions ``0 .. N - 1``."""
    heads, groups = q.shape[1], keys.shape[1]
    out = np.zeros((q.shape[0], heads, values.shape[2]), dtype=F64)
    for t in range(q.shape[0]):
        p = int(positions[t])
        lo = seen_from(p, mask)
        for h in range(heads):
            g = h // (heads // groups)
            scores = keys[lo : p + 1, g] @ q[t, h] * scale
            out[t, h] = softmax_with_sink(scores, None if sink is None else float(sink[h])) @ values[lo : p + 1, g]
    return out


def window_attention(h: np.ndarray, w: dict, p: str, m: dict, eps: float, positions, state: dict) -> np.ndarray:
    heads, groups, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    count = h.shape[0]
    q = plain_norm(linear(h, w[p + "q"]), w[p + "q.norm"], eps).reshape(count, heads, dim)
    k = plain_norm(linear(h, w[p + "k"]), w[p + "k.norm"], eps).reshape(count, groups, dim)
    v = linear(h, w[p + "v"]).reshape(count, groups, vdim)
    keys = _grow(state, "keys", rotate_halves(k, positions, m.get("rot")))
    values = _grow(state, "values", v)
    out = attend(rotate_halves(q, positions, m.get("rot")), keys, values, positions, m["scale"], m.get("mask"), w[p + "sink"])
    out = out * sigmoid(linear(h, w[p + "g"]))[:, :, None]
    return linear(out.reshape(count, heads * vdim), w[p + "o"])


# -- attention over latents, positions not entering --------------------------------------------------------------


def latent_attention(h: np.ndarray, w: dict, p: str, m: dict, eps: float, positions, state: dict) -> np.ndarray:
    """Keys and values of every token expanded per head from its latent, which is all that is kept."""
    heads, dim, vdim = m["heads"], m["dim"], m["vdim"]
    count = h.shape[0]
    q = linear(plain_norm(linear(h, w[p + "dq"]), w[p + "dq.norm"], eps), w[p + "uq"]).reshape(count, heads, dim)
    c = _grow(state, "latents", plain_norm(linear(h, w[p + "dkv"]), w[p + "dkv.norm"], eps))
    keys = linear(c, w[p + "uk"]).reshape(len(c), heads, dim)
    values = linear(c, w[p + "uv"]).reshape(len(c), heads, vdim)
    out = attend(q, keys, values, positions, m["scale"])
    return linear(out.reshape(count, heads * vdim), w[p + "o"])


# -- the gated delta rule with one decay per head ------------------------------------------------------------------


def short_convolution(x: np.ndarray, taps: np.ndarray, state: dict, name: str) -> np.ndarray:
    """Per channel ``y_t = sum_j taps[:, n - 1 - j] x_(t - j)`` over ``n`` taps, zeros in front of the sequence, then silu."""
    n = taps.shape[1]
    before = state.get(name)
    if before is None:
        before = np.zeros((n - 1, x.shape[1]), dtype=F64)
    rows = np.concatenate([before, x.astype(F64)])
    state[name] = rows[len(rows) - (n - 1) :]
    y = np.zeros((x.shape[0], x.shape[1]), dtype=F64)
    for j in range(n):
        y += taps[:, j].astype(F64) * rows[j : j + x.shape[0]]
    return silu(y)


def unit_vectors(x: np.ndarray) -> np.ndarray:
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + 1e-6)


def delta_step(S: np.ndarray, q: np.ndarray, k: np.ndarray, v: np.ndarray, g: float, beta: float) -> tuple[np.ndarray, np.ndarray]:
    """One token of one head: the state decays, the key's row is corrected towards ``v``, the query reads the new state."""
    S = g * S
    u = beta * (v - S.T @ k)
    S = S + np.outer(k, u)
    return S, S.T @ q


def delta_rule(h: np.ndarray, w: dict, p: str, m: dict, eps: float, positions, state: dict) -> np.ndarray:
    heads, groups, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    count = h.shape[0]
    q = short_convolution(linear(h, w[p + "q"]), w[p + "q.conv"], state, "q").reshape(count, groups, dim)
    k = short_convolution(linear(h, w[p + "k"]), w[p + "k.conv"], state, "k").reshape(count, groups, dim)
    v = short_convolution(linear(h, w[p + "v"]), w[p + "v.conv"], state, "v").reshape(count, heads, vdim)
    q, k = unit_vectors(q) / np.sqrt(float(dim)), unit_vectors(k)
    beta = sigmoid(linear(h, w[p + "b"]))
    g = np.exp(-np.exp(w[p + "A_log"].astype(F64)) * softplus(linear(h, w[p + "a"]) + w[p + "dt_bias"].astype(F64)))
    S = state.setdefault("S", np.zeros((heads, dim, vdim), dtype=F64))
    out = np.zeros((count, heads, vdim), dtype=F64)
    for t in range(count):
        for n in range(heads):
            j = n // (heads // groups)
            S[n], out[t, n] = delta_step(S[n], q[t, j], k[t, j], v[t, n], g[t, n], beta[t, n])
    out = plain_norm(out, w[p + "norm"], eps) * silu(linear(h, w[p + "g"]).reshape(count, heads, vdim))
    return linear(out.reshape(count, heads * vdim), w[p + "o"])


# -- feed-forward, layers, model ------------------------------------------------------------------------------------


def gelu_unit(h: np.ndarray, w: dict, p: str) -> np.ndarray:
    return linear(gelu_tanh(linear(h, w[p + "gate"])) * linear(h, w[p + "up"]), w[p + "down"])


MIXERS = {"attention": window_attention, "latent_attention": latent_attention, "delta": delta_rule}


def owner_of(layers: list, index: int) -> int:
    while layers[index].get("weights_of") is not None:
        index = layers[index]["weights_of"]
    return index


def forward(config: dict, weights: dict, tokens, state: dict | None = None, layer_outputs: list | None = None) -> np.ndarray:
    """Logits ``[T, vocab]`` of ``tokens`` that follow what ``state`` has seen (changed in place)."""
    state = {} if state is None else state
    eps = config["norm"]["eps"]
    w = {name: np.asarray(value, dtype=F64) for name, value in weights.items()}
    start = state.get("count", 0)
    positions = np.arange(start, start + len(tokens))
    state["count"] = start + len(tokens)
    x = w["embed"][np.asarray(tokens)] * float((config.get("embedding") or {}).get("scale", 1.0))
    for index, layer in enumerate(config["layers"]):
        p = f"l{owner_of(config['layers'], index)}."
        own = state.setdefault(index, {})
        branch = MIXERS[layer["type"]](x, w, p + "mix.", layer["mixer"], eps, positions, own)
        x = x + offset_norm(branch, w[p + "norm1"], eps)
        if layer.get("mlp") is not None:
            x = x + offset_norm(gelu_unit(x, w, p + "mlp."), w[p + "norm2"], eps)
        if layer_outputs is not None:
            layer_outputs.append(x.copy())
    return linear(offset_norm(x, w["final.norm"], eps), w["head"])


def greedy(config: dict, weights: dict, prompt, count: int) -> list[int]:
    """``count`` tokens, each the likeliest after everything in front of it."""
    state: dict = {}
    logits = forward(config, weights, prompt, state)[-1]
    out: list[int] = []
    while len(out) < count:
        out.append(int(np.argmax(logits)))
        logits = forward(config, weights, [out[-1]], state)[-1]
    return out
