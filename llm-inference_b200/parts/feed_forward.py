"""Feed-forward parts."""

from __future__ import annotations

import torch

from ..weights.loader import TensorSpec
from . import ops
from .base import Part, register_part
from .context import StepContext


class SwiGLU(Part):
    """``down(silu(gate(h)) * up(h))`` without biases (python/instinct/backends/dense.py:124-128).
    The gate and up matrices are stored as one ``[2 * intermediate, hidden]`` matrix with their
    rows interleaved (row 2j is gate_j, row 2j + 1 is up_j), so one matrix product yields each
    gate next to its up value and the activation can run in that product's epilogue."""

    activation = "silu"
    names = ("gate_proj.weight", "up_proj.weight", "down_proj.weight")

    def __init__(self, *, prefix: str, hidden_size: int, intermediate_size: int) -> None:
        self.prefix, self.hidden_size, self.intermediate_size = prefix, hidden_size, intermediate_size
        self.w_gate_up = self.w_down = None

    def tensor_specs(self) -> list[TensorSpec]:
        p, h, i = self.prefix, self.hidden_size, self.intermediate_size
        return [
            TensorSpec(p + self.names[0], (i, h)),
            TensorSpec(p + self.names[1], (i, h)),
            TensorSpec(p + self.names[2], (h, i)),
        ]

    def load(self, tensors, dtype, device) -> None:
        p = self.prefix
        gate, up = (tensors[p + n].to(device=device, dtype=dtype) for n in self.names[:2])
        self.w_gate_up = torch.stack([gate, up], dim=1).reshape(2 * self.intermediate_size, self.hidden_size).contiguous()
        self.w_down = tensors[p + self.names[2]].to(device=device, dtype=dtype).contiguous()

    def weight_bytes(self) -> int:
        return (self.w_gate_up.numel() + self.w_down.numel()) * self.w_down.element_size()

    takes_folded = True  # `h` may be ops.FoldedRows: the gate/up product applies the norm's 1 / rms
    takes_sink = True  # with a sink the down product adds into the residual stream itself

    def forward(self, ctx: StepContext, h, sink: ops.ResidualSink | None = None):
        t, i = ctx.num_tokens, self.intermediate_size
        act = ctx.buffer("act", (t, i))
        if not ops.linear_gated(ctx, h, self.w_gate_up, act, self.activation):
            gate_up = ops.linear(ctx, h, self.w_gate_up, ctx.buffer("gate_up", (t, 2 * i)))
            ops.gated_mul(ctx, gate_up, act, self.activation)
        if sink is not None:
            folded = ops.linear_into_residual(ctx, act, self.w_down, sink)
            if folded is not None:
                return folded
        return ops.linear(ctx, act, self.w_down, ctx.buffer("branch", (t, self.hidden_size)))


class GeGLU(SwiGLU):
    """``down(gelu(gate(h)) * up(h))`` without biases, ``gelu`` in its tanh form: the same products with another activation
    in the first one's epilogue (which has no form for a folded norm's rows). Tensor names: ``prefix + gate | up | down``."""

    activation = "gelu"
    names = ("gate", "up", "down")
    takes_folded = False


class PolyNormFeedForward(Part):
    """``down(act(up(h)))`` without biases, ``act(z) = a N(z) + b N(z^2) + c N(z^3) + e`` with powers
    taken element by element and ``N`` dividing a token's row by its root mean square
    (``eps`` inside the root); ``a, b, c, e`` are the four numbers of the ``act`` tensor."""

    def __init__(self, *, prefix: str, hidden_size: int, intermediate_size: int, eps: float) -> None:
        self.prefix, self.hidden_size, self.intermediate_size, self.eps = prefix, hidden_size, intermediate_size, float(eps)
        self.w_up = self.w_down = self.coefficients = None

    def tensor_specs(self) -> list[TensorSpec]:
        p, h, i = self.prefix, self.hidden_size, self.intermediate_size
        return [TensorSpec(f"{p}up", (i, h)), TensorSpec(f"{p}down", (h, i)), TensorSpec(f"{p}act", (4,), init="half_plus_normal")]

    def load(self, tensors, dtype, device) -> None:
        p = self.prefix
        self.w_up = tensors[f"{p}up"].to(device=device, dtype=dtype).contiguous()
        self.w_down = tensors[f"{p}down"].to(device=device, dtype=dtype).contiguous()
        self.coefficients = tensors[f"{p}act"].to(device=device, dtype=torch.float32).contiguous()

    def weight_bytes(self) -> int:
        return (self.w_up.numel() + self.w_down.numel()) * self.w_down.element_size()

    def forward(self, ctx: StepContext, h: torch.Tensor) -> torch.Tensor:
        t, i = ctx.num_tokens, self.intermediate_size
        z = ops.linear(ctx, h, self.w_up, ctx.buffer("ff_up", (t, i)))
        act = ops.poly_norm(ctx, z, self.coefficients, self.eps, ctx.buffer("act", (t, i)))
        return ops.linear(ctx, act, self.w_down, ctx.buffer("branch", (t, self.hidden_size)))


class ClampedGLU(Part):
    """``down(y)`` with ``g = min(gate(h), limit)``, ``u = clamp(up(h), -limit, limit)``, ``y = g * sigmoid(1.702 g) * (u + 1)``,
    no biases. The gate and up matrices are one ``[2 * intermediate, hidden]`` matrix (gate rows first), so one
    product gives both. Tensor names: ``prefix + gate | up | down``."""

    def __init__(self, *, prefix: str, hidden_size: int, intermediate_size: int, limit: float) -> None:
        self.prefix, self.hidden_size, self.intermediate_size, self.limit = prefix, hidden_size, int(intermediate_size), float(limit)
        self.w_gate_up = self.w_down = None

    def tensor_specs(self) -> list[TensorSpec]:
        p, h, i = self.prefix, self.hidden_size, self.intermediate_size
        return [TensorSpec(p + "gate", (i, h)), TensorSpec(p + "up", (i, h)), TensorSpec(p + "down", (h, i))]

    def load(self, tensors, dtype, device) -> None:
        p = self.prefix
        self.w_gate_up = torch.cat([tensors[p + "gate"].to(device=device, dtype=dtype), tensors[p + "up"].to(device=device, dtype=dtype)]).contiguous()
        self.w_down = tensors[p + "down"].to(device=device, dtype=dtype).contiguous()

    def weight_bytes(self) -> int:
        return (self.w_gate_up.numel() + self.w_down.numel()) * self.w_down.element_size()

    def forward(self, ctx: StepContext, h: torch.Tensor) -> torch.Tensor:
        t, i = ctx.num_tokens, self.intermediate_size
        gate_up = ops.linear(ctx, h, self.w_gate_up, ctx.buffer("gate_up", (t, 2 * i)))
        act = ops.clamped_glu(ctx, gate_up, self.limit, ctx.buffer("act", (t, i)))
        return ops.linear(ctx, act, self.w_down, ctx.buffer("branch", (t, self.hidden_size)))


class RoutedExperts(Part):
    """A mixture of ``experts`` small gated feed-forward layers of which each token uses ``top``, plus an
    optional shared expert that every token uses.

    Expert (no biases): ``g = min(W_gate h, limit)``, ``u = clamp(W_up h, -limit, limit)``,
    ``y = g * sigmoid(1.702 g) * (u + 1)``, output ``W_down y``. Router, in 32-bit: ``s = sigmoid(W_router h)``;
    the experts form ``group_count`` equal groups of neighbours, a group scores the sum of its two
    largest ``s``, and only experts of the ``group_keep`` best groups can be chosen; the ``top`` largest
    ``s`` among them are chosen and weighted ``s / (sum of the chosen s + 1e-20) * route_scale``. The output
    is the weighted sum of the chosen experts' outputs plus the shared expert's.

    ``router="softmax_chosen"`` is another router: the ``top`` largest logits ``W_router h`` (+ ``router.b`` with
    ``router_bias``) are chosen and weighted by the softmax over the chosen logits alone (times ``route_scale``); it has no
    groups. ``router="softmax_all"`` is a third: scores are the softmax over all experts, ``correction`` (with ``router_bias``) is
    added to the scores that compete only, a group counts by the largest of them, and a chosen expert's weight is its score
    (times ``route_scale``), not renormalised. A ``limit`` of zero makes an expert ``W_down (silu(W_gate h) * (W_up h))``, without clamps. ``out_name`` is the
    buffer the result goes to (a layer that runs its feed-forward beside its mixer gives it one of its own).

    ``activation="squared_relu"``: experts (and the shared one) are ungated, ``W_down max(W_up h, 0)^2``. The last ``identity``
    of the ``experts + identity`` the router chooses from are identity experts: their output is ``h``. ``shared_gate``: the
    shared expert's output is multiplied by ``sigmoid(W_sg h)``, one number per token; its row is one more of the router's
    product.

    The experts' matrices are stacked (``[experts, 2 ff, hidden]`` with the gate rows first, and
    ``[experts, hidden, ff]``); a step sorts its (token, choice) pairs by expert and the two products
    walk the sorted runs, so only chosen experts' weights are read. Tensor names: ``prefix + router |
    router.b (or correction) | e<j>.{gate,up,down} | shared.{gate,up,down,sg}``."""

    def __init__(self, *, prefix: str, hidden_size: int, experts: int, top: int, intermediate_size: int, limit: float,
                 route_scale: float = 1.0, group_count: int = 1, group_keep: int = 1, shared_size: int | None = None,
                 shared_limit: float | None = None, router: str = "sigmoid_groups", router_bias: bool = False,
                 out_name: str = "branch", activation: str = "gated", identity: int = 0, shared_gate: bool = False) -> None:
        if router not in ("sigmoid_groups", "softmax_chosen", "softmax_all"):
            raise ValueError(f"router={router!r} must be 'sigmoid_groups', 'softmax_chosen' or 'softmax_all'")
        if activation not in ("gated", "squared_relu"):
            raise ValueError(f"activation={activation!r} must be 'gated' or 'squared_relu'")
        if shared_gate and not shared_size:
            raise ValueError("a gate on the shared expert wants a shared expert")
        if router == "softmax_chosen" and (group_count != 1 or group_keep != 1):
            raise ValueError("the router that weighs by a softmax over the chosen logits has no groups")
        self.prefix, self.hidden_size = prefix, hidden_size
        self.router, self.router_bias, self.out_name = router, bool(router_bias), out_name
        self.bias_name = "correction" if router == "softmax_all" else "router.b"
        self.gated, self.identity, self.shared_gate = activation == "gated", int(identity), bool(shared_gate)
        self.choices = int(experts) + self.identity  # what the router chooses from
        self.b_router = None
        self.experts, self.top, self.intermediate_size, self.limit = int(experts), int(top), int(intermediate_size), float(limit)
        self.route_scale, self.group_count, self.group_keep = float(route_scale), int(group_count), int(group_keep)
        self.shared_size = int(shared_size) if shared_size else 0
        self.shared_limit = float(shared_limit) if shared_limit is not None else self.limit
        self.w_router = self.w_gate_up = self.w_down = self.w_shared_gate_up = self.w_shared_down = None

    def tensor_specs(self) -> list[TensorSpec]:
        p, h, i = self.prefix, self.hidden_size, self.intermediate_size
        specs = [TensorSpec(p + "router", (self.choices, h))]
        if self.router_bias:
            specs.append(TensorSpec(p + self.bias_name, (self.choices,)))

        def unit(name: str, size: int) -> list[TensorSpec]:
            front = ("gate", "up") if self.gated else ("up",)
            return [TensorSpec(f"{p}{name}.{part}", (size, h)) for part in front] + [TensorSpec(f"{p}{name}.down", (h, size))]

        for e in range(self.experts):
            specs += unit(f"e{e}", i)
        if self.shared_size:
            specs += unit("shared", self.shared_size)
        if self.shared_gate:
            specs.append(TensorSpec(p + "shared.sg", (1, h)))
        return specs

    def load(self, tensors, dtype, device) -> None:
        p = self.prefix

        def get(name: str) -> torch.Tensor:
            return tensors[p + name].to(device=device, dtype=dtype)

        self.w_router = torch.cat([get("router"), get("shared.sg")]).contiguous() if self.shared_gate else get("router").contiguous()
        if self.router_bias:
            self.b_router = tensors[p + self.bias_name].to(device=device, dtype=torch.float32).contiguous()

        def front(name: str) -> torch.Tensor:
            return torch.cat([get(name + ".gate"), get(name + ".up")]) if self.gated else get(name + ".up")

        self.w_gate_up = torch.stack([front(f"e{e}") for e in range(self.experts)]).contiguous()
        self.w_down = torch.stack([get(f"e{e}.down") for e in range(self.experts)]).contiguous()
        if self.shared_size:
            self.w_shared_gate_up = front("shared").contiguous()
            self.w_shared_down = get("shared.down").contiguous()

    def weight_bytes(self) -> int:
        """What a step reads at most: the router, the shared expert and ``top`` experts per token is the
        least; counted here is the router, the shared expert and every expert once."""
        tensors = [self.w_router, self.w_gate_up, self.w_down, self.w_shared_gate_up, self.w_shared_down]
        return sum(w.numel() * w.element_size() for w in tensors if w is not None)

    def forward(self, ctx: StepContext, h: torch.Tensor) -> torch.Tensor:
        t, width = ctx.num_tokens, self.hidden_size
        logits = ops.linear(ctx, h, self.w_router, ctx.buffer("moe_logits", (t, self.w_router.shape[0]), torch.float32))
        # Every routed layer keeps the step's choices in a buffer of its own, so that they can be read after
        # the step (expert load statistics, tests), also when the step was replayed from a captured graph.
        ids = ctx.buffer("moe_ids:" + self.prefix, (t, self.top), torch.int32)
        weights = ctx.buffer("moe_weights", (t, self.top), torch.float32)
        ops.moe_route(ctx, logits[:, : self.choices], self.group_count, self.group_keep, self.top, self.route_scale, ids, weights, bias=self.b_router,
                      softmax_chosen=self.router == "softmax_chosen", softmax_all=self.router == "softmax_all")
        expert_out = ops.moe_experts(
            ctx, h, ids, self.w_gate_up, self.w_down, self.limit, ctx.buffer("moe_expert_out", (t * self.top, width), torch.float32, per_token=False)
        )
        shared = None
        if self.shared_size:
            if self.gated:
                gate_up = ops.linear(ctx, h, self.w_shared_gate_up, ctx.buffer("gate_up", (t, 2 * self.shared_size)))
                act = ops.clamped_glu(ctx, gate_up, self.shared_limit, ctx.buffer("act", (t, self.shared_size)))
            else:
                act = ops.linear_squared_relu(ctx, h, self.w_shared_gate_up, ctx.buffer("act", (t, self.shared_size)))
            shared = ops.linear(ctx, act, self.w_shared_down, ctx.buffer("moe_shared", (t, width)))
        return ops.moe_combine(
            ctx, expert_out, weights, shared, ctx.buffer(self.out_name, (t, width)),
            identity=(ids, self.experts, h) if self.identity else None, shared_gate=logits[:, self.choices] if self.shared_gate else None,
        )


class SquaredReLUFeedForward(Part):
    """``down(max(up(h), 0)^2)`` without biases. Tensor names: ``prefix + up | down``."""

    def __init__(self, *, prefix: str, hidden_size: int, intermediate_size: int) -> None:
        self.prefix, self.hidden_size, self.intermediate_size = prefix, hidden_size, int(intermediate_size)
        self.w_up = self.w_down = None

    def tensor_specs(self) -> list[TensorSpec]:
        p, h, i = self.prefix, self.hidden_size, self.intermediate_size
        return [TensorSpec(p + "up", (i, h)), TensorSpec(p + "down", (h, i))]

    def load(self, tensors, dtype, device) -> None:
        self.w_up, self.w_down = (tensors[self.prefix + n].to(device=device, dtype=dtype).contiguous() for n in ("up", "down"))

    def weight_bytes(self) -> int:
        return (self.w_up.numel() + self.w_down.numel()) * self.w_down.element_size()

    def forward(self, ctx: StepContext, h: torch.Tensor) -> torch.Tensor:
        t = ctx.num_tokens
        act = ops.linear_squared_relu(ctx, h, self.w_up, ctx.buffer("act", (t, self.intermediate_size)))
        return ops.linear(ctx, act, self.w_down, ctx.buffer("branch", (t, self.hidden_size)))


register_part("feed_forward", "swiglu", SwiGLU)
register_part("feed_forward", "geglu", GeGLU)
register_part("feed_forward", "poly_norm", PolyNormFeedForward)
register_part("feed_forward", "routed_experts", RoutedExperts)
register_part("feed_forward", "clamped_glu", ClampedGLU)
register_part("feed_forward", "squared_relu", SquaredReLUFeedForward)
