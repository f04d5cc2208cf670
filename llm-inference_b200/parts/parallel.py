"""A mixer that is two mixers side by side."""

from __future__ import annotations

import torch

from ..weights.loader import TensorSpec
from . import ops
from .base import CacheSpecs, Part, PartSpec, build_part, register_part
from .context import CacheView, StepContext


class ParallelMixers(Part):
    """Two mixers read the same input; the result is ``(w_a * a / rms(a) + w_b * b / rms(b)) / 2`` with ``a`` and ``b``
    their outputs, each divided by its root mean square over the model width (``eps`` inside the root) and
    multiplied by a weight per column (tensors ``names[0]``, ``names[1]``).

    Each member keeps its own cache entry (:class:`CacheSpecs`). What the part returns is :class:`ops.BranchPair`,
    the two outputs not yet combined: the norm that adds the layer's result to the stream combines them in the
    same kernel, in 32-bit.

    With ``scales`` instead of ``names`` the result is ``scales[0] * a + scales[1] * b`` and what is returned
    :class:`ops.ScaledPair`; a member's bias on its output product (a float32 ``out_bias``) then travels as that pair's
    constant instead of being added in the product."""

    def __init__(self, *, first: PartSpec, second: PartSpec, hidden_size: int, eps: float = 0.0, names: tuple[str, str] = (),
                 scales: tuple[float, float] | None = None) -> None:
        if (scales is None) == (not names):
            raise ValueError("side by side, two mixers are combined either by norms (names) or by scales")
        self.members = (build_part("mixer", first), build_part("mixer", second))
        self.names, self.hidden_size, self.eps = tuple(names), hidden_size, float(eps)
        self.scales = tuple(float(s) for s in scales) if scales is not None else None
        self.constant: torch.Tensor | None = None
        self.graph_safe = all(m.graph_safe for m in self.members)
        # Members that say where their output goes write to buffers of their own; another member's output is copied.
        for member, name in zip(self.members, ("branch_first", "branch_second")):
            if hasattr(member, "out_name"):
                member.out_name = name
            if self.scales is not None and getattr(member, "has_out_bias", False):
                member.adds_out_bias = False
        self.weights: list[torch.Tensor] = []

    def cache_spec(self) -> CacheSpecs:
        return CacheSpecs(tuple(m.cache_spec() for m in self.members))

    def tensor_specs(self) -> list[TensorSpec]:
        specs = [spec for m in self.members for spec in m.tensor_specs()]
        return specs + [TensorSpec(name, (self.hidden_size,), init="one_plus_normal") for name in self.names]

    def load(self, tensors, dtype, device) -> None:
        for m in self.members:
            m.load(tensors, dtype, device)
        if self.scales is not None:
            biases = [s * m.out_bias for s, m in zip(self.scales, self.members) if getattr(m, "has_out_bias", False)]
            self.constant = sum(biases[1:], biases[0]).contiguous() if biases else None
        self.weights = [tensors[name].to(device=device, dtype=torch.float32).contiguous() for name in self.names]

    def weight_bytes(self) -> int:
        return sum(m.weight_bytes() for m in self.members)

    def forward(self, ctx: StepContext, cache: CacheView, h: torch.Tensor) -> ops.BranchPair | ops.ScaledPair:
        outs = []
        for index, member in enumerate(self.members):
            view = cache.members[index] if cache is not None else None
            out = member.forward(ctx, view, h)
            if not hasattr(member, "out_name"):
                keep = ctx.buffer(("branch_first", "branch_second")[index], tuple(out.shape), out.dtype)
                keep.copy_(out)
                out = keep
            outs.append(out)
        if self.scales is not None:
            return ops.ScaledPair(outs[0], outs[1], *self.scales, constant=self.constant)
        return ops.BranchPair(outs[0], outs[1], self.weights[0], self.weights[1], self.eps)


register_part("mixer", "parallel_mixers", ParallelMixers)
