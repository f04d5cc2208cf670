"""A recurrent mixer: a matrix memory per head with an exponential input gate, a forget gate and a normaliser (xLSTM's mLSTM)."""

from __future__ import annotations

import torch

from ..weights.loader import TensorSpec
from . import ops
from .base import Part, StateSpec, register_part
from .context import CacheView, StepContext


class MatrixMemory(Part):
    """``q = W_q h * dim^(-1/2)``, ``k = W_k h`` (``heads x dim``), ``v = W_v h`` (``heads x vdim``). Per head the log gates are
    ``i = c tanh((W_i h + b_i) / c)`` and ``f = logsigmoid(c tanh((W_f h + b_f) / c))`` with ``c = gate_cap``, and a state of
    ``S [dim, vdim]``, ``n [dim]`` and a running maximum ``m`` (32-bit, all zero at a request's start) is carried from token to
    token: ``m' = max(f + m, i)``, ``S <- exp(f + m - m') S + exp(i - m') k v^T``, ``n`` likewise with ``k`` alone, ``o = S^T q /
    (max(|n . q|, exp(-m')) + 1e-6)``. Each head's ``o`` is divided by its root mean square, times ``norm`` (all heads' size),
    times ``sigmoid(W_g h)``; then ``W_o``.

    The six projections are one matrix ``[q | k | v | g | i | f]`` whose product has a 32-bit result: it is what the recurrence
    reads, without a pass that widens it. Tensor names: ``prefix + q | k | v | g | i | i.b | f | f.b | norm | o``."""

    def __init__(self, *, prefix: str, hidden_size: int, heads: int, dim: int, vdim: int, gate_cap: float, eps: float, out_name: str = "branch") -> None:
        self.prefix, self.hidden_size, self.out_name = prefix, hidden_size, out_name
        self.heads, self.dim, self.vdim, self.gate_cap, self.eps = int(heads), int(dim), int(vdim), float(gate_cap), float(eps)
        qk, vw = self.heads * self.dim, self.heads * self.vdim
        self.widths = {"q": qk, "k": qk, "v": vw, "g": vw, "i": self.heads, "f": self.heads}
        starts = [0]
        for width in self.widths.values():
            starts.append(starts[-1] + width)
        self.columns = tuple(starts[:-1])
        self.w_in = self.w_o = self.i_bias = self.f_bias = self.norm_weight = None

    def cache_spec(self) -> StateSpec:
        f32 = torch.float32
        return StateSpec(((self.heads, self.dim, self.vdim), (self.heads, self.dim), (self.heads,)), (f32, f32, f32))

    def tensor_specs(self) -> list[TensorSpec]:
        p, d = self.prefix, self.hidden_size
        specs = [TensorSpec(p + name, (width, d)) for name, width in self.widths.items()]
        return specs + [
            TensorSpec(p + "i.b", (self.heads,)), TensorSpec(p + "f.b", (self.heads,)),
            TensorSpec(p + "norm", (self.heads * self.vdim,), init="one_plus_normal"), TensorSpec(p + "o", (d, self.heads * self.vdim)),
        ]

    def load(self, tensors, dtype, device) -> None:
        p, f32 = self.prefix, torch.float32

        def get(name: str, to=dtype) -> torch.Tensor:
            return tensors[p + name].to(device=device, dtype=to).contiguous()

        self.w_in = torch.cat([get(name) for name in self.widths])
        if self.w_in.shape[0] % 8:  # whole 16-byte steps from row to row of the product (the added columns are read by nobody)
            self.w_in = torch.cat([self.w_in, self.w_in.new_zeros((-self.w_in.shape[0] % 8, self.hidden_size))])
        self.w_in = self.w_in.contiguous()
        self.w_o = get("o")
        self.i_bias, self.f_bias, self.norm_weight = get("i.b", f32), get("f.b", f32), get("norm", f32)

    def weight_bytes(self) -> int:
        return (self.w_in.numel() + self.w_o.numel()) * self.w_o.element_size()

    def forward(self, ctx: StepContext, cache: CacheView, h: torch.Tensor) -> torch.Tensor:
        t = ctx.num_tokens
        proj = ops.linear(ctx, h, self.w_in, ctx.buffer("mlstm_proj", (t, self.w_in.shape[0]), torch.float32))
        y = ops.mlstm(ctx, proj, self.columns, self.i_bias, self.f_bias, self.gate_cap, cache.state, self.heads, self.dim, self.vdim,
                      self.norm_weight, self.eps, ctx.buffer("mlstm_out", (t, self.heads * self.vdim)))
        return ops.linear(ctx, y, self.w_o, ctx.buffer(self.out_name, (t, self.hidden_size)))


register_part("mixer", "matrix_memory", MatrixMemory)
