"""Mixers made of other mixers.

``parallel_sum``: several mixers side by side that read the same input; the result is the sum of
their outputs, each times its own factor.  Every branch keeps its own cache (a tuple of requests,
a tuple of bindings).  Branches that can all leave their first and last product to the sum
(``leaves_products``) share one product each: the stacked rows of their input matrices, and their output matrices side
by side over their results side by side, whose sum is the sum of the branches; each takes its factor into its
result before that is rounded.
"""

from __future__ import annotations

from ..config.spec import PartSpec
from .base import BuildEnv, Mixer
from .registry import build_part, register_part


def _part_spec(raw) -> PartSpec:
    return raw if isinstance(raw, PartSpec) else PartSpec(raw["kind"], dict(raw.get("params", {})))


@register_part("mixer", "parallel_sum")
class ParallelSum(Mixer):
    def __init__(self, branches: list[Mixer], scales: list[float], hidden_size: int) -> None:
        if len(branches) < 2 or len(branches) != len(scales):
            raise ValueError("a sum of mixers needs at least two branches, each with its factor")
        self.branches, self.scales, self.hidden_size = branches, [float(s) for s in scales], hidden_size
        self.joined = all(b.leaves_products for b in branches)
        for b, scale in zip(branches, self.scales):
            if self.joined:
                b.products_elsewhere, b.output_scale = True, scale
            else:
                b.allow_split = False  # the sum below takes whole outputs
        self.w_in = self.w_o = None

    @classmethod
    def from_spec(cls, params: dict, env: BuildEnv, **_):
        branches = [build_part("mixer", _part_spec(b["mixer"]), env) for b in params["branches"]]
        return cls(branches, [b["scale"] for b in params["branches"]], params.get("hidden_size", env.hidden_size))

    @property
    def captures(self) -> bool:
        return all(getattr(b, "captures", True) for b in self.branches)

    def parts(self):
        return list(self.branches)

    def cache_request(self):
        return tuple(b.cache_request() for b in self.branches)

    def weights(self):
        """(the branches' own: the joined products are made of them)"""
        return {name: decl for b in self.branches for name, decl in b.weights().items()} if self.joined else {}

    def bind(self, tensors, env: BuildEnv) -> None:
        import torch

        if not self.joined:
            return
        rows, self.columns, at = [], [], 0
        for b in self.branches:
            own = b.input_rows(tensors)
            count = sum(r.shape[0] for r in own)
            self.columns.append((at, at + count))
            # (zero rows up to a multiple of four: every branch's columns start on 16 bytes)
            rows += own + ([own[0].new_zeros(-count % 4, own[0].shape[1])] if count % 4 else [])
            at += count + -count % 4
        self.w_in = torch.cat(rows).contiguous()
        self.w_o = torch.cat([b.output_matrix(tensors) for b in self.branches], dim=1).contiguous()
        self.dtype = self.w_o.dtype

    def _forward_joined(self, x, ctx, binding):
        import torch

        ops, ws = ctx.ops, ctx.ws
        proj = ops.linear(x, self.w_in, ws=ws, tag="parallel.in", out_dtype=torch.float32)
        out = ws.buffer("parallel.out", x.shape[0], self.w_o.shape[1], self.dtype)
        at = 0
        for b, bind, (first, end) in zip(self.branches, binding, self.columns):
            b.run(proj[:, first:end], ctx, bind, out[:, at: at + b.out_size])
            at += b.out_size
        return ops.linear(out, self.w_o, ws=ws, tag="parallel.delta", out_dtype=torch.float32, allow_split=True)

    def forward(self, x, ctx, binding):
        import torch

        if self.joined:
            return self._forward_joined(x, ctx, binding)
        outs = [b.forward(x, ctx, bind) for b, bind in zip(self.branches, binding)]
        total = ctx.ws.buffer("parallel.sum", x.shape[0], self.hidden_size, torch.float32)
        ctx.ops.weighted_sum(outs[0], self.scales[0], outs[1], self.scales[1], total)
        for o, s in zip(outs[2:], self.scales[2:]):
            ctx.ops.weighted_sum(total, 1.0, o, s, total)
        return total
