"""Norms over the last dimension, with the residual add fused in: root mean square, layer norm, dynamic
tanh, none at all; and what may be done to a sublayer's output on its way into the residual stream or streams.

Formula (engine/model/layers.py:41-43): ``normed = x * rsqrt(mean(x^2) + eps)`` in 32-bit,
then ``weight * normed``.  The residual stream is kept in 32-bit here, so square, mean,
rsqrt and both products are 32-bit and the result is rounded once to the compute dtype.
"""

from __future__ import annotations

from .base import BuildEnv, Norm, WeightDecl
from .registry import register_part


@register_part("norm", "rms")
class RMSNorm(Norm):
    """``offset``: what is added to the stored weight (1 for weights stored around zero, so that the
    factor is ``1 + w``; 0 for weights stored around one)."""

    def __init__(self, weight: str, size: int, eps: float, dtype, offset: float = 0.0) -> None:
        self.weight_name, self.size, self.eps, self.dtype = weight, int(size), float(eps), dtype
        self.offset = float(offset)
        self.weight = None

    @classmethod
    def from_spec(cls, params: dict, env: BuildEnv, **_):
        return cls(params["weight"], params.get("size", env.hidden_size), params["eps"],
                   env.torch_dtype, params.get("offset", 0.0))

    def weights(self) -> dict[str, WeightDecl]:
        init = "normal" if self.offset else "ones_plus_normal"
        return {self.weight_name: WeightDecl((self.size,), "vector", init)}

    def bind(self, tensors, env: BuildEnv) -> None:
        self.weight = (tensors[self.weight_name].float() + self.offset).contiguous()

    def add_norm(self, h, delta, ctx, rows=None, tag: str = "norm", delta_scale: float = 1.0,
                 delta_post: "PostNorm | None" = None):
        n = h.shape[0] if rows is None else rows.shape[0]
        out = ctx.ws.buffer(tag, n, self.size, self.dtype)
        if delta_post is not None:
            # something is done to the delta before it is added (it is normalised and takes its bias,
            # or passes a learned gate): one kernel for that, the add and this norm
            if delta_scale != 1.0:
                raise ValueError("a delta that is treated before the add has no residual multiplier")
            delta_post.add_norm(h, delta, ctx, self.weight, self.eps, out, rows)
        elif delta_scale == 1.0:
            ctx.ops.rmsnorm(h, delta, self.weight, self.eps, out, rows)
        else:
            ctx.ops.rmsnorm(h, delta, self.weight, self.eps, out, rows, delta_scale=float(delta_scale))
        return out


@register_part("norm", "identity")
class NoNorm(Norm):
    """No norm where an arrangement has one: a sublayer that reads the residual stream as it is.  The stream is
    brought up to date and handed on in the compute dtype (the 32-bit stream itself where that is 32-bit
    and nothing selects rows)."""

    def __init__(self, size: int, dtype) -> None:
        self.size, self.dtype = int(size), dtype

    @classmethod
    def from_spec(cls, params: dict, env: BuildEnv, **_):
        return cls(params.get("size", env.hidden_size), env.torch_dtype)

    def add_norm(self, h, delta, ctx, rows=None, tag: str = "norm", delta_scale: float = 1.0, delta_post=None):
        import torch

        if delta_scale != 1.0:
            raise ValueError("a stream that is handed on as it is takes a delta without a residual multiplier")
        out = None
        if rows is not None or self.dtype != torch.float32:
            out = ctx.ws.buffer(tag, h.shape[0] if rows is None else rows.shape[0], self.size, self.dtype)
        if delta_post is not None:
            delta_post.add_norm(h, delta, ctx, None, 0.0, out, rows)
        elif delta is not None or out is not None:
            ctx.ops.sandwich_norm(h, delta, None, None, 0.0, None, 0.0, out, rows)
        return h if out is None else out


class PostNorm:
    """What a block wants done to a sublayer's output before it enters the residual stream: a bias
    (or None), then an RMS norm.  Carried beside the pending delta to whoever adds it."""

    def __init__(self, norm: RMSNorm, bias=None) -> None:
        self.norm, self.bias = norm, bias

    def add_norm(self, h, delta, ctx, weight, eps, out, rows) -> None:
        """``h += norm(delta + bias)`` (not with ``rows``); ``out = rms(h) * weight`` (no weight: ``h`` as it is)."""
        ctx.ops.sandwich_norm(h, delta, self.bias, self.norm.weight, self.norm.eps, weight, eps, out, rows)

    def settle(self, h, delta, ctx) -> None:
        """``h += norm(delta + bias)`` with no normalised output."""
        ctx.ops.sandwich_norm(h, delta, self.bias, self.norm.weight, self.norm.eps, None, 0.0, None)


class AddedTerms:
    """What enters the residual stream together with a pending delta, in the same add: the output of
    a second sublayer that read the same input (``second``: whole, or in parts like a delta), a bias
    row of the sublayer that left the delta (``bias``), and a second stream of the rows' shape
    (``rows_like_stream``: the embedding's output that a looped model adds again before a pass).
    ``h += delta + second + bias + rows_like_stream`` and the next norm are one kernel."""

    def __init__(self, bias=None, second=None, rows_like_stream=None) -> None:
        self.bias, self.second, self.rows_like_stream = bias, second, rows_like_stream

    def with_stream_rows(self, x0) -> "AddedTerms":
        if self.rows_like_stream is not None:
            raise ValueError("one second stream per add")
        return AddedTerms(self.bias, self.second, x0)

    def add_norm(self, h, delta, ctx, weight, eps, out, rows) -> None:
        ctx.ops.sandwich_norm(h, delta, self.bias, None, 0.0, weight, eps, out, rows, second=self.second,
                              extra=self.rows_like_stream)

    def settle(self, h, delta, ctx) -> None:
        ctx.ops.sandwich_norm(h, delta, self.bias, None, 0.0, None, 0.0, None, second=self.second,
                              extra=self.rows_like_stream)


class ResidualGate:
    """A sublayer's output enters the residual stream through a gate: ``h += sigmoid(gate_pre + bias) *
    delta`` element by element.  ``gate_pre`` is the 32-bit pre-activation ``[N, hidden]`` of this
    step; carried beside the pending delta to whoever adds it, like :class:`PostNorm`."""

    def __init__(self, gate_pre, bias=None) -> None:
        self.gate_pre, self.bias = gate_pre, bias

    def add_norm(self, h, delta, ctx, weight, eps, out, rows) -> None:
        ctx.ops.gated_add_norm(h, delta, self.gate_pre, self.bias, weight, eps, out, rows)

    def settle(self, h, delta, ctx) -> None:
        ctx.ops.gated_add_norm(h, delta, self.gate_pre, self.bias, None, 0.0, None)


@register_part("norm", "layer")
class LayerNorm(Norm):
    """Layer norm over the last dimension with a weight and no bias, the residual add fused in:
    ``(x - mean(x)) / sqrt(mean((x - mean(x))^2) + eps) * weight``, all in 32-bit on the 32-bit
    residual stream; the result is rounded once to the compute dtype."""

    def __init__(self, weight: str, size: int, eps: float, dtype) -> None:
        self.weight_name, self.size, self.eps, self.dtype = weight, int(size), float(eps), dtype
        self.weight = None

    @classmethod
    def from_spec(cls, params: dict, env: BuildEnv, **_):
        return cls(params["weight"], params.get("size", env.hidden_size), params["eps"],
                   env.torch_dtype)

    def weights(self) -> dict[str, WeightDecl]:
        return {self.weight_name: WeightDecl((self.size,), "vector", "ones_plus_normal")}

    def bind(self, tensors, env: BuildEnv) -> None:
        self.weight = tensors[self.weight_name].float().contiguous()

    def add_norm(self, h, delta, ctx, rows=None, tag: str = "norm", delta_scale: float = 1.0):
        n = h.shape[0] if rows is None else rows.shape[0]
        out = ctx.ws.buffer(tag, n, self.size, self.dtype)
        ctx.ops.layernorm(h, delta, self.weight, self.eps, out, rows, delta_scale=float(delta_scale))
        return out


class StreamMix:
    """Several residual streams side by side in a row of ``h`` (``[N, streams * width]``).  What a sublayer
    returned enters all of them at once: ``x_t <- sum_s mix[s, t] x_s + out[t] * delta`` (``mix[from, to]``), and
    what the next sublayer reads is ``sum_t read[t] x_t`` (no ``read``: the streams' plain sum, as at a
    model's end).  Carried beside the pending delta to whoever adds it, like :class:`PostNorm`; the
    mixing, the reading and the next norm are one kernel.  Without coefficients nothing is mixed."""

    def __init__(self, streams: int, mix=None, out=None, read=None) -> None:
        self.streams, self.mix, self.out, self.read = int(streams), mix, out, read

    def reading(self, read) -> "StreamMix":
        return StreamMix(self.streams, self.mix, self.out, read)

    def add_norm(self, h, delta, ctx, weight, eps, out, rows, bias=None, alpha=None) -> None:
        ctx.ops.stream_mix_norm(h, self.streams, delta, self.mix, self.out, self.read, weight, bias, alpha, eps, out,
                                rows)

    def settle(self, h, delta, ctx) -> None:
        ctx.ops.stream_mix_norm(h, self.streams, delta, self.mix, self.out, None, None, None, None, 0.0, None)


@register_part("norm", "dynamic_tanh")
class DynamicTanh(Norm):
    """``tanh(alpha * x) * weight + bias`` entry by entry: no mean, no variance.  ``alpha`` is one stored number.
    32-bit throughout; the result is rounded once to the compute dtype."""

    def __init__(self, weight: str, bias: str, alpha: str, size: int, dtype) -> None:
        self.weight_name, self.bias_name, self.alpha_name = weight, bias, alpha
        self.size, self.dtype = int(size), dtype
        self.weight = self.bias = self.alpha = None

    @classmethod
    def from_spec(cls, params: dict, env: BuildEnv, **_):
        return cls(params["weight"], params["bias"], params["alpha"], params.get("size", env.hidden_size),
                   env.torch_dtype)

    def weights(self) -> dict[str, WeightDecl]:
        return {self.weight_name: WeightDecl((self.size,), "vector", "ones_plus_normal"),
                self.bias_name: WeightDecl((self.size,), "vector"),
                self.alpha_name: WeightDecl((), "vector", "ones_plus_normal")}

    def bind(self, tensors, env: BuildEnv) -> None:
        self.weight = tensors[self.weight_name].float().contiguous()
        self.bias = tensors[self.bias_name].float().contiguous()
        self.alpha = tensors[self.alpha_name].float().reshape(1).contiguous()

    def add_norm(self, h, delta, ctx, rows=None, tag: str = "norm", delta_scale: float = 1.0, delta_post=None):
        if delta_scale != 1.0:
            raise ValueError("the tanh norm's kernel adds a delta without a residual multiplier")
        post = delta_post if delta_post is not None else StreamMix(1)
        if not isinstance(post, StreamMix):
            raise ValueError(f"the tanh norm's kernel cannot treat a delta by {type(post).__name__}")
        n = h.shape[0] if rows is None else rows.shape[0]
        out = ctx.ws.buffer(tag, n, self.size, self.dtype)
        post.add_norm(h, delta, ctx, self.weight, 0.0, out, rows, bias=self.bias, alpha=self.alpha)
        return out
