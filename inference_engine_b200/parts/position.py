"""Position encodings.

``learned``: a table of vectors added to the embedding.

``rotary``: rotation of query and key halves by position-dependent angles, with the
optional Llama 3 or YaRN frequency scaling.  Frequencies follow engine/model/layers.py:55-73 and
angles engine/model/layers.py:75-79: everything is 32-bit; the table holds cos and sin of
``position * inv_freq`` for every position the engine can feed, so the kernels read the
same values a whole-sequence computation would.
"""

from __future__ import annotations

import math

from .base import BuildEnv, PositionEncoding
from .registry import register_part


def rotary_inv_freq(rotary_dim: int, theta: float, scaling: dict | None):
    """``inv_freq[j] = theta^(-2j/dim)``; with ``scaling`` (llama3) long wavelengths are
    divided by ``factor``, short ones kept, the band between interpolated."""
    import torch

    inv_freq = 1.0 / (theta ** (torch.arange(0, rotary_dim, 2, dtype=torch.int64).float() / rotary_dim))
    if not scaling:
        return inv_freq
    factor = float(scaling["factor"])
    low_f, high_f = float(scaling["low_freq_factor"]), float(scaling["high_freq_factor"])
    orig = float(scaling["original_max_position_embeddings"])
    low_wavelen, high_wavelen = orig / low_f, orig / high_f
    wavelen = 2 * math.pi / inv_freq
    scaled = torch.where(wavelen > low_wavelen, inv_freq / factor, inv_freq)
    smooth = (orig / wavelen - low_f) / (high_f - low_f)
    smoothed = (1 - smooth) * scaled / factor + smooth * scaled
    medium = ~(wavelen < high_wavelen) & ~(wavelen > low_wavelen)
    return torch.where(medium, smoothed, scaled)


def exact_frequencies(rotary_dim: int, theta: float, scaling: dict | None):
    """``(frequencies, amplitude)`` worked out in 64-bit: ``theta^(-2j/dim)``, then the scaling.  ``kind`` ``llama3``
    (the default): as in :func:`rotary_inv_freq`.  ``kind`` ``yarn`` (``factor``, ``original``, ``fast``, ``slow``): the pair
    that turns ``t`` times over the original length is number ``dim * ln(original / (2 pi t)) / (2 ln theta)``; pairs up
    to the one at ``fast`` turns keep their frequency, pairs from the one at ``slow`` turns on have it divided by
    ``factor``, a straight line between; cos and sin are multiplied by the amplitude ``0.1 ln(factor) + 1``."""
    import torch

    j = torch.arange(0, rotary_dim, 2, dtype=torch.float64)
    freq = torch.exp(-(j / rotary_dim) * math.log(theta))
    if not scaling:
        return freq, 1.0
    factor = float(scaling["factor"])
    kind = scaling.get("kind", "llama3")
    if kind == "yarn":
        def pair_at(turns: float) -> float:
            return rotary_dim * math.log(float(scaling["original"]) / (2 * math.pi * turns)) / (2 * math.log(theta))

        low = max(math.floor(pair_at(float(scaling["fast"]))), 0)
        high = min(math.ceil(pair_at(float(scaling["slow"]))), rotary_dim - 1)
        ramp = ((torch.arange(rotary_dim // 2, dtype=torch.float64) - low) / max(high - low, 0.001)).clamp(0.0, 1.0)
        return freq / factor * ramp + freq * (1.0 - ramp), 0.1 * math.log(factor) + 1.0
    if kind != "llama3":
        raise ValueError(f"no rotary frequency scaling of kind {kind!r}")
    low_f, high_f = float(scaling["low_freq_factor"]), float(scaling["high_freq_factor"])
    original = float(scaling["original_max_position_embeddings"])
    wavelength = 2 * math.pi / freq
    blend = (original / wavelength - low_f) / (high_f - low_f) if high_f != low_f else torch.zeros_like(freq)
    between = (1 - blend) * freq / factor + blend * freq
    scaled = torch.where(wavelength > original / low_f, freq / factor, between)
    return torch.where(wavelength < original / high_f, freq, scaled), 1.0


@register_part("position", "rotary")
class RotaryEncoding(PositionEncoding):
    LAYOUTS = ("halves", "interleaved")

    def __init__(self, rotary_dim: int, theta: float, scaling: dict | None,
                 max_positions: int, layout: str = "halves", angles: str = "float32") -> None:
        if rotary_dim % 2:
            raise ValueError(f"rotary_dim ({rotary_dim}) must be even")
        if layout not in self.LAYOUTS:
            raise ValueError(f"rotary layout {layout!r} is not one of {self.LAYOUTS}")
        # which entries form the pair rotated by angle j: "halves": j and j + rotary_dim/2 (Llama's);
        # "interleaved": 2j and 2j + 1.  The table of angles is the same; the consumer reads `layout`.
        self.layout = layout
        if angles not in ("float32", "float64"):
            raise ValueError(f"rotary angles are computed in float32 or float64, not {angles!r}")
        # "float64": frequencies (scaled or not), angles and their cos and sin are worked out in
        # 64-bit and rounded once to the 32-bit table
        self.angles = angles
        if angles == "float32" and scaling and scaling.get("kind", "llama3") != "llama3":
            raise ValueError("32-bit rotary angles know the llama3 frequency scaling only")
        self.rotary_dim, self.theta, self.scaling = int(rotary_dim), float(theta), scaling
        self.max_positions = int(max_positions)
        self.inv_freq = self._table = None

    @classmethod
    def from_spec(cls, params: dict, env: BuildEnv, **_):
        return cls(params["rotary_dim"], params["theta"], params.get("scaling"),
                   env.max_positions, params.get("layout", "halves"), params.get("angles", "float32"))

    def bind(self, tensors, env: BuildEnv) -> None:
        """No stored tensor (the reference keeps ``inv_freq`` out of checkpoints,
        engine/model/layers.py:52-53): the table is computed here, on the device."""
        import torch

        if self.angles == "float64":
            inv_freq, amplitude = exact_frequencies(self.rotary_dim, self.theta, self.scaling)
            freqs = torch.arange(self.max_positions, dtype=torch.float64)[:, None] * inv_freq[None, :]
            self.inv_freq = inv_freq.float().to(env.device)
            self._table = (torch.stack((freqs.cos(), freqs.sin()), dim=1) * amplitude).float().contiguous().to(env.device)
            return
        self.inv_freq = rotary_inv_freq(self.rotary_dim, self.theta, self.scaling).to(env.device)
        pos = torch.arange(self.max_positions, device=env.device).float()
        freqs = pos[:, None] * self.inv_freq.float()[None, :]
        self._table = torch.stack((freqs.cos(), freqs.sin()), dim=1).contiguous()  # [P, 2, half]

    def rotary_table(self):
        return self._table


@register_part("position", "learned")
class LearnedPositions(PositionEncoding):
    """A learned vector per position, added (unscaled) to the embedded tokens in the 32-bit
    residual stream.  The table's rows bound the positions a request can reach."""

    def __init__(self, weight: str, positions: int, hidden_size: int) -> None:
        self.weight_name, self.positions, self.hidden_size = weight, int(positions), int(hidden_size)
        self.table = None

    @classmethod
    def from_spec(cls, params: dict, env: BuildEnv, **_):
        return cls(params["weight"], params["positions"], params.get("hidden_size", env.hidden_size))

    def weights(self):
        from .base import WeightDecl

        return {self.weight_name: WeightDecl((self.positions, self.hidden_size), "table")}

    def bind(self, tensors, env: BuildEnv) -> None:
        self.table = tensors[self.weight_name].to(env.torch_dtype).contiguous()

    def apply_to_embedding(self, h, ctx) -> None:
        ctx.ops.add_position_rows(h, self.table, ctx.positions)


@register_part("position", "none")
class NoPositionEncoding(PositionEncoding):
    """Leaves queries, keys and embeddings as they are."""

    @classmethod
    def from_spec(cls, params: dict, env: BuildEnv, **_):
        return cls()
