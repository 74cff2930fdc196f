"""Kolisun: a decoder-only model that normalises what its sublayers return and nothing they read, with
latent attention layers and layers that run a windowed attention beside a state-space recurrence.

Configuration keys: ``vocab``, ``width``, ``norm.eps`` and ``layers``; each layer gives its ``type``
(``latent_attention`` or ``parallel``), the mixer's sizes and constants under ``mixer`` and its feed-forward under
``mlp`` (``null``: none; ``kind`` ``dense``: gated by silu, ``ff`` units).  ``latent_attention``: ``heads``, ``dim``,
``rot_dim``, ``vdim``, ``kv_rank``, ``q_rank``, ``scale``, ``rot.dims`` / ``rot.base`` and, optionally, ``rot.scaling``
(YaRN: ``factor``, ``original``, ``fast``, ``slow``).  ``parallel``: ``left_scale``, ``right_scale``; ``left``: ``heads``,
``kv_heads``, ``dim``, ``vdim``, ``scale``, ``mask.size``, ``rot.dims`` / ``rot.base`` and, optionally, ``rot.scaling`` (Llama 3.1:
``factor``, ``low``, ``high``, ``original``); ``right``: ``heads``, ``groups``, ``state``, ``vdim``, ``conv`` (taps),
``norm_groups``.  What is absent does not exist; ``max_positions`` is optional.
Tensors: ``embed``, ``l<i>.norm1`` / ``norm2``, ``l<i>.mix.*`` (``dq``, ``dq.norm``, ``uq``, ``dkv``, ``dkv.norm``, ``uk``, ``uv``,
``sink``, ``o``; or ``left.q`` / ``k`` / ``v`` with ``.b`` and ``.norm``, ``left.o``, ``right.in``, ``right.conv`` and ``.b``,
``right.dt_bias``, ``right.A_log``, ``right.D``, ``right.norm``, ``right.o``), ``l<i>.mlp.gate`` / ``up`` / ``down``,
``final.norm``, ``head``.

The model: ``x <- x + norm1(mixer(x))``, ``x <- x + norm2(ff(x))`` with RMS norms; the logits read the stream
through the final norm.  ``latent_attention``: queries through a latent of their own, keys and values from a cached
latent and a shared rotated part (halves), a sink per head.  ``parallel``: grouped-query attention over a
window with biases, norms over all query and all key columns and rotated interleaved pairs, beside a state-space
recurrence with a short convolution and a gated norm in parts; their outputs are added, each times its factor.
No torch import here.
"""

from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Any

from ..config.model_config import ConfigError, Footprint, id_tuple
from ..config.registry import register_architecture
from ..config.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

NAME = "Kolisun"
LAYER_TYPES = ("latent_attention", "parallel")
NO_POSITION_LIMIT = 1 << 30  # rotary tables are as long as the engine's longest request


def _need(raw, key: str, kind, where: str):
    if not isinstance(raw, dict) or key not in raw or raw[key] is None:
        raise ConfigError(f"config.json: {where} is missing the key {key!r}")
    try:
        return kind(raw[key])
    except (TypeError, ValueError) as exc:
        raise ConfigError(f"config.json: {where}.{key} = {raw[key]!r} is not a {kind.__name__}") from exc


def _positive(value, what: str):
    if not value > 0 or not math.isfinite(value):
        raise ConfigError(f"config.json: {what} must be a positive number")
    return value


def _sizes(raw, keys, where: str) -> dict:
    out = {k: _need(raw, k, int, where) for k in keys}
    for k, v in out.items():
        if v < 1:
            raise ConfigError(f"config.json: {where}.{k} must be at least 1")
    return out


def _parse_rotation(raw, widest: int, scaling_keys: tuple[str, ...], where: str) -> dict | None:
    """``{"dims", "base", "scaling"}`` or None if nothing is rotated."""
    dims = int((raw or {}).get("dims") or 0)
    if dims == 0:
        return None
    if dims < 0 or dims % 2 or dims > widest:
        raise ConfigError(f"config.json: {where}.dims must be even and at most {widest}")
    base = _positive(_need(raw, "base", float, where), where + ".base")
    scaling = raw.get("scaling")
    if scaling is not None:
        scaling = {k: _positive(_need(scaling, k, float, where + ".scaling"), f"{where}.scaling.{k}") for k in scaling_keys}
        if "fast" in scaling and base == 1.0:
            raise ConfigError(f"config.json: {where}.base = 1 has no pairs for YaRN to tell apart")
    return {"dims": dims, "base": base, "scaling": scaling}


def _parse_latent(raw: dict, where: str) -> dict:
    out = _sizes(raw, ("heads", "dim", "vdim", "kv_rank", "q_rank"), where)
    out["rot_dim"] = _need(raw, "rot_dim", int, where)
    if out["rot_dim"] < 0:
        raise ConfigError(f"config.json: {where}.rot_dim cannot be negative")
    out["scale"] = _need(raw, "scale", float, where)
    out["rot"] = _parse_rotation(raw.get("rot"), out["rot_dim"], ("factor", "original", "fast", "slow"), where + ".rot")
    return out


def _parse_parallel(raw: dict, where: str) -> dict:
    left_raw, lw = raw.get("left"), where + ".left"
    left = _sizes(left_raw, ("heads", "dim", "vdim"), lw)
    # (a mixer that does not share keys and values among heads need not say so)
    left["kv_heads"] = _need(left_raw, "kv_heads", int, lw) if left_raw.get("kv_heads") is not None else left["heads"]
    if left["kv_heads"] < 1 or left["heads"] % left["kv_heads"]:
        raise ConfigError(f"config.json: {lw}.heads is not a multiple of kv_heads")
    left["scale"] = _need(left_raw, "scale", float, lw)
    left["rot"] = _parse_rotation(left_raw.get("rot"), left["dim"], ("factor", "low", "high", "original"), lw + ".rot")
    mask = left_raw.get("mask")
    left["window"] = _need(mask, "size", int, lw + ".mask") if mask is not None else None
    if left["window"] is not None and left["window"] < 1:
        raise ConfigError(f"config.json: {lw}.mask.size must be at least 1")
    right_raw, rw = raw.get("right"), where + ".right"
    right = _sizes(right_raw, ("heads", "vdim", "state", "conv"), rw)
    for key in ("groups", "norm_groups"):
        right[key] = _need(right_raw, key, int, rw) if right_raw.get(key) is not None else 1
    if right["groups"] < 1 or right["heads"] % right["groups"]:
        raise ConfigError(f"config.json: {rw}.heads is not a multiple of groups")
    if right["norm_groups"] < 1 or (right["heads"] * right["vdim"]) % right["norm_groups"]:
        raise ConfigError(f"config.json: {rw}.norm_groups does not divide heads * vdim")
    return {"left": left, "right": right, "left_scale": _need(raw, "left_scale", float, where),
            "right_scale": _need(raw, "right_scale", float, where)}


def _parse_mlp(raw, where: str):
    if raw is None:
        return None
    kind = _need(raw, "kind", str, where)
    if kind != "dense":
        raise ConfigError(f"config.json: {where}.kind = {kind!r} is not 'dense'")
    return _sizes(raw, ("ff",), where)


@dataclass(frozen=True)
class KolisunLayer:
    type: str
    mixer: dict
    mlp: dict | None


@dataclass(frozen=True)
class KolisunConfig:
    architecture: str
    vocab_size: int
    hidden_size: int
    max_position_embeddings: int
    norm_eps: float
    layers: tuple[KolisunLayer, ...]
    eos_token_ids: tuple[int, ...] = ()
    torch_dtype: str = "bfloat16"

    @classmethod
    def from_dict(cls, raw: dict[str, Any]) -> "KolisunConfig":
        listed = raw.get("layers")
        if not isinstance(listed, list) or not listed:
            raise ConfigError("config.json: 'layers' must list at least one layer")
        layers = []
        for i, entry in enumerate(listed):
            where = f"layers[{i}]"
            kind = _need(entry, "type", str, where)
            if kind not in LAYER_TYPES:
                raise ConfigError(f"config.json: {where}.type = {kind!r} is not one of {LAYER_TYPES}")
            parse = _parse_latent if kind == "latent_attention" else _parse_parallel
            layers.append(KolisunLayer(kind, parse(entry.get("mixer") or {}, where + ".mixer"),
                                       _parse_mlp(entry.get("mlp"), where + ".mlp")))
        cfg = cls(
            architecture=str(raw.get("architecture", NAME)),
            vocab_size=_need(raw, "vocab", int, "the model"),
            hidden_size=_need(raw, "width", int, "the model"),
            max_position_embeddings=int(raw.get("max_positions") or NO_POSITION_LIMIT),
            norm_eps=_positive(_need(raw.get("norm") or {}, "eps", float, "norm"), "norm.eps"),
            layers=tuple(layers),
            eos_token_ids=id_tuple(raw.get("eos_token_id")),
            torch_dtype=str(raw.get("torch_dtype", "bfloat16")),
        )
        for key in ("vocab_size", "hidden_size", "max_position_embeddings"):
            if getattr(cfg, key) < 1:
                raise ConfigError(f"config.json: {key} must be >= 1")
        return cfg


def _rotations(layer: KolisunLayer) -> tuple[str | None, PartSpec | None]:
    """(name, encoding) of the layer's rotation; layers with equal rotations share a table."""
    latent = layer.type == "latent_attention"
    rot = layer.mixer["rot"] if latent else layer.mixer["left"]["rot"]
    if rot is None:
        return None, None
    scaling = rot["scaling"]
    if scaling is not None and latent:
        scaling = {"kind": "yarn", **scaling}
    elif scaling is not None:
        scaling = {"kind": "llama3", "factor": scaling["factor"], "low_freq_factor": scaling["low"],
                   "high_freq_factor": scaling["high"], "original_max_position_embeddings": scaling["original"]}
    params = {"rotary_dim": rot["dims"], "theta": rot["base"], "scaling": scaling, "angles": "float64",
              "layout": "halves" if latent else "interleaved"}
    tail = "" if scaling is None else "_" + "_".join(str(v) for v in scaling.values())
    return f"rot_{params['layout']}_{rot['dims']}_{rot['base']!r}{tail}", PartSpec("rotary", params)


def _mixer_spec(cfg: KolisunConfig, i: int, layer: KolisunLayer) -> PartSpec:
    p, m = f"l{i}.mix", layer.mixer
    position = _rotations(layer)[0]
    if layer.type == "latent_attention":
        return PartSpec("latent_attention", {
            "names": {"dq": f"{p}.dq", "dq_norm": f"{p}.dq.norm", "uq": f"{p}.uq", "dkv": f"{p}.dkv",
                      "latent_norm": f"{p}.dkv.norm", "uk": f"{p}.uk", "uv": f"{p}.uv", "sink": f"{p}.sink", "o": f"{p}.o"},
            **{k: m[k] for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank", "scale")},
            "eps": cfg.norm_eps, "position": position})
    left, right, lp, rp = m["left"], m["right"], p + ".left", p + ".right"
    attention = PartSpec("sink_attention", {
        "names": {**{k: f"{lp}.{k}" for k in "qkvo"}, **{f"{k}_bias": f"{lp}.{k}.b" for k in "qkv"},
                  "q_norm": f"{lp}.q.norm", "k_norm": f"{lp}.k.norm"},
        **{k: left[k] for k in ("heads", "kv_heads", "dim", "vdim", "scale", "window")},
        "eps": cfg.norm_eps, "position": position})
    recurrence = PartSpec("state_space", {
        "names": {"in": f"{rp}.in", "conv": f"{rp}.conv", "conv_bias": f"{rp}.conv.b", "dt_bias": f"{rp}.dt_bias",
                  "A_log": f"{rp}.A_log", "skip": f"{rp}.D", "out_norm": f"{rp}.norm", "o": f"{rp}.o"},
        "heads": right["heads"], "vdim": right["vdim"], "state": right["state"], "groups": right["groups"],
        "taps": right["conv"], "norm_parts": right["norm_groups"], "eps": cfg.norm_eps})
    return PartSpec("parallel_sum", {"branches": [{"mixer": attention, "scale": m["left_scale"]},
                                                  {"mixer": recurrence, "scale": m["right_scale"]}]})


def kolisun_spec(cfg: KolisunConfig) -> ModelSpec:
    layers, positions = [], {}
    as_it_is = PartSpec("identity")
    for i, layer in enumerate(cfg.layers):
        name, encoding = _rotations(layer)
        if name is not None:
            positions.setdefault(name, encoding)
        norms = {"pre_mixer": as_it_is, "post_mixer": PartSpec("rms", {"weight": f"l{i}.norm1", "eps": cfg.norm_eps})}
        feed_forward, p = None, f"l{i}.mlp"
        if layer.mlp is not None:
            norms.update(pre_feed_forward=as_it_is,
                         post_feed_forward=PartSpec("rms", {"weight": f"l{i}.norm2", "eps": cfg.norm_eps}))
            feed_forward = PartSpec("swiglu", {"gate_proj": f"{p}.gate", "up_proj": f"{p}.up", "down_proj": f"{p}.down",
                                               "intermediate_size": layer.mlp["ff"]})
        layers.append(LayerSpec(prefix=f"l{i}", block=PartSpec("sandwich_residual"), mixer=_mixer_spec(cfg, i, layer),
                                feed_forward=feed_forward, norms=norms))
    return ModelSpec(
        architecture=cfg.architecture, vocab_size=cfg.vocab_size, hidden_size=cfg.hidden_size,
        max_position_embeddings=cfg.max_position_embeddings,
        embedding=PartSpec("token", {"weight": "embed", "vocab_size": cfg.vocab_size}),
        positions=positions, layers=tuple(layers), schedule=tuple(ScheduleEntry(i) for i in range(len(layers))),
        final_norm=PartSpec("rms", {"weight": "final.norm", "eps": cfg.norm_eps}),
        head=PartSpec("linear", {"weight": "head", "vocab_size": cfg.vocab_size}),
        eos_token_ids=cfg.eos_token_ids)


def kolisun_footprint(cfg: KolisunConfig) -> Footprint:
    h = cfg.hidden_size
    params = cfg.vocab_size * h * 2 + h
    per_token = per_request = 0
    for layer in cfg.layers:
        m = layer.mixer
        params += h
        if layer.type == "latent_attention":
            row, heads = m["kv_rank"] + m["rot_dim"], m["heads"]
            params += (m["q_rank"] + row) * h + m["q_rank"] + m["kv_rank"] + heads
            params += heads * (m["dim"] + m["rot_dim"]) * m["q_rank"] + heads * (m["dim"] + m["vdim"]) * m["kv_rank"]
            params += h * heads * m["vdim"]
            per_token += row
        else:
            left, right = m["left"], m["right"]
            q, k, v = left["heads"] * left["dim"], left["kv_heads"] * left["dim"], left["kv_heads"] * left["vdim"]
            params += (q + k + v) * (h + 1) + q + k + left["heads"] * left["vdim"] * h
            per_token += k + v
            inner = right["heads"] * right["vdim"]
            channels = inner + 2 * right["groups"] * right["state"]
            params += (inner + channels + right["heads"]) * h + channels * (right["conv"] + 1) + 3 * right["heads"]
            params += inner + inner * h
            per_request += inner * right["state"] + (right["conv"] - 1) * channels
        if layer.mlp is not None:
            params += h + 3 * layer.mlp["ff"] * h
    return Footprint(params, per_token, per_request)


def describe_kolisun(cfg: KolisunConfig) -> list[str]:
    kinds = [layer.type + ("" if layer.mlp is None else "+dense") for layer in cfg.layers]
    fp = kolisun_footprint(cfg)
    return [
        f"architecture        {cfg.architecture}",
        f"layers / width      {len(cfg.layers)} / {cfg.hidden_size}",
        f"layer kinds         {', '.join(kinds)}",
        f"parameters          {fp.parameters / 1e9:.3f} B",
        f"cache per token     {fp.cache_bytes_per_token(2)} B (bf16), state per request {fp.state_values_per_request * 4} B",
    ]


register_architecture(NAME, KolisunConfig, kolisun_spec, describe_kolisun, kolisun_footprint)
