"""Livitar: a decoder-only model with several residual streams (hyper-connections), norms without
statistics (dynamic tanh), retention layers and two kinds of softmax attention in which positions
enter as a bias by distance, and mixtures of experts beside a shared one.

Configuration keys: ``vocab``, ``width``, ``streams``, ``norm.eps`` and ``layers``; each layer gives its
``type`` (``retention``, ``attention`` or ``attention_2``), the mixer's sizes and constants under ``mixer``
(``retention``: ``heads``, ``dim``, ``vdim``, ``decay`` (one number per head), ``rot.dims`` / ``rot.base``;
the attentions: ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``; ``attention_2`` also ``bias_max`` and
``q_temp.coef`` / ``q_temp.every``) and its feed-forward under ``mlp`` (``null``: none; ``kind`` ``moe``:
``router.experts`` gated experts of ``expert.ff`` units, ``router.top`` per token, ``router.scale``, and a
shared expert of ``shared.ff`` units).  What is absent does not exist.  ``max_positions`` is optional, and
so is ``bias_buckets`` of an ``attention_2`` mixer, whose number the shape of ``mix.rel`` gives.
Tensors: ``embed``, ``l<i>.norm1`` / ``norm2`` with ``.b`` and ``.alpha``, ``l<i>.hc1.in`` / ``mix`` / ``out`` and
``hc2``, ``l<i>.mix.q`` / ``k`` / ``v`` / ``g`` / ``o`` (``attention``: also ``temp``, ``r1``, ``r2``;
``attention_2``: ``rel``), ``l<i>.mlp.router`` / ``e<j>.gate`` / ``up`` / ``down`` / ``shared.*``,
``final.norm``, ``head``.

The model: every stream starts as the token's embedding.  A sublayer reads ``u = sum_s in[s] x_s`` through
its norm ``tanh(alpha u) w + b``, and then ``x_t <- sum_s mix[s, t] x_s + out[t] y`` for all streams at once;
the logits read the streams' sum through the final norm.  ``retention``: a matrix state per head with a
constant decay, rotated queries and keys, unit-RMS read-out times a silu gate.  ``attention``: scores
times a temperature per head, less ``r1 ln(1 + r2 distance)``.  ``attention_2``: unit-RMS queries and keys,
queries warmed up by ``1 + coef ln(floor((p + 1) / every) + 1)``, a learned bias per bucket of distances.
Both attentions see every earlier position and multiply their heads by a sigmoid gate entry by entry.
The router weighs the ``top`` experts by their softmax scores over their sum, times a constant; the
shared expert's output is added.  No torch import here.
"""

from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Any

from ..config.model_config import ConfigError, Footprint, id_tuple
from ..config.registry import register_architecture
from ..config.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry
from .rugedra import read_tensor_shapes

NAME = "Livitar"
LAYER_TYPES = ("retention", "attention", "attention_2")
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


def _parse_retention(raw: dict, out: dict, where: str) -> None:
    try:
        out["decay"] = tuple(float(d) for d in raw["decay"])
    except (KeyError, TypeError, ValueError) as exc:
        raise ConfigError(f"config.json: {where}.decay must list a number per head") from exc
    if len(out["decay"]) != out["heads"]:
        raise ConfigError(f"config.json: {where}.decay lists {len(out['decay'])} numbers for {out['heads']} heads")
    rot = raw.get("rot") or {}
    out["rot_dims"] = int(rot.get("dims") or 0)
    if out["rot_dims"] < 0 or out["rot_dims"] % 2 or out["rot_dims"] > out["dim"]:
        raise ConfigError(f"config.json: {where}.rot.dims must be even and at most dim")
    out["rot_base"] = _positive(_need(rot, "base", float, where + ".rot"), where + ".rot.base") if out["rot_dims"] else 1.0


def _parse_attention(kind: str, raw: dict, out: dict, where: str) -> None:
    # (a mixer that does not share keys and values among heads need not say so)
    out["kv_heads"] = _need(raw, "kv_heads", int, where) if raw.get("kv_heads") is not None else out["heads"]
    if out["kv_heads"] < 1 or out["heads"] % out["kv_heads"]:
        raise ConfigError(f"config.json: {where}.heads is not a multiple of kv_heads")
    out["scale"] = _need(raw, "scale", float, where)
    if kind == "attention":
        return
    out["bias_max"] = _positive(_need(raw, "bias_max", float, where), where + ".bias_max")
    out["buckets"] = int(raw["bias_buckets"]) if raw.get("bias_buckets") is not None else None
    warmth = raw.get("q_temp")
    out["warmth"] = None
    if warmth is not None:
        every = _need(warmth, "every", float, where + ".q_temp")
        if every < 1 or every != int(every):
            raise ConfigError(f"config.json: {where}.q_temp.every must be a whole number of positions")
        out["warmth"] = (_need(warmth, "coef", float, where + ".q_temp"), int(every))


def _parse_mixer(kind: str, raw: dict, where: str) -> dict:
    out = {k: _need(raw, k, int, where) for k in ("heads", "dim", "vdim")}
    for k in ("heads", "dim", "vdim"):
        if out[k] < 1:
            raise ConfigError(f"config.json: {where}.{k} must be at least 1")
    if kind == "retention":
        _parse_retention(raw, out, where)
    else:
        _parse_attention(kind, raw, out, where)
    return out


def _parse_mlp(raw, where: str):
    if raw is None:
        return None
    kind = _need(raw, "kind", str, where)
    if kind != "moe":
        raise ConfigError(f"config.json: {where}.kind = {kind!r} is not 'moe'")
    router, shared = raw.get("router") or {}, raw.get("shared")
    out = {"ff": _need(raw.get("expert") or {}, "ff", int, where + ".expert"),
           "experts": _need(router, "experts", int, where + ".router"),
           "top": _need(router, "top", int, where + ".router"),
           "scale": float(router["scale"]) if router.get("scale") is not None else 1.0,
           "shared": _need(shared, "ff", int, where + ".shared") if shared else None}
    if out["ff"] < 1 or (out["shared"] is not None and out["shared"] < 1):
        raise ConfigError(f"config.json: {where}: an expert has at least one unit")
    if not 1 <= out["top"] <= out["experts"]:
        raise ConfigError(f"config.json: {where}.router.top must be between 1 and the number of experts")
    return out


@dataclass(frozen=True)
class LivitarLayer:
    type: str
    mixer: dict
    mlp: dict | None


@dataclass(frozen=True)
class LivitarConfig:
    architecture: str
    vocab_size: int
    hidden_size: int
    max_position_embeddings: int
    norm_eps: float
    streams: int
    layers: tuple[LivitarLayer, ...]
    eos_token_ids: tuple[int, ...] = ()
    torch_dtype: str = "bfloat16"

    @classmethod
    def from_dict(cls, raw: dict[str, Any]) -> "LivitarConfig":
        listed = raw.get("layers")
        if not isinstance(listed, list) or not listed:
            raise ConfigError("config.json: 'layers' must list at least one layer")
        layers = []
        for i, entry in enumerate(listed):
            where = f"layers[{i}]"
            kind = _need(entry, "type", str, where)
            if kind not in LAYER_TYPES:
                raise ConfigError(f"config.json: {where}.type = {kind!r} is not one of {LAYER_TYPES}")
            layers.append(LivitarLayer(kind, _parse_mixer(kind, entry.get("mixer") or {}, where + ".mixer"),
                                       _parse_mlp(entry.get("mlp"), where + ".mlp")))
        cfg = cls(
            architecture=str(raw.get("architecture", NAME)),
            vocab_size=_need(raw, "vocab", int, "the model"),
            hidden_size=_need(raw, "width", int, "the model"),
            max_position_embeddings=int(raw.get("max_positions") or NO_POSITION_LIMIT),
            norm_eps=_positive(_need(raw.get("norm") or {}, "eps", float, "norm"), "norm.eps"),
            streams=_need(raw, "streams", int, "the model"),
            layers=tuple(layers),
            eos_token_ids=id_tuple(raw.get("eos_token_id")),
            torch_dtype=str(raw.get("torch_dtype", "bfloat16")),
        )
        for key in ("vocab_size", "hidden_size", "max_position_embeddings"):
            if getattr(cfg, key) < 1:
                raise ConfigError(f"config.json: {key} must be >= 1")
        if not 1 <= cfg.streams <= 16:
            raise ConfigError("config.json: streams must be between 1 and 16")
        return cfg

    def complete_from_folder(self, model_dir) -> "LivitarConfig":
        return self.with_tensor_shapes(read_tensor_shapes(model_dir))

    def with_tensor_shapes(self, shapes: dict[str, tuple[int, ...]]) -> "LivitarConfig":
        """Fill in the size only a tensor's shape gives: the number of distance buckets."""
        layers = []
        for i, layer in enumerate(self.layers):
            mixer, name = dict(layer.mixer), f"l{i}.mix.rel"
            if layer.type == "attention_2" and mixer.get("buckets") is None and name in shapes:
                mixer["buckets"] = int(shapes[name][0])
            layers.append(LivitarLayer(layer.type, mixer, layer.mlp))
        return LivitarConfig(**{**self.__dict__, "layers": tuple(layers)})


def _rotary_name(layer: LivitarLayer) -> str | None:
    if not layer.mixer.get("rot_dims"):
        return None
    return f"rot_{layer.mixer['rot_dims']}_{layer.mixer['rot_base']!r}"


def _mixer_spec(cfg: LivitarConfig, i: int, layer: LivitarLayer) -> PartSpec:
    p, m = f"l{i}.mix", layer.mixer
    names = {k: f"{p}.{k}" for k in ("q", "k", "v", "o")}
    sizes = {k: m[k] for k in ("heads", "dim", "vdim")}
    if layer.type == "retention":
        return PartSpec("retention", {"names": {**names, "g": f"{p}.g"}, **sizes, "decay": m["decay"],
                                      "eps": cfg.norm_eps, "position": _rotary_name(layer)})
    params = {**sizes, "kv_heads": m["kv_heads"], "scale": m["scale"], "window": None, "eps": cfg.norm_eps}
    names["gate"] = f"{p}.g"
    if layer.type == "attention":
        names.update({k: f"{p}.{k}" for k in ("temp", "r1", "r2")})
    else:
        if m.get("buckets") is None:
            raise ConfigError(f"layers[{i}].mixer: the number of distance buckets is known neither from the shape of "
                              "rel nor from 'bias_buckets'")
        if m["buckets"] < 1 or not m["bias_max"] > m["buckets"] // 2:
            raise ConfigError(f"layers[{i}].mixer.bias_max must lie beyond half the {m['buckets']} buckets")
        names["rel"] = f"{p}.rel"
        params.update(unit_qk=True, warmth=m["warmth"], rel_buckets=m["buckets"], bias_max=m["bias_max"])
    return PartSpec("sink_attention", {"names": names, **params})


def _mlp_spec(i: int, mlp: dict | None) -> PartSpec | None:
    if mlp is None:
        return None
    p = f"l{i}.mlp"
    shared = None
    if mlp["shared"] is not None:
        shared = PartSpec("swiglu", {"gate_proj": f"{p}.shared.gate", "up_proj": f"{p}.shared.up",
                                     "down_proj": f"{p}.shared.down", "intermediate_size": mlp["shared"]})
    # experts: down(silu(gate(x)) * up(x)); nothing is clamped
    return PartSpec("routed_experts", {
        "router": f"{p}.router", "expert_prefix": f"{p}.e", "experts": mlp["experts"], "top": mlp["top"],
        "groups": 1, "keep_groups": 1, "weight_scale": mlp["scale"], "intermediate_size": mlp["ff"],
        "limit": None, "alpha": 1.0, "up_offset": 0.0, "shared": shared})


def _norm_spec(name: str) -> PartSpec:
    return PartSpec("dynamic_tanh", {"weight": name, "bias": name + ".b", "alpha": name + ".alpha"})


def livitar_spec(cfg: LivitarConfig) -> ModelSpec:
    layers, positions = [], {}
    for i, layer in enumerate(cfg.layers):
        name = _rotary_name(layer)
        if name is not None:
            positions.setdefault(name, PartSpec("rotary", {"rotary_dim": layer.mixer["rot_dims"],
                                                           "theta": layer.mixer["rot_base"], "angles": "float64"}))
        hc = {which: {k: f"l{i}.{tensor}.{k}" for k in ("in", "mix", "out")}
              for which, tensor in (("mixer", "hc1"), ("feed_forward", "hc2"))}
        norms = {"pre_mixer": _norm_spec(f"l{i}.norm1")}
        if layer.mlp is not None:
            norms["pre_feed_forward"] = _norm_spec(f"l{i}.norm2")
        layers.append(LayerSpec(prefix=f"l{i}", block=PartSpec("hyper_residual", {"streams": cfg.streams, **hc}),
                                mixer=_mixer_spec(cfg, i, layer), feed_forward=_mlp_spec(i, layer.mlp), norms=norms))
    return ModelSpec(
        architecture=cfg.architecture, vocab_size=cfg.vocab_size, hidden_size=cfg.hidden_size,
        max_position_embeddings=cfg.max_position_embeddings,
        embedding=PartSpec("token", {"weight": "embed", "vocab_size": cfg.vocab_size, "copies": cfg.streams}),
        positions=positions, layers=tuple(layers), schedule=tuple(ScheduleEntry(i) for i in range(len(layers))),
        final_norm=_norm_spec("final.norm"),
        head=PartSpec("linear", {"weight": "head", "vocab_size": cfg.vocab_size}),
        eos_token_ids=cfg.eos_token_ids)


def livitar_footprint(cfg: LivitarConfig) -> Footprint:
    h, s = cfg.hidden_size, cfg.streams
    norm, mixing = 2 * h + 1, s * s + 2 * s
    params = cfg.vocab_size * h * 2 + norm
    per_token = per_request = 0
    for layer in cfg.layers:
        m = layer.mixer
        q, v_out = m["heads"] * m["dim"], m["heads"] * m["vdim"]
        params += norm + mixing + q * h + 2 * v_out * h  # queries, gate, output
        if layer.type == "retention":
            params += (q + v_out) * h
            per_request += q * m["vdim"]
        else:
            k, v = m["kv_heads"] * m["dim"], m["kv_heads"] * m["vdim"]
            params += (k + v) * h + (3 if layer.type == "attention" else m.get("buckets") or 0) * m["heads"]
            per_token += k + v
        if layer.mlp is not None:
            params += norm + mixing + layer.mlp["experts"] * (3 * layer.mlp["ff"] * h + h)
            params += 3 * (layer.mlp["shared"] or 0) * h
    return Footprint(params, per_token, per_request)


def describe_livitar(cfg: LivitarConfig) -> list[str]:
    kinds = [layer.type + ("" if layer.mlp is None else "+moe") for layer in cfg.layers]
    fp = livitar_footprint(cfg)
    return [
        f"architecture        {cfg.architecture}",
        f"layers / width      {len(cfg.layers)} / {cfg.hidden_size}",
        f"residual streams    {cfg.streams}",
        f"layer kinds         {', '.join(kinds)}",
        f"parameters          {fp.parameters / 1e9:.3f} B",
        f"cache per token     {fp.cache_bytes_per_token(2)} B (bf16), state per request {fp.state_values_per_request * 4} B",
    ]


register_architecture(NAME, LivitarConfig, livitar_spec, describe_livitar, livitar_footprint)
