"""The Lomopel architecture: config.json keys and tensor names.

A pre-norm decoder whose layers are listed one by one in ``layers``: x += ls1 * mixer(norm1(x)); x += ls2 * ff(norm2(x)), ls1
and ls2 learned vectors (layer scale), the second half absent when ``mlp`` is null.  The norms are RMS norms whose weight is
stored around zero (the gain is 1 + w).  The mixer (``type``) is one of

  "attention"   grouped-query attention without rotation, with biases on all four projections; the query is multiplied by a
                factor that grows with the logarithm of the position (``q_temp``), the softmax has a learned sink per head,
                and with ``v_mix`` a layer's values are mixed with those of the first such layer, by a learned weight;
  "parallel"    two mixers that read the same input, their outputs added with a scale each: on the left grouped-query
                attention with rotated, unit-normed queries and keys, a sliding window (``mask.size``) and a sigmoid gate per
                coordinate; on the right the gated delta rule with a decay per head and key channel, decay and output gate
                each from two thin matrices whose inner size the tensors give.

The feed-forward (``mlp.kind`` "dense") is a gated unit with the tanh form of gelu.  The embedding's rows are multiplied by
``embedding.scale``; the output has a matrix of its own.

Every size and every constant that may differ between models of the design is read here from config.json (or, for the
thin matrices, from the tensors); nothing is taken from a particular model.
"""
from __future__ import annotations

from typing import Any, Dict, Optional, Tuple

from ..config.model_config import (ConfigError, EmbeddingSpec, FeedForwardSpec, HeadSpec, LayerRun, LayerSpec, MixerSpec,
                                   ModelConfig, NormSpec, PositionSpec, optional, require)
from ..config.registry import register_architecture

NAME = "Lomopel"

# Positions are computed, not looked up, so nothing ends a sequence but the cache.
NO_POSITION_LIMIT = 1 << 30


def _count(raw: Dict[str, Any], key: str, where: str) -> int:
    n = require(raw, key, int)
    if n <= 0:
        raise ConfigError(f"config.json: {where}.{key} must be positive (found {n})")
    return n


def _object(raw: Dict[str, Any], key: str, where: str) -> Optional[Dict[str, Any]]:
    found = raw.get(key)
    if found is not None and not isinstance(found, dict):
        raise ConfigError(f"config.json: {where}.{key} must be an object or null")
    return found


def _heads(where: str, m: Dict[str, Any]) -> Tuple[int, int, int, int]:
    heads, dim = _count(m, "heads", where), _count(m, "dim", where)
    kv_heads = _count(m, "kv_heads", where) if m.get("kv_heads") is not None else heads
    vdim = _count(m, "vdim", where) if m.get("vdim") is not None else dim
    if heads % kv_heads:
        raise ConfigError(f"config.json: {where}: heads {heads} must be a multiple of kv_heads {kv_heads}")
    return heads, kv_heads, dim, vdim


def _position(where: str, m: Dict[str, Any], dim: int) -> PositionSpec:
    rot = _object(m, "rot", where)
    if rot is None:
        return PositionSpec(kind="none")
    dims = require(rot, "dims", int)
    if dims < 0 or dims % 2 or dims > dim:
        raise ConfigError(f"config.json: {where}.rot.dims {dims} must be even and at most {dim}")
    if dims == 0:
        return PositionSpec(kind="none")
    return PositionSpec(kind="rope_exact", theta=require(rot, "base", float), rotary_dim=dims, pairing="half")


def _attention(where: str, m: Dict[str, Any], eps: float, value_mix: Optional[str]) -> MixerSpec:
    heads, kv_heads, dim, vdim = _heads(where, m)
    temperature = _object(m, "q_temp", where)
    if temperature is not None:
        temperature = (require(temperature, "coef", float), require(temperature, "every", float))
        if not temperature[1] > 0:
            raise ConfigError(f"config.json: {where}.q_temp.every must be positive")
    return MixerSpec(kind="normed_qk_attention", num_heads=heads, num_kv_heads=kv_heads, head_dim=dim,
                     softmax_scale=require(m, "scale", float), position=PositionSpec(kind="none"),
                     extra=(("value_dim", vdim), ("norm_eps", eps), ("bias", True), ("output_bias", True), ("qk_norm", False),
                            ("sink", "learned"), ("temperature", temperature), ("value_mix", value_mix)))


def _window_attention(where: str, m: Dict[str, Any], eps: float) -> MixerSpec:
    heads, kv_heads, dim, vdim = _heads(where, m)
    mask = _object(m, "mask", where)
    return MixerSpec(kind="normed_qk_attention", num_heads=heads, num_kv_heads=kv_heads, head_dim=dim,
                     window=_count(mask, "size", where + ".mask") if mask is not None else None,
                     softmax_scale=require(m, "scale", float), position=_position(where, m, dim),
                     extra=(("value_dim", vdim), ("norm_eps", eps), ("bias", False), ("qk_norm", False),
                            ("head_unit_norm", True), ("element_gate", True)))


def _delta(where: str, m: Dict[str, Any], eps: float) -> MixerSpec:
    heads, kv_heads, dim, vdim = _heads(where, m)
    return MixerSpec(kind="gated_delta", num_heads=heads, num_kv_heads=kv_heads, head_dim=dim, position=PositionSpec(kind="none"),
                     extra=(("value_dim", vdim), ("conv_taps", _count(m, "conv", where)), ("norm_eps", eps),
                            ("decay", "key_channel"), ("gate", "low_rank_sigmoid")))


def _mixer(i: int, layer: Dict[str, Any], eps: float, value_mix: Optional[str]) -> MixerSpec:
    kind, m = require(layer, "type", str), require(layer, "mixer", dict)
    where = f"layers[{i}].mixer"
    if kind == "attention":
        return _attention(where, m, eps, value_mix)
    if kind == "parallel":
        left = _window_attention(where + ".left", require(m, "left", dict), eps)
        right = _delta(where + ".right", require(m, "right", dict), eps)
        return MixerSpec(kind="parallel_mixers",
                         extra=(("left", left), ("right", right), ("left_scale", require(m, "left_scale", float)),
                                ("right_scale", require(m, "right_scale", float)), ("join", True)))
    raise ConfigError(f"config.json: layers[{i}].type '{kind}' is not a mixer of this architecture (attention, parallel)")


def _value_mixes(layers_raw) -> Dict[int, str]:
    """Per attention layer that mixes values: "first" for the one the others mix in, "later" for those.  Their values must
    have one shape."""
    mixes, shape = {}, None
    for i, layer in enumerate(layers_raw):
        m = layer.get("mixer")
        if layer.get("type") != "attention" or not isinstance(m, dict) or not optional(m, "v_mix", bool, False):
            continue
        _, kv_heads, _, vdim = _heads(f"layers[{i}].mixer", m)
        if shape is None:
            shape = kv_heads * vdim
        elif kv_heads * vdim != shape:
            raise ConfigError(f"config.json: layers[{i}].mixer: layers that mix values must have values of one size")
        mixes[i] = "later" if mixes else "first"
    return mixes


def _feed_forward(i: int, layer: Dict[str, Any]) -> Optional[FeedForwardSpec]:
    mlp = _object(layer, "mlp", f"layers[{i}]")
    if mlp is None:
        return None
    kind = require(mlp, "kind", str)
    if kind != "dense":
        raise ConfigError(f"config.json: layers[{i}].mlp.kind '{kind}' is not supported (dense)")
    return FeedForwardSpec(kind="swiglu", intermediate_size=_count(mlp, "ff", f"layers[{i}].mlp"),
                           extra=(("activation", "gelu_tanh"), ("f32_out", True)))


def parse_config(raw: Dict[str, Any]) -> ModelConfig:
    width, vocab = _count(raw, "width", "config"), _count(raw, "vocab", "config")
    eps = require(require(raw, "norm", dict), "eps", float)
    layers_raw = raw.get("layers")
    if not isinstance(layers_raw, list) or not layers_raw or not all(isinstance(x, dict) for x in layers_raw):
        raise ConfigError("config.json: 'layers' must be a non-empty list of objects")
    emb = _object(raw, "embedding", "config") or {}
    norm = NormSpec(kind="rmsnorm_one_plus", eps=eps)
    mixes = _value_mixes(layers_raw)
    layers = []
    for i, layer in enumerate(layers_raw):
        ffn = _feed_forward(i, layer)
        layers.append(LayerSpec(mixer=_mixer(i, layer, eps, mixes.get(i)), feed_forward=ffn, mixer_norm=norm,
                                ffn_norm=norm if ffn is not None else None, arrangement="pre_norm",
                                extra=(("layer_scale", True),)))
    return ModelConfig(
        architecture=NAME, hidden_size=width, vocab_size=vocab, max_position_embeddings=NO_POSITION_LIMIT,
        layers=tuple(layers), schedule=tuple(LayerRun(layer=i) for i in range(len(layers))), final_norm=norm,
        tie_word_embeddings=False,
        embedding=EmbeddingSpec(kind="table", extra=(("row_scale", optional(emb, "scale", float, 1.0)),)),
        head=HeadSpec(kind="linear", tied=False), raw=tuple(sorted((k, repr(v)) for k, v in raw.items())))


_NORMS = {"mixer_norm": "norm1", "ffn_norm": "norm2"}


def tensor_name(scope: Tuple, slot: str) -> str:
    if scope == ("embedding",):
        return "embed"
    if scope == ("lm_head",):
        return "head"
    if scope == ("final_norm",):
        return "final.norm"
    if scope[0] == "layer":
        _, i, what = scope
        if what == "mixer":
            return f"l{i}.mix.{slot}"
        if what == "feed_forward":
            return f"l{i}.mlp.{slot}"
        if what == "block":
            return f"l{i}.{slot}"
        if what in _NORMS:
            return f"l{i}.{_NORMS[what]}"
    raise ConfigError(f"{NAME}: no tensor name for scope {scope} slot '{slot}'")


# A layer without a feed-forward has no use for a second norm or scale, nor one that mixes no values for a mixing weight.
register_architecture(NAME, parse_config, tensor_name, replace=True,
                      ignored_tensors=("l[0-9]*.norm2", "l[0-9]*.ls2", "l[0-9]*.mix.vmix"))
