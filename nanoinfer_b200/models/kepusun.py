"""The Kepusun architecture: config.json keys and tensor names.

A decoder whose layers are listed one by one in ``layers`` and which carries ``streams`` residual streams side by side
(hyper-connections): a sublayer reads a weighted sum of them through its norm, and afterwards every stream is made anew
from all the old ones and the sublayer's output.  The norm is tanh(alpha x) * w + b, without statistics.  The mixer
(``type``) is one of

  "mlstm"       a matrix memory with exponential gates: S <- decay S + strength k v^T, its decay and strength numbers of
                every token, kept in a stabilised form with a normaliser; a norm per head, a sigmoid gate;
  "attention"   differential attention: two causal softmax maps per head over the same values, the second taken off the
                first, the rest normed per head; no position encoding.  A layer with ``kv_from``: j has no keys and
                values of its own: it reads layer j's cache.

The feed-forward (``mlp.kind`` "moe", or null) routes every token to ``top`` of many small squared-relu units: softmax
scores, the best groups of neighbouring experts first, then the best experts in them, weights over their sum times a factor.
The output has a matrix of its own.

Every size and every constant that may differ between models of the design is read here from config.json; nothing is
taken from a particular model.
"""
from __future__ import annotations

from typing import Any, Dict, Optional, Tuple

from ..config.model_config import (ConfigError, EmbeddingSpec, FeedForwardSpec, HeadSpec, LayerRun, LayerSpec, MixerSpec,
                                   ModelConfig, NormSpec, PositionSpec, require)
from ..config.registry import register_architecture

NAME = "Kepusun"

# Nothing in the design depends on positions, so nothing ends a sequence but the cache.
NO_POSITION_LIMIT = 1 << 30


def _count(raw: Dict[str, Any], key: str, where: str) -> int:
    n = require(raw, key, int)
    if n <= 0:
        raise ConfigError(f"config.json: {where}.{key} must be positive (found {n})")
    return n


def _matrix_memory(where: str, m: Dict[str, Any], eps: float) -> MixerSpec:
    heads, dim = _count(m, "heads", where), _count(m, "dim", where)
    vdim = _count(m, "vdim", where) if m.get("vdim") is not None else dim
    cap = require(m, "gate_cap", float)
    if not cap > 0.0:
        raise ConfigError(f"config.json: {where}.gate_cap must be positive (found {cap})")
    return MixerSpec(kind="matrix_memory", num_heads=heads, num_kv_heads=heads, head_dim=dim, position=PositionSpec(kind="none"),
                     extra=(("value_dim", vdim), ("gate_cap", cap), ("norm_eps", eps)))


def _differential_attention(where: str, m: Dict[str, Any], eps: float, own: bool) -> MixerSpec:
    heads, dim = _count(m, "heads", where), _count(m, "dim", where)
    kv_heads = _count(m, "kv_heads", where) if m.get("kv_heads") is not None else heads
    vdim = _count(m, "vdim", where) if m.get("vdim") is not None else dim
    if heads % kv_heads:
        raise ConfigError(f"config.json: {where}: heads {heads} must be a multiple of kv_heads {kv_heads}")
    return MixerSpec(kind="differential_attention", num_heads=heads, num_kv_heads=kv_heads, head_dim=dim,
                     softmax_scale=require(m, "scale", float), position=PositionSpec(kind="none"),
                     extra=(("value_dim", vdim), ("norm_eps", eps), ("diff", require(m, "diff", float)), ("own_kv", own)))


def _kv_source(i: int, layers_raw) -> Optional[int]:
    """The layer whose keys and values attention layer i reads, or None if it has its own."""
    where = f"config.json: layers[{i}].mixer.kv_from"
    m = layers_raw[i]["mixer"]
    j = m.get("kv_from")
    if j is None:
        return None
    if not isinstance(j, int) or isinstance(j, bool) or not 0 <= j < i:
        raise ConfigError(f"{where} must name an earlier layer")
    src = layers_raw[j]
    if src.get("type") != "attention" or not isinstance(src.get("mixer"), dict) or src["mixer"].get("kv_from") is not None:
        raise ConfigError(f"{where}: layer {j} has no keys and values of its own")

    def sizes(x):
        heads, dim = x.get("heads"), x.get("dim")
        return (x.get("kv_heads") if x.get("kv_heads") is not None else heads, dim, x.get("vdim") if x.get("vdim") is not None else dim)

    if sizes(m) != sizes(src["mixer"]):
        raise ConfigError(f"{where}: layer {j}'s keys and values have other sizes")
    return j


def _feed_forward(i: int, layer: Dict[str, Any]) -> Optional[FeedForwardSpec]:
    mlp = layer.get("mlp")
    if mlp is None:
        return None
    where = f"layers[{i}].mlp"
    if not isinstance(mlp, dict):
        raise ConfigError(f"config.json: {where} must be an object or null")
    kind = require(mlp, "kind", str)
    if kind != "moe":
        raise ConfigError(f"config.json: {where}.kind '{kind}' is not supported (moe)")
    r = require(mlp, "router", dict)
    experts, top = _count(r, "experts", where + ".router"), _count(r, "top", where + ".router")
    if top > experts:
        raise ConfigError(f"config.json: {where}.router: top {top} of {experts} experts")
    count = keep = 1
    if r.get("groups") is not None:
        groups = require(r, "groups", dict)
        count, keep = _count(groups, "count", where + ".router.groups"), _count(groups, "keep", where + ".router.groups")
        if experts % count or keep > count or keep * (experts // count) < top:
            raise ConfigError(f"config.json: {where}.router.groups: {keep} of {count} groups do not fit {experts} experts with top {top}")
    return FeedForwardSpec(kind="routed_experts", intermediate_size=_count(require(mlp, "expert", dict), "ff", where + ".expert"),
                           extra=(("experts", experts), ("top", top), ("unit", "relu2"), ("scores", "softmax"), ("renormalize", True),
                                  ("weight_scale", require(r, "scale", float)), ("groups", count), ("keep_groups", keep)))


def parse_config(raw: Dict[str, Any]) -> ModelConfig:
    width, vocab, streams = (_count(raw, k, "config") for k in ("width", "vocab", "streams"))
    eps = require(require(raw, "norm", dict), "eps", float)
    layers_raw = raw.get("layers")
    if not isinstance(layers_raw, list) or not layers_raw or not all(isinstance(x, dict) for x in layers_raw):
        raise ConfigError("config.json: 'layers' must be a non-empty list of objects")
    norm = NormSpec(kind="dynamic_tanh", eps=eps)
    layers, schedule = [], []
    for i, layer in enumerate(layers_raw):
        kind, m = require(layer, "type", str), require(layer, "mixer", dict)
        where = f"layers[{i}].mixer"
        source = None
        if kind == "mlstm":
            mixer = _matrix_memory(where, m, eps)
        elif kind == "attention":
            source = _kv_source(i, layers_raw)
            mixer = _differential_attention(where, m, eps, source is None)
        else:
            raise ConfigError(f"config.json: layers[{i}].type '{kind}' is not a mixer of this architecture (mlstm, attention)")
        ffn = _feed_forward(i, layer)
        layers.append(LayerSpec(mixer=mixer, feed_forward=ffn, mixer_norm=norm, ffn_norm=norm if ffn is not None else None,
                                arrangement="hyper_connections", extra=(("streams", streams),)))
        schedule.append(LayerRun(layer=i, cache_of=source))
    return ModelConfig(
        architecture=NAME, hidden_size=width, vocab_size=vocab, max_position_embeddings=NO_POSITION_LIMIT,
        layers=tuple(layers), schedule=tuple(schedule), final_norm=norm, tie_word_embeddings=False, streams=streams,
        embedding=EmbeddingSpec(kind="table"), head=HeadSpec(kind="linear", tied=False),
        raw=tuple(sorted((k, repr(v)) for k, v in raw.items())))


_NORMS = {"mixer_norm": "norm1", "ffn_norm": "norm2"}


def _norm_tensor(name: str, slot: str) -> str:
    return name if slot == "weight" else f"{name}.{slot}"


def tensor_name(scope: Tuple, slot: str) -> str:
    if scope == ("embedding",):
        return "embed"
    if scope == ("lm_head",):
        return "head"
    if scope == ("final_norm",):
        return _norm_tensor("final.norm", slot)
    if scope[0] == "layer":
        _, i, what = scope
        if what == "mixer":
            return f"l{i}.mix.{slot}"
        if what == "feed_forward":
            return f"l{i}.mlp.{slot}"
        if what == "block":
            return f"l{i}.{slot}"
        if what in _NORMS:
            return _norm_tensor(f"l{i}.{_NORMS[what]}", slot)
    raise ConfigError(f"{NAME}: no tensor name for scope {scope} slot '{slot}'")


register_architecture(NAME, parse_config, tensor_name, replace=True)
