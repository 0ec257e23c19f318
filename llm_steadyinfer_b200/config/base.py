"""Typed model configuration: the base class, the architecture registry and the
specs that describe one model layer by layer.

A model is described as data:

* ``MixerSpec`` / ``FeedForwardSpec`` / ``NormSpec`` / ``PositionSpec`` name a
  registered part kind and carry its sizes and constants.
* ``LayerSpec`` puts one mixer, one feed-forward and their norms together and says
  which cache group the mixer stores into (or which other layer's cache it reads).
* ``ModelSpec`` holds the layer list and ``order``: the sequence in which layers run,
  which may name a layer twice.

The reference keeps a 36-byte binary header (src/include/model/config.h:4-31) and
derives sizes in ``Model::generate_model_infos`` (src/source/model/model.cpp:355-383);
here every size and constant comes from config.json keys.
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass, field
from typing import Any, Callable, Dict, List, Optional


class ConfigError(ValueError):
    """A config.json key is missing, has the wrong type or an unsupported value."""


@dataclass(frozen=True)
class PositionSpec:
    kind: str                      # registered position-encoding kind, e.g. "rotary"
    params: Dict[str, Any] = field(default_factory=dict)


@dataclass(frozen=True)
class NormSpec:
    kind: str                      # e.g. "rmsnorm"
    params: Dict[str, Any] = field(default_factory=dict)


@dataclass(frozen=True)
class MixerSpec:
    kind: str                      # e.g. "attention"
    params: Dict[str, Any] = field(default_factory=dict)
    position: Optional[PositionSpec] = None


@dataclass(frozen=True)
class FeedForwardSpec:
    kind: str                      # e.g. "gated_mlp"
    params: Dict[str, Any] = field(default_factory=dict)


@dataclass(frozen=True)
class EmbedderSpec:
    kind: str = "table"            # registered embedder kind
    params: Dict[str, Any] = field(default_factory=dict)


@dataclass(frozen=True)
class LayerSpec:
    """One block: ``h += mixer(norm(h)); h += ffn(norm(h))`` for arrangement "pre_norm".

    With arrangement "sandwich" each sublayer has a second norm behind it, applied to the sublayer's result before
    it joins the stream (``mixer_post_norm``, ``feed_forward_post_norm``):
    ``h += norm_b(mixer(norm(h))); h += norm_b(ffn(norm(h)))``.

    With arrangement "parallel_gated" both sublayers read the same stream, each through its own norm, and each result
    passes a learned gate: ``h += residual_scale * (sigmoid(W1 x1 + b1) * mixer(x1) + sigmoid(W2 x2 + b2) * ffn(x2))``,
    ``x1 = norm1(h)``, ``x2 = norm2(h)`` (``mixer_gate_name``, ``feed_forward_gate_name``).

    With arrangement "streams" the residual stream has ``ModelSpec.streams`` copies and each sublayer has connections to
    them (``mixer_streams_prefix``, ``feed_forward_streams_prefix``; see ``StreamConnections``).

    ``weight_prefix`` is the checkpoint prefix of this layer ("model.layers.3.").
    ``cache_from`` is None when the layer owns its cache, or the index of the layer
    whose cache it reads (it then writes nothing): that of the latest run of that layer
    before it in the run order.
    """
    mixer: MixerSpec
    feed_forward: Optional[FeedForwardSpec]      # None: the block has the mixer's sublayer only
    mixer_norm: NormSpec
    feed_forward_norm: Optional[NormSpec]
    weight_prefix: str
    arrangement: str = "pre_norm"
    cache_from: Optional[int] = None
    # checkpoint names of the parts below weight_prefix
    mixer_prefix: str = "self_attn."
    feed_forward_prefix: str = "mlp."
    mixer_norm_name: str = "input_layernorm."
    feed_forward_norm_name: str = "post_attention_layernorm."
    # norms behind the sublayers (arrangement "sandwich")
    mixer_post_norm: Optional[NormSpec] = None
    feed_forward_post_norm: Optional[NormSpec] = None
    mixer_post_norm_name: str = "post_mixer_norm."
    feed_forward_post_norm_name: str = "post_feed_forward_norm."
    # learned gates on the sublayers' results (arrangement "parallel_gated"): tensor names below weight_prefix of the
    # matrices [hidden, hidden]; their biases are ``<name>.b``
    mixer_gate_name: Optional[str] = None
    feed_forward_gate_name: Optional[str] = None
    # connections to a stream of several copies (arrangement "streams"): tensor prefixes below weight_prefix
    mixer_streams_prefix: Optional[str] = None
    feed_forward_streams_prefix: Optional[str] = None
    token_side_prefix: Optional[str] = None      # tensor prefix of the layer's own input for each token (``ModelSpec.token_side``)
    residual_scale: float = 1.0                  # what a block adds to the stream is multiplied by it


@dataclass(frozen=True)
class StreamAddSpec:
    """Something the residual stream gains between layers: before the run at ``place`` of the run order, the
    embedder's output (the stream as it was before the first layer) is added again if ``embedding`` is set, and row
    ``row`` of the checkpoint tensor ``vector_name`` ([rows, hidden]) if a name is given. Models that run a span
    of layers several times use it at the start of each pass."""
    place: int
    embedding: bool = False
    vector_name: Optional[str] = None
    row: int = 0


@dataclass(frozen=True)
class TokenSideSpec:
    """A second embedding table whose columns are shared out among the layers (``TokenSideInput``): layer i's input for a token is the part
    [i * dim, (i + 1) * dim) of the token's row of ``table_name`` ([vocab, layers * dim])."""
    dim: int
    eps: float
    table_name: str = "side.embed"


@dataclass(frozen=True)
class ModelSpec:
    hidden_size: int
    vocab_size: int
    layers: List[LayerSpec]
    order: List[int]               # run order: indices into ``layers``
    final_norm: NormSpec
    tie_word_embeddings: bool
    embed_name: str = "model.embed_tokens.weight"
    final_norm_name: str = "model.norm."
    lm_head_name: str = "lm_head.weight"
    max_position: int = 0
    embedder: Optional[EmbedderSpec] = None      # None: the plain table under ``embed_name``
    stream_adds: tuple = ()                      # StreamAddSpec entries, at most one a place
    stream_vector_shapes: Optional[Dict[str, tuple]] = None   # the tensors that ``stream_adds`` name: name -> shape
    streams: Optional[int] = None                # copies of the residual stream (arrangement "streams"); None: the one stream
    token_side: Optional[TokenSideSpec] = None   # layers with a ``token_side_prefix`` have an input of their own for each token
    logit_scale: float = 1.0                     # logits are multiplied by it (before the soft cap)
    logit_softcap: float = 0.0                   # > 0: logits <- cap * tanh(logits / cap)


class ModelConfig:
    """Base of every architecture's typed configuration."""

    architecture: str = ""

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "ModelConfig":
        raise NotImplementedError

    def to_dict(self) -> Dict[str, Any]:
        raise NotImplementedError

    def model_spec(self) -> ModelSpec:
        raise NotImplementedError


_ARCHITECTURES: Dict[str, Callable[[Dict[str, Any]], ModelConfig]] = {}


def register_architecture(name: str, config_cls) -> None:
    """Map config.json's ``architectures[0]`` to a configuration class.

    The class's ``model_spec()`` is the architecture's model: the list of layers
    and the order they run in, built from registered parts.
    """
    _ARCHITECTURES[name] = config_cls


def registered_architectures() -> List[str]:
    return sorted(_ARCHITECTURES)


def config_from_dict(d: Dict[str, Any]) -> ModelConfig:
    archs = d.get("architectures")
    if archs is None and isinstance(d.get("architecture"), str):       # some designs name themselves with one string
        archs = [d["architecture"]]
    if not isinstance(archs, list) or not archs or not isinstance(archs[0], str):
        raise ConfigError("config.json: key 'architectures' must be a non-empty list of names "
                          "(or 'architecture' one name)")
    name = archs[0]
    if name not in _ARCHITECTURES:
        raise ConfigError(
            f"config.json: architecture {name!r} is not registered; "
            f"registered: {registered_architectures()}")
    return _ARCHITECTURES[name].from_dict(d)


def load_config(model_dir: str) -> ModelConfig:
    path = os.path.join(model_dir, "config.json")
    if not os.path.isfile(path):
        raise ConfigError(f"no config.json in {model_dir!r}")
    with open(path, "r", encoding="utf-8") as f:
        try:
            d = json.load(f)
        except json.JSONDecodeError as e:
            raise ConfigError(f"{path}: not valid JSON ({e})") from None
    if not isinstance(d, dict):
        raise ConfigError(f"{path}: top level must be an object")
    return config_from_dict(d)


# ---- helpers for typed reading -------------------------------------------------

_MISSING = object()


def read_key(d: Dict[str, Any], key: str, typ, default=_MISSING, *, positive=False):
    """Read ``d[key]`` as ``typ`` (int, float, bool, str); name the key on failure."""
    if key not in d or d[key] is None:
        if default is _MISSING:
            raise ConfigError(f"config.json: required key {key!r} is missing")
        return default
    v = d[key]
    if typ is float and isinstance(v, int) and not isinstance(v, bool):
        v = float(v)
    if typ is int and isinstance(v, bool):
        raise ConfigError(f"config.json: key {key!r} must be an integer, found {v!r}")
    if not isinstance(v, typ):
        raise ConfigError(
            f"config.json: key {key!r} must be {typ.__name__}, found {type(v).__name__} {v!r}")
    if positive and not v > 0:
        raise ConfigError(f"config.json: key {key!r} must be positive, found {v!r}")
    return v
