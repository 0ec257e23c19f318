"""Risizen: a decoder whose residual stream has several copies ("streams") with learned connections between them and every
sublayer. config.json lists the layers one by one: a grouped-query attention mixer without rotation (projections with
biases, a short causal convolution on every channel of q, k and v, queries and keys scaled to a root mean square of one,
positions in chunks that see only themselves, a sink whose score is 0 in the softmax denominator), some layers of which read
the keys and values of an earlier one, and a gated feed-forward with limits. The embedding's output is normalised and the
logits are scaled.

config.json:
    architecture    "Risizen"
    vocab, width    sizes of the embedding and of the residual stream
    streams         copies of the residual stream
    norm.eps        of every RMS norm, those of queries and keys included
    logit_scale     logits are multiplied by it
    layers[i]       {type: "attention", mixer{heads, kv_heads, dim, vdim, conv, scale, mask{size}, [kv_from]},
                     mlp{kind: "dense", ff, limit} | null}
                    conv: taps of the convolutions; mask.size: the chunk's length (no mask: every earlier position is seen);
                    kv_from: the layer whose keys and values are read (it has no projections of keys and values itself)
Tensors: embed, embed.norm, l<i>.norm1, l<i>.norm2, l<i>.hc1.{in,out,mix}, l<i>.hc2.{in,out,mix},
l<i>.mix.{q,k,v}[.b|.conv], l<i>.mix.o, l<i>.mlp.{gate,up,down}, final.norm, head.

Everything is expressed with registered parts: the model below is a ``ModelSpec`` and nothing else.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Dict, List, Optional, Tuple

from ..config.base import (ConfigError, EmbedderSpec, FeedForwardSpec, LayerSpec, MixerSpec, ModelConfig, ModelSpec, NormSpec,
                           read_key, register_architecture)

# constants of the design
SINK_SCORE = 0.0                # one is added to the softmax denominator
GATE_ALPHA = 1.702              # g * sigmoid(alpha g)

MIXER_KEYS = (("heads", int), ("kv_heads", int), ("dim", int), ("vdim", int), ("conv", int))


def _sub(d: Dict[str, Any], key: str, where: str, optional: bool = False) -> Optional[Dict[str, Any]]:
    v = d.get(key)
    if v is None and optional:
        return None
    if not isinstance(v, dict):
        raise ConfigError(f"config.json: {where}{key!r} must be an object")
    return v


def _keyed(fn, where: str):
    try:
        return fn()
    except ConfigError as e:
        raise ConfigError(str(e).replace("key ", f"key {where}", 1)) from None


@dataclass(frozen=True)
class RisizenConfig(ModelConfig):
    vocab: int
    width: int
    streams: int
    eps: float
    logit_scale: float
    layers: Tuple[Dict[str, Any], ...]              # as in config.json, checked

    architecture = "Risizen"

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "RisizenConfig":
        vocab = read_key(d, "vocab", int, positive=True)
        width = read_key(d, "width", int, positive=True)
        streams = read_key(d, "streams", int, positive=True)
        eps = _keyed(lambda: read_key(_sub(d, "norm", ""), "eps", float, positive=True), "norm.")
        logit_scale = read_key(d, "logit_scale", float, 1.0)
        raw = d.get("layers")
        if not isinstance(raw, list) or not raw:
            raise ConfigError("config.json: key 'layers' must be a non-empty list")
        layers: List[Dict[str, Any]] = []
        for i, ent in enumerate(raw):
            where = f"layers[{i}]."
            if not isinstance(ent, dict):
                raise ConfigError(f"config.json: layers[{i}] must be an object")
            kind = read_key(ent, "type", str)
            if kind != "attention":
                raise ConfigError(f"config.json: {where}type {kind!r} is not supported (supported: 'attention')")
            mx = _sub(ent, "mixer", where)
            for key, typ in MIXER_KEYS:
                _keyed(lambda: read_key(mx, key, typ, positive=True), where + "mixer.")
            _keyed(lambda: read_key(mx, "scale", float), where + "mixer.")
            if mx["heads"] % mx["kv_heads"]:
                raise ConfigError(f"config.json: {where}mixer.heads is not a multiple of kv_heads")
            mask = _sub(mx, "mask", where + "mixer.", optional=True)
            if mask is not None:
                _keyed(lambda: read_key(mask, "size", int, positive=True), where + "mixer.mask.")
            src = _keyed(lambda: read_key(mx, "kv_from", int, None), where + "mixer.")
            if src is not None:
                if not 0 <= src < i or layers[src]["mixer"].get("kv_from") is not None:
                    raise ConfigError(f"config.json: {where}mixer.kv_from must name an earlier layer with keys of its own, found {src}")
                if any(layers[src]["mixer"][k] != mx[k] for k in ("kv_heads", "dim", "vdim")):
                    raise ConfigError(f"config.json: {where}mixer reads the keys of layer {src}, whose head counts or sizes differ")
            mlp = _sub(ent, "mlp", where, optional=True)
            if mlp is not None:
                if _keyed(lambda: read_key(mlp, "kind", str), where + "mlp.") != "dense":
                    raise ConfigError(f"config.json: {where}mlp.kind {mlp['kind']!r} is not supported (supported: 'dense')")
                _keyed(lambda: read_key(mlp, "ff", int, positive=True), where + "mlp.")
                _keyed(lambda: read_key(mlp, "limit", float, positive=True), where + "mlp.")
            layers.append(copy.deepcopy(ent))
        return cls(vocab=vocab, width=width, streams=streams, eps=eps, logit_scale=logit_scale, layers=tuple(layers))

    def to_dict(self) -> Dict[str, Any]:
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "streams": self.streams,
                "norm": {"eps": self.eps}, "logit_scale": self.logit_scale, "layers": copy.deepcopy(list(self.layers))}

    def eos_token_ids(self) -> List[int]:
        return []

    # ---- the model as data ---------------------------------------------------------------------
    def _mixer(self, mx: Dict[str, Any]) -> MixerSpec:
        return MixerSpec("attention", {
            "hidden_size": self.width, "num_heads": mx["heads"], "num_kv_heads": mx["kv_heads"], "head_dim": mx["dim"],
            "value_dim": mx["vdim"], "scale": float(mx["scale"]), "chunk": (mx.get("mask") or {}).get("size"),
            "conv_taps": mx["conv"], "conv_suffix": ".conv", "biases": True, "bias_suffix": ".b", "qk_norm": {"eps": self.eps},
            "sink_score": SINK_SCORE, "own_keys": mx.get("kv_from") is None, "names": {"q": "q", "k": "k", "v": "v", "o": "o"}})

    def model_spec(self) -> ModelSpec:
        norm = NormSpec("rmsnorm", {"size": self.width, "eps": self.eps, "weight_name": ""})
        specs: List[LayerSpec] = []
        for i, ent in enumerate(self.layers):
            mlp = ent.get("mlp")
            ffn = None if mlp is None else FeedForwardSpec("gated_mlp_limited", {
                "hidden_size": self.width, "intermediate_size": mlp["ff"], "limit": float(mlp["limit"]), "alpha": GATE_ALPHA,
                "biases": False, "names": {"gate": "gate", "up": "up", "down": "down"}})
            specs.append(LayerSpec(
                mixer=self._mixer(ent["mixer"]), feed_forward=ffn, mixer_norm=norm, feed_forward_norm=None if ffn is None else norm,
                weight_prefix=f"l{i}.", arrangement="streams", cache_from=ent["mixer"].get("kv_from"), mixer_prefix="mix.",
                feed_forward_prefix="mlp.", mixer_norm_name="norm1", feed_forward_norm_name="norm2", mixer_streams_prefix="hc1.",
                feed_forward_streams_prefix=None if ffn is None else "hc2."))
        return ModelSpec(hidden_size=self.width, vocab_size=self.vocab, layers=specs, order=list(range(len(specs))),
                         final_norm=norm, tie_word_embeddings=False, embed_name="embed", final_norm_name="final.norm",
                         lm_head_name="head", max_position=0, streams=self.streams, logit_scale=self.logit_scale,
                         embedder=EmbedderSpec("table", {"norm": {"eps": self.eps, "name": "embed.norm"}}))


register_architecture(RisizenConfig.architecture, RisizenConfig)
