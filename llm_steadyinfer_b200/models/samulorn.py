"""Samulorn: a decoder whose config.json lists its layers one by one. A layer's mixer is a gated delta rule with a decay per key channel,
or a pair of mixers side by side, grouped-query attention (biases, short convolutions, rotation in neighbouring pairs with scaled
frequencies, queries and keys scaled to a root mean square of one) and a recurrent block with a real-gated linear recurrence; its
feed-forward is dense or routed with groups of experts. Every norm of the stream is a dynamic tanh, before and behind each
sublayer, and every layer ends with an input of its own for the token. A span of the layers may run several times in a row with
the same weights and a cache or state of its own per pass. The embedding table, without its scale, is the head.

config.json:
    architecture    "Samulorn"
    vocab, width    sizes of the embedding and of the residual stream
    norm.eps        of every root mean square
    embedding.scale the embedding's rows are multiplied by it (absent: 1)
    token_side.dim  entries of a layer's input for a token (absent: the layers have none)
    layers[i]       {type, mixer{...}, mlp{...} | null}
      type "channel_delta": mixer {heads, kv_heads, dim, vdim, conv} (and ``rank``, of the low-rank products, where no checkpoint is
                    there to say it)
      type "parallel": mixer {left, right, left_scale, right_scale}
        left        {heads, kv_heads, dim, vdim, conv, scale, rot{base, dims, scaling{factor, low, high, original} | null} | null}
        right       {width, blocks, conv}
      mlp           {kind: "dense", ff} or {kind: "moe", expert{ff}, router{experts, top, scale, groups{count, keep} | null}}
    loop            {start, stop, times}: layers start .. stop-1 run ``times`` times before the rest follow (absent: every layer once)
Tensors: embed, side.embed, l<i>.{norm1,norm1b,norm2,norm2b}[.b|.alpha], l<i>.mix.*, l<i>.mlp.*, l<i>.side.{gate,proj,norm},
final.norm[.b|.alpha].

Everything is expressed with registered parts: the model below is a ``ModelSpec`` and nothing else.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Dict, List, Optional, Tuple

from ..config.base import (ConfigError, EmbedderSpec, FeedForwardSpec, LayerSpec, MixerSpec, ModelConfig, ModelSpec, NormSpec,
                           TokenSideSpec, read_key, register_architecture)

RENORM_EPS = 1e-20              # joins the sum that the chosen experts' scores are divided by

SIZES = {
    "channel_delta": ("heads", "kv_heads", "dim", "vdim", "conv"),
    "left": ("heads", "kv_heads", "dim", "vdim", "conv"),
    "right": ("width", "blocks", "conv"),
}


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


def _sizes(d: Dict[str, Any], kind: str, where: str) -> None:
    for key in SIZES[kind]:
        _keyed(lambda: read_key(d, key, int, positive=True), where)
    if "kv_heads" in SIZES[kind] and d["heads"] % d["kv_heads"]:
        raise ConfigError(f"config.json: {where}heads is not a multiple of kv_heads")


def _check_mixer(kind: str, mx: Dict[str, Any], where: str) -> None:
    if kind == "channel_delta":
        _sizes(mx, kind, where)
        _keyed(lambda: read_key(mx, "rank", int, 1, positive=True), where)
        return
    for side in ("left_scale", "right_scale"):
        _keyed(lambda: read_key(mx, side, float, 1.0), where)
    left, right = _sub(mx, "left", where), _sub(mx, "right", where)
    _sizes(left, "left", where + "left.")
    _keyed(lambda: read_key(left, "scale", float), where + "left.")
    rot = _sub(left, "rot", where + "left.", optional=True)
    if rot is not None:
        _keyed(lambda: read_key(rot, "base", float, positive=True), where + "left.rot.")
        dims = _keyed(lambda: read_key(rot, "dims", int), where + "left.rot.")
        if dims < 0 or dims % 2 or dims > left["dim"]:
            raise ConfigError(f"config.json: {where}left.rot.dims must be even and at most dim")
        sc = _sub(rot, "scaling", where + "left.rot.", optional=True)
        if sc is not None:
            for key in ("factor", "low", "high", "original"):
                _keyed(lambda: read_key(sc, key, float, positive=True), where + "left.rot.scaling.")
    _sizes(right, "right", where + "right.")
    if right["width"] % right["blocks"]:
        raise ConfigError(f"config.json: {where}right.width is not a multiple of blocks")


def _check_mlp(mlp: Dict[str, Any], where: str) -> None:
    kind = _keyed(lambda: read_key(mlp, "kind", str), where)
    if kind == "dense":
        _keyed(lambda: read_key(mlp, "ff", int, positive=True), where)
        return
    if kind != "moe":
        raise ConfigError(f"config.json: {where}kind {kind!r} is not supported (supported: 'dense', 'moe')")
    _keyed(lambda: read_key(_sub(mlp, "expert", where), "ff", int, positive=True), where + "expert.")
    router = _sub(mlp, "router", where)
    experts = _keyed(lambda: read_key(router, "experts", int, positive=True), where + "router.")
    top = _keyed(lambda: read_key(router, "top", int, positive=True), where + "router.")
    _keyed(lambda: read_key(router, "scale", float, 1.0), where + "router.")
    if top > experts:
        raise ConfigError(f"config.json: {where}router.top exceeds experts")
    groups = _sub(router, "groups", where + "router.", optional=True)
    if groups is not None:
        count = _keyed(lambda: read_key(groups, "count", int, positive=True), where + "router.groups.")
        keep = _keyed(lambda: read_key(groups, "keep", int, positive=True), where + "router.groups.")
        if experts % count or keep > count or keep * (experts // count) < top:
            raise ConfigError(f"config.json: {where}router.groups: {count} groups of which {keep} are kept do not go with {experts} experts "
                              f"and top {top}")


@dataclass(frozen=True)
class SamulornConfig(ModelConfig):
    vocab: int
    width: int
    eps: float
    embedding_scale: float
    side_dim: Optional[int]
    loop: Optional[Tuple[int, int, int]]            # start, stop, times
    layers: Tuple[Dict[str, Any], ...]              # as in config.json, checked

    architecture = "Samulorn"

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "SamulornConfig":
        vocab = read_key(d, "vocab", int, positive=True)
        width = read_key(d, "width", int, positive=True)
        eps = _keyed(lambda: read_key(_sub(d, "norm", ""), "eps", float, positive=True), "norm.")
        emb = _sub(d, "embedding", "", optional=True)
        scale = 1.0 if emb is None else _keyed(lambda: read_key(emb, "scale", float, 1.0), "embedding.")
        side = _sub(d, "token_side", "", optional=True)
        side_dim = None if side is None else _keyed(lambda: read_key(side, "dim", int, positive=True), "token_side.")
        raw = d.get("layers")
        if not isinstance(raw, list) or not raw:
            raise ConfigError("config.json: key 'layers' must be a non-empty list")
        layers: List[Dict[str, Any]] = []
        for i, ent in enumerate(raw):
            where = f"layers[{i}]."
            if not isinstance(ent, dict):
                raise ConfigError(f"config.json: layers[{i}] must be an object")
            kind = read_key(ent, "type", str)
            if kind not in ("channel_delta", "parallel"):
                raise ConfigError(f"config.json: {where}type {kind!r} is not one of ['channel_delta', 'parallel']")
            _check_mixer(kind, _sub(ent, "mixer", where), where + "mixer.")
            mlp = _sub(ent, "mlp", where, optional=True)
            if mlp is not None:
                _check_mlp(mlp, where + "mlp.")
            layers.append(copy.deepcopy(ent))
        loop = None
        lp = _sub(d, "loop", "", optional=True)
        if lp is not None:
            a = _keyed(lambda: read_key(lp, "start", int), "loop.")
            b = _keyed(lambda: read_key(lp, "stop", int), "loop.")
            times = _keyed(lambda: read_key(lp, "times", int, positive=True), "loop.")
            if not 0 <= a < b <= len(layers):
                raise ConfigError(f"config.json: loop.start and loop.stop must name a span of the {len(layers)} layers")
            loop = (a, b, times)
        return cls(vocab=vocab, width=width, eps=eps, embedding_scale=scale, side_dim=side_dim, loop=loop, layers=tuple(layers))

    def to_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps},
                             "embedding": {"scale": self.embedding_scale}, "layers": copy.deepcopy(list(self.layers))}
        if self.side_dim is not None:
            d["token_side"] = {"dim": self.side_dim}
        if self.loop is not None:
            d["loop"] = {"start": self.loop[0], "stop": self.loop[1], "times": self.loop[2]}
        return d

    def eos_token_ids(self) -> List[int]:
        return []

    # ---- the model as data ---------------------------------------------------------------------
    def _mixer(self, kind: str, mx: Dict[str, Any]) -> MixerSpec:
        if kind == "channel_delta":
            return MixerSpec("channel_delta", {
                "hidden_size": self.width, "num_heads": mx["heads"], "num_kv_heads": mx["kv_heads"], "head_dim": mx["dim"],
                "value_dim": mx["vdim"], "conv_taps": mx["conv"], "eps": self.eps, "rank": mx.get("rank")})
        left, right = mx["left"], mx["right"]
        rot, position = left.get("rot"), None
        if rot is not None and rot["dims"] > 0:
            sc = rot.get("scaling")
            scaling = None if sc is None else {"rope_type": "llama3", "factor": sc["factor"], "low_freq_factor": sc["low"],
                                               "high_freq_factor": sc["high"], "original_max_position_embeddings": sc["original"]}
            position = {"kind": "rotary", "params": {"head_dim": left["dim"], "rot_dim": rot["dims"], "theta": float(rot["base"]),
                                                     "scaling": scaling}}
        return MixerSpec("mixer_pair", {
            "hidden_size": self.width, "left_scale": float(mx.get("left_scale", 1.0)), "right_scale": float(mx.get("right_scale", 1.0)),
            "left": {"kind": "attention", "position": position, "params": {
                "hidden_size": self.width, "num_heads": left["heads"], "num_kv_heads": left["kv_heads"], "head_dim": left["dim"],
                "value_dim": left["vdim"], "scale": float(left["scale"]), "conv_taps": left["conv"], "conv_suffix": ".conv",
                "biases": True, "bias_suffix": ".b", "rot_interleaved": True, "qk_norm": {"eps": self.eps},
                "names": {"q": "q", "k": "k", "v": "v", "o": "o"}}},
            "right": {"kind": "gated_recurrence", "position": None, "params": {
                "hidden_size": self.width, "width": right["width"], "blocks": right["blocks"], "conv_taps": right["conv"]}}})

    def _feed_forward(self, mlp: Optional[Dict[str, Any]]) -> Optional[FeedForwardSpec]:
        if mlp is None:
            return None
        if mlp["kind"] == "dense":
            return FeedForwardSpec("gated_mlp", {"hidden_size": self.width, "intermediate_size": mlp["ff"], "activation": "silu",
                                                 "names": {"gate": "gate", "up": "up", "down": "down"}})
        r = mlp["router"]
        groups = r.get("groups")
        return FeedForwardSpec("routed_mlp", {
            "hidden_size": self.width, "intermediate_size": mlp["expert"]["ff"], "experts": r["experts"], "top": r["top"],
            "scale": float(r.get("scale", 1.0)), "scores": "sigmoid", "renorm": True, "renorm_eps": RENORM_EPS, "activation": "silu_glu",
            "choice_bias": "correction", "groups": None if groups is None else {"count": groups["count"], "keep": groups["keep"]},
            "shared": None})

    def run_order(self) -> List[int]:
        n = len(self.layers)
        if self.loop is None:
            return list(range(n))
        a, b, times = self.loop
        return list(range(a)) + list(range(a, b)) * times + list(range(b, n))

    def model_spec(self) -> ModelSpec:
        norm = NormSpec("dynamic_tanh", {"size": self.width, "weight_name": "", "bias_name": ".b", "alpha_name": ".alpha"})
        specs: List[LayerSpec] = []
        for i, ent in enumerate(self.layers):
            ffn = self._feed_forward(ent.get("mlp"))
            specs.append(LayerSpec(
                mixer=self._mixer(ent["type"], ent["mixer"]), feed_forward=ffn, mixer_norm=norm,
                feed_forward_norm=None if ffn is None else norm, weight_prefix=f"l{i}.", arrangement="sandwich", mixer_prefix="mix.",
                feed_forward_prefix="mlp.", mixer_norm_name="norm1", feed_forward_norm_name="norm2", mixer_post_norm=norm,
                feed_forward_post_norm=None if ffn is None else norm, mixer_post_norm_name="norm1b", feed_forward_post_norm_name="norm2b",
                token_side_prefix=None if self.side_dim is None else "side."))
        return ModelSpec(hidden_size=self.width, vocab_size=self.vocab, layers=specs, order=self.run_order(), final_norm=norm,
                         tie_word_embeddings=True, embed_name="embed", final_norm_name="final.norm", lm_head_name="head", max_position=0,
                         embedder=EmbedderSpec("table", {"scale": self.embedding_scale}),
                         token_side=None if self.side_dim is None else TokenSideSpec(self.side_dim, self.eps, "side.embed"))


register_architecture(SamulornConfig.architecture, SamulornConfig)
