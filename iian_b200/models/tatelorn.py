"""Tatelorn: typed configuration, layer description and tensor names.

A decoder-only model whose layers normalise what they ADD and read the stream as it is: ``x += n1(mixer(x))``, ``x += n2(ff(x))``
(``iian_b200/parts/block.py: sandwich_residual`` with the ``identity`` norm in front of the sub-layers).  The stream starts as the
token's row times ``embedding.scale`` plus a learned row per position, normalised; the logits are the embedding table times the
normalised stream times ``logit_scale``.  Every norm of the model is an RMS norm whose stored weight sits around zero.
``config.json`` lists the layers one by one (``layers``: ``type`` names the mixer, ``mixer`` its sizes, ``mlp`` the feed-forward or
null) besides a few model-wide values (``vocab``, ``width``, ``max_positions``, ``norm.eps``).  Per layer:

* mixer ``attention``: no rotation; q and k normalised per head with a weight, scores through a tanh cap, a fixed sink of score 0 in
  the softmax's denominator, values that take a share of the first mixing layer's (``v_mix``)
  (``iian_b200/parts/window_attention.py``);
* feed-forward ``dense`` (gated, relu) or ``moe``: experts with the clamped activation, the largest router logits chosen and weighed
  by the softmax over the chosen ones, plus an expert of its own limit that every token uses, times a sigmoid per token
  (``iian_b200/parts/experts.py``).

A position beyond the table of learned positions does not exist: requests longer than ``max_positions`` are refused.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Mapping, Optional, Tuple

from ..config.registry import Architecture, register_architecture
from ..config.spec import LayerCall, LayerSpec, ModelSpec, PartSpec
from .galodra import _get
from .qwen3 import ConfigError

SINK = 0.0                      # the score of the sink, fixed by the design


@dataclass(frozen=True)
class CappedAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: Optional[float]
    v_mix: bool


@dataclass(frozen=True)
class TatelornFeedForwardConfig:
    kind: str                      # "moe" | "dense"
    ff: int                        # of one expert for "moe"
    limit: float = 0.0             # of the experts' activation
    experts: int = 0
    top: int = 0
    shared_ff: int = 0             # 0: no expert that every token uses
    shared_limit: float = 0.0


@dataclass(frozen=True)
class TatelornLayerConfig:
    type: str                      # "attention"
    mixer: CappedAttentionConfig
    mlp: Optional[TatelornFeedForwardConfig]


@dataclass(frozen=True)
class TatelornConfig:
    vocab: int
    width: int
    max_positions: int
    norm_eps: float
    embedding_scale: float
    logit_scale: float
    layers: Tuple[TatelornLayerConfig, ...]
    eos_token_ids: Tuple[int, ...] = ()

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def hidden_size(self) -> int:
        return self.width

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    def value_mix(self, i: int) -> Optional[str]:
        """What layer ``i`` does about mixed values: nothing, leave its own to later layers, or take a share of them."""
        if not self.layers[i].mixer.v_mix:
            return None
        return "later" if any(lc.mixer.v_mix for lc in self.layers[:i]) else "first"


def _mixer_from_dict(kind: Any, raw: Mapping[str, Any], where: str) -> CappedAttentionConfig:
    if kind != "attention":
        raise ConfigError(f"config.json: {where} has unknown type {kind!r} (attention)")
    heads, kv_heads = _get(raw, "heads", int, where), _get(raw, "kv_heads", int, where)
    if heads % kv_heads:
        raise ConfigError(f"config.json: {where} has {heads} heads for {kv_heads} key/value heads")
    cap = _get(raw, "softcap", float, where, optional=True)
    if cap is not None and cap <= 0:
        raise ConfigError(f"config.json: {where} softcap must be positive, got {cap}")
    scale = _get(raw, "scale", float, where)
    if scale <= 0:
        raise ConfigError(f"config.json: {where} scale must be positive, got {scale}")
    mix = raw.get("v_mix")
    if mix is not None and not isinstance(mix, bool):
        raise ConfigError(f"config.json: {where} 'v_mix' must be true or false, got {mix!r}")
    return CappedAttentionConfig(heads=heads, kv_heads=kv_heads, dim=_get(raw, "dim", int, where), vdim=_get(raw, "vdim", int, where),
                                 scale=scale, softcap=cap, v_mix=bool(mix))


def _limit(raw: Mapping[str, Any], where: str) -> float:
    limit = _get(raw, "limit", float, where)
    if limit <= 0:
        raise ConfigError(f"config.json: {where} limit must be positive, got {limit}")
    return limit


def _mlp_from_dict(raw: Optional[Mapping[str, Any]], where: str) -> Optional[TatelornFeedForwardConfig]:
    if raw is None:
        return None
    kind = raw.get("kind") if isinstance(raw, Mapping) else None
    if kind == "dense":
        return TatelornFeedForwardConfig("dense", _get(raw, "ff", int, where))
    if kind == "moe":
        expert, router = _get(raw, "expert", dict, where), _get(raw, "router", dict, where)
        experts, top = _get(router, "experts", int, where + " router"), _get(router, "top", int, where + " router")
        if top > experts:
            raise ConfigError(f"config.json: {where} router takes {top} of {experts} experts")
        ew, sw = where + " expert", where + " shared"
        shared = raw.get("shared")
        return TatelornFeedForwardConfig("moe", _get(expert, "ff", int, ew), _limit(expert, ew), experts, top,
                                         _get(shared, "ff", int, sw) if shared is not None else 0,
                                         _limit(shared, sw) if shared is not None else 0.0)
    raise ConfigError(f"config.json: {where} has unknown kind {kind!r} (moe, dense)")


def tatelorn_config_from_dict(raw: Mapping[str, Any]) -> TatelornConfig:
    layers_raw = raw.get("layers")
    if not isinstance(layers_raw, list) or not layers_raw:
        raise ConfigError("config.json: 'layers' must be a non-empty list")
    layers = []
    first = None
    for i, lr in enumerate(layers_raw):
        where = f"layer {i}"
        kind = lr.get("type") if isinstance(lr, Mapping) else None
        mixer = _mixer_from_dict(kind, _get(lr, "mixer", dict, where) if isinstance(lr, Mapping) else {}, where + " mixer")
        if mixer.v_mix:
            if first is None:
                first = (i, mixer)
            elif (mixer.kv_heads, mixer.vdim) != (first[1].kv_heads, first[1].vdim):
                raise ConfigError(f"config.json: {where} mixes its values with those of layer {first[0]}, which have other sizes")
        layers.append(TatelornLayerConfig(kind, mixer, _mlp_from_dict(lr.get("mlp"), where + " mlp")))
    norm = _get(raw, "norm", dict, "the model")
    emb = raw.get("embedding")
    scale = _get(emb, "scale", float, "embedding", optional=True) if emb is not None else None
    logit_scale = _get(raw, "logit_scale", float, "the model", optional=True)
    eos = raw.get("eos_token_id")
    eos_ids = () if eos is None else (eos,) if isinstance(eos, int) else tuple(eos)
    return TatelornConfig(vocab=_get(raw, "vocab", int, "the model"), width=_get(raw, "width", int, "the model"),
                          max_positions=_get(raw, "max_positions", int, "the model"), norm_eps=_get(norm, "eps", float, "norm"),
                          embedding_scale=1.0 if scale is None else scale, logit_scale=1.0 if logit_scale is None else logit_scale,
                          layers=tuple(layers), eos_token_ids=eos_ids)


@register_architecture
class Tatelorn(Architecture):
    name = "Tatelorn"
    reads_tensor_shapes = True

    def with_tensor_sizes(self, raw: Mapping[str, Any], shapes: Mapping[str, Tuple[int, ...]]) -> Dict[str, Any]:
        """``raw`` completed with the number of learned positions where it is not stated: the rows of ``pos``."""
        out = dict(raw)
        shape = shapes.get("pos")
        if out.get("max_positions") is None and shape is not None and len(shape) == 2:
            out["max_positions"] = int(shape[0])
        return out

    def load_config(self, raw: Mapping[str, Any]) -> TatelornConfig:
        return tatelorn_config_from_dict(raw)

    def config_to_dict(self, c: TatelornConfig) -> Dict[str, Any]:
        layers = []
        for lc in c.layers:
            m, f = lc.mixer, lc.mlp
            mixer: Dict[str, Any] = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale,
                                     "v_mix": m.v_mix}
            if m.softcap is not None:
                mixer["softcap"] = m.softcap
            mlp: Optional[Dict[str, Any]] = None
            if f is not None and f.kind == "dense":
                mlp = {"kind": "dense", "ff": f.ff}
            elif f is not None:
                mlp = {"kind": "moe", "expert": {"ff": f.ff, "limit": f.limit}, "router": {"experts": f.experts, "top": f.top}}
                if f.shared_ff:
                    mlp["shared"] = {"ff": f.shared_ff, "limit": f.shared_limit}
            layers.append({"type": lc.type, "mixer": mixer, "mlp": mlp})
        d: Dict[str, Any] = {"architecture": self.name, "vocab": c.vocab, "width": c.width, "max_positions": c.max_positions,
                             "norm": {"eps": c.norm_eps}, "embedding": {"scale": c.embedding_scale}, "logit_scale": c.logit_scale,
                             "layers": layers}
        if c.eos_token_ids:
            d["eos_token_id"] = list(c.eos_token_ids)
        return d

    def build_spec(self, c: TatelornConfig) -> ModelSpec:
        norm = PartSpec("rms_norm", {"size": c.width, "eps": c.norm_eps, "weight_offset": 1.0})
        stream = PartSpec("identity")
        layers = []
        for i, lc in enumerate(c.layers):
            m, f = lc.mixer, lc.mlp
            mixer = PartSpec("window_attention", {
                "hidden_size": c.width, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "head_dim": m.dim, "v_dim": m.vdim,
                "scale": m.scale, "softcap": m.softcap, "sink_value": SINK, "head_norm": True, "head_norm_eps": c.norm_eps,
                "value_mix": c.value_mix(i)})
            ffn, extra = None, [("mixer_post_norm", norm)]
            if f is not None:
                if f.kind == "dense":
                    ffn = PartSpec("gated_mlp", {"hidden_size": c.width, "intermediate_size": f.ff, "activation": "relu",
                                                 "names": ("gate", "up", "down")})
                else:
                    ffn = PartSpec("routed_experts", {
                        "hidden_size": c.width, "num_experts": f.experts, "top": f.top, "intermediate_size": f.ff,
                        "activation": "clamped_swish", "limit": f.limit, "score": "softmax_top", "router_bias": False,
                        "weight_on": "output", "shared_intermediate_size": f.shared_ff, "shared_limit": f.shared_limit,
                        "shared_gate": True})
                extra.append(("feed_forward_post_norm", norm))
            layers.append(LayerSpec(mixer=mixer, feed_forward=ffn, mixer_norm=stream, feed_forward_norm=stream if ffn is not None else None,
                                    arrangement="sandwich_residual", extra=tuple(extra)))
        return ModelSpec(
            hidden_size=c.width, vocab_size=c.vocab, max_position=c.max_positions,
            embedding=PartSpec("token_embedding", {"vocab_size": c.vocab, "hidden_size": c.width, "scale": c.embedding_scale,
                                                   "positions": c.max_positions, "norm": {"eps": c.norm_eps, "weight_offset": 1.0}}),
            layers=tuple(layers), order=tuple(LayerCall(layer=i, cache=i) for i in range(len(layers))), final_norm=norm,
            head=PartSpec("lm_head", {"hidden_size": c.width, "vocab_size": c.vocab, "tied": True, "scale": c.logit_scale}))

    EMBEDDING = {"weight": "embed", "positions": "pos", "norm": "embed.norm"}
    SLOTS = {"mixer_post_norm": "norm1", "feed_forward_post_norm": "norm2"}

    def tensor_name(self, scope: tuple, local: str) -> str:
        if scope[0] == "embedding":
            return self.EMBEDDING[local]
        if scope[0] == "final_norm":
            return "final.norm"
        if scope[0] == "layer":
            i, slot = scope[1], scope[2]
            if slot == "mixer":
                return f"l{i}.mix.{local}"
            if slot == "feed_forward":
                return f"l{i}.mlp.{local}"
            if slot in self.SLOTS:
                return f"l{i}.{self.SLOTS[slot]}"
        raise KeyError(scope)
