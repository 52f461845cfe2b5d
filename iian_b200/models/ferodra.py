"""Ferodra: typed configuration, layer description and tensor names.

A decoder-only model whose layers put a norm before AND after each sub-layer and a learned factor per column behind the second
one: ``x += c1 * n1b(mixer(n1 x))``, ``x += c2 * n2b(ff(n2 x))`` (``iian_b200/parts/block.py: sandwich_residual``); every norm is
``w tanh(alpha x) + b`` (``parts/norm.py: dynamic_tanh``).  ``config.json`` lists the layers one by one (``layers``: ``type`` names
the mixer, ``mixer`` its sizes, ``mlp`` the feed-forward or null) besides a few model-wide values (``vocab``, ``width``,
``norm.eps``, which only the mixers' inner norms use, ``loop``).  Per layer:

* mixer ``attention``: every head is the difference of two softmax maps over the same values, scores through a tanh cap,
  interleaved rotation with frequencies rescaled by a ramp (``parts/difference_attention.py``);
* mixer ``delta``: the gated delta rule with one decay per head, short convolutions in front, a full silu gate
  (``parts/delta_rule.py``);
* feed-forward ``dense`` (gated, silu) or ``moe``: experts without a gate (squared relu) chosen by softmax plus a correction only
  the choice sees, some of the router's outputs passing their input on, plus a gated shared expert (``parts/experts.py``).

``loop`` makes the layers ``start .. stop - 1`` run ``times`` times in a row with the same weights; every run has caches and
states of its own and begins with ``x <- x + step_t``, a learned vector per run (``parts/stream.py: add_turn_vector``).  The output
is the model's norm and the embedding table as the head.  Positions have no stated limit.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Mapping, Optional, Tuple

from ..config.registry import Architecture, register_architecture
from ..config.spec import LayerCall, LayerSpec, ModelSpec, PartSpec
from .galodra import _get
from .lekilix import LoopConfig
from .nogelorn import RAMP_KEYS, RotationConfig, _rotation_from_dict, _rotation_to_dict
from .qwen3 import ConfigError

MAX_POSITION = 1 << 24          # the design states no limit; angles are float64 products


@dataclass(frozen=True)
class DifferenceAttentionConfig:
    heads: int
    kv_heads: int
    dim: int                       # of one map
    vdim: int
    scale: float
    diff: float
    softcap: Optional[float]
    rot: Optional[RotationConfig]


@dataclass(frozen=True)
class HeadDecayDeltaConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int


@dataclass(frozen=True)
class FerodraFeedForwardConfig:
    kind: str                      # "moe" | "dense"
    ff: int                        # of one expert for "moe"
    experts: int = 0
    identity: int = 0              # router outputs behind the experts that pass their input on
    top: int = 0
    scale: float = 1.0
    shared_ff: int = 0             # 0: no expert that every token uses


@dataclass(frozen=True)
class FerodraLayerConfig:
    type: str                      # "attention" | "delta"
    mixer: object
    mlp: Optional[FerodraFeedForwardConfig]


@dataclass(frozen=True)
class FerodraConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: Tuple[FerodraLayerConfig, ...]
    loop: Optional[LoopConfig] = None
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

    def run_order(self) -> Tuple[Tuple[int, Optional[int]], ...]:
        """(layer, number of the looped stretch's run that starts here, or None) in the order the layers run."""
        n = len(self.layers)
        if self.loop is None:
            return tuple((i, None) for i in range(n))
        lp = self.loop
        order = [(i, None) for i in range(lp.start)]
        for t in range(lp.times):
            order += [(i, t if i == lp.start else None) for i in range(lp.start, lp.stop)]
        order += [(i, None) for i in range(lp.stop, n)]
        return tuple(order)


def _non_negative(raw: Mapping[str, Any], key: str, where: str, default: Optional[int] = None) -> int:
    v = raw.get(key, default)
    if v is None and default is not None:
        v = default
    if isinstance(v, bool) or not isinstance(v, int) or v < 0:
        raise ConfigError(f"config.json: {where} '{key}' must be a non-negative integer, got {v!r}")
    return v


def _mixer_from_dict(kind: Any, raw: Mapping[str, Any], where: str):
    if kind not in ("attention", "delta"):
        raise ConfigError(f"config.json: {where} has unknown type {kind!r} (attention, delta)")
    heads, kv_heads = _get(raw, "heads", int, where), _get(raw, "kv_heads", int, where)
    if heads % kv_heads:
        raise ConfigError(f"config.json: {where} has {heads} heads for {kv_heads} "
                          f"{'key/value' if kind == 'attention' else 'query/key'} heads")
    dim, vdim = _get(raw, "dim", int, where), _get(raw, "vdim", int, where)
    if kind == "delta":
        return HeadDecayDeltaConfig(heads, kv_heads, dim, vdim, _get(raw, "conv", int, where))
    cap = _get(raw, "softcap", float, where, optional=True)
    if cap is not None and cap <= 0:
        raise ConfigError(f"config.json: {where} softcap must be positive, got {cap}")
    return DifferenceAttentionConfig(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=_get(raw, "scale", float, where),
                                     diff=_get(raw, "diff", float, where), softcap=cap,
                                     rot=_rotation_from_dict(raw.get("rot"), dim, where + " rot", RAMP_KEYS))


def _mlp_from_dict(raw: Optional[Mapping[str, Any]], where: str) -> Optional[FerodraFeedForwardConfig]:
    if raw is None:
        return None
    kind = raw.get("kind") if isinstance(raw, Mapping) else None
    if kind == "dense":
        return FerodraFeedForwardConfig("dense", _get(raw, "ff", int, where))
    if kind == "moe":
        expert, router = _get(raw, "expert", dict, where), _get(raw, "router", dict, where)
        rw = where + " router"
        experts, top = _get(router, "experts", int, rw), _get(router, "top", int, rw)
        identity = _non_negative(router, "identity", rw, 0)
        if top > experts + identity:
            raise ConfigError(f"config.json: {rw} takes {top} of {experts} experts and {identity} identity outputs")
        scale = _get(router, "scale", float, rw, optional=True)
        shared = raw.get("shared")
        return FerodraFeedForwardConfig("moe", _get(expert, "ff", int, where + " expert"), experts, identity, top,
                                        1.0 if scale is None else scale,
                                        _get(shared, "ff", int, where + " shared") if shared is not None else 0)
    raise ConfigError(f"config.json: {where} has unknown kind {kind!r} (moe, dense)")


def ferodra_config_from_dict(raw: Mapping[str, Any]) -> FerodraConfig:
    layers_raw = raw.get("layers")
    if not isinstance(layers_raw, list) or not layers_raw:
        raise ConfigError("config.json: 'layers' must be a non-empty list")
    layers = []
    for i, lr in enumerate(layers_raw):
        where = f"layer {i}"
        kind = lr.get("type") if isinstance(lr, Mapping) else None
        mixer_raw = _get(lr, "mixer", dict, where) if isinstance(lr, Mapping) else None
        layers.append(FerodraLayerConfig(kind, _mixer_from_dict(kind, mixer_raw, where + " mixer"),
                                         _mlp_from_dict(lr.get("mlp"), where + " mlp")))
    norm = _get(raw, "norm", dict, "the model")
    loop = None
    if raw.get("loop") is not None:
        lr = _get(raw, "loop", dict, "the model")
        start, stop, times = (_non_negative(lr, k, "loop") for k in ("start", "stop", "times"))
        if not start < stop <= len(layers) or times < 1:
            raise ConfigError(f"config.json: loop runs layers {start} .. {stop} - 1 {times} times; the model has {len(layers)} layers")
        loop = LoopConfig(start, stop, times)
    eos = raw.get("eos_token_id")
    eos_ids = () if eos is None else (eos,) if isinstance(eos, int) else tuple(eos)
    return FerodraConfig(vocab=_get(raw, "vocab", int, "the model"), width=_get(raw, "width", int, "the model"),
                         norm_eps=_get(norm, "eps", float, "norm"), layers=tuple(layers), loop=loop, eos_token_ids=eos_ids)


@register_architecture
class Ferodra(Architecture):
    name = "Ferodra"

    def load_config(self, raw: Mapping[str, Any]) -> FerodraConfig:
        return ferodra_config_from_dict(raw)

    def config_to_dict(self, c: FerodraConfig) -> Dict[str, Any]:
        layers = []
        for lc in c.layers:
            m = lc.mixer
            mixer: Dict[str, Any] = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim}
            if lc.type == "delta":
                mixer["conv"] = m.conv
            else:
                mixer["scale"], mixer["diff"] = m.scale, m.diff
                if m.softcap is not None:
                    mixer["softcap"] = m.softcap
                if m.rot is not None:
                    mixer["rot"] = _rotation_to_dict(m.rot)
            mlp: Optional[Dict[str, Any]] = None
            if lc.mlp is not None and lc.mlp.kind == "dense":
                mlp = {"kind": "dense", "ff": lc.mlp.ff}
            elif lc.mlp is not None:
                f = lc.mlp
                mlp = {"kind": "moe", "expert": {"ff": f.ff},
                       "router": {"experts": f.experts, "identity": f.identity, "scale": f.scale, "top": f.top}}
                if f.shared_ff:
                    mlp["shared"] = {"ff": f.shared_ff}
            layers.append({"type": lc.type, "mixer": mixer, "mlp": mlp})
        d: Dict[str, Any] = {"architecture": self.name, "vocab": c.vocab, "width": c.width, "norm": {"eps": c.norm_eps}, "layers": layers}
        if c.loop is not None:
            d["loop"] = {"start": c.loop.start, "stop": c.loop.stop, "times": c.loop.times}
        if c.eos_token_ids:
            d["eos_token_id"] = list(c.eos_token_ids)
        return d

    @staticmethod
    def _position(rot: Optional[RotationConfig]) -> PartSpec:
        if rot is None or not rot.dims:
            return PartSpec("none")
        params: Dict[str, Any] = {"dim": rot.dims, "base": rot.base, "style": "interleaved", "max_position": MAX_POSITION}
        if rot.scaling is None:
            return PartSpec("rotary", params)
        return PartSpec("scaled_rotary", dict(params, scaling=dict(rot.scaling, kind="ramp")))

    def build_spec(self, c: FerodraConfig) -> ModelSpec:
        norm = PartSpec("dynamic_tanh", {"size": c.width})
        scale = PartSpec("column_scale", {"size": c.width})
        layers = []
        for lc in c.layers:
            m = lc.mixer
            if lc.type == "attention":
                mixer = PartSpec("difference_attention", {
                    "hidden_size": c.width, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "head_dim": m.dim, "v_dim": m.vdim,
                    "scale": m.scale, "softcap": m.softcap, "diff": m.diff, "norm_eps": c.norm_eps, "position": self._position(m.rot)})
            else:
                mixer = PartSpec("gated_delta_rule", {
                    "hidden_size": c.width, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "dim": m.dim, "v_dim": m.vdim,
                    "conv": m.conv, "decay": "head", "gate": "full", "gate_act": "silu", "norm_eps": c.norm_eps})
            ffn, extra = None, [("mixer_post_norm", norm), ("mixer_scale", scale)]
            if lc.mlp is not None:
                f = lc.mlp
                if f.kind == "dense":
                    ffn = PartSpec("gated_mlp", {"hidden_size": c.width, "intermediate_size": f.ff, "activation": "silu",
                                                 "names": ("gate", "up", "down")})
                else:
                    ffn = PartSpec("routed_experts", {
                        "hidden_size": c.width, "num_experts": f.experts, "identity_experts": f.identity, "top": f.top,
                        "intermediate_size": f.ff, "activation": "relu2", "score": "softmax", "weight_scale": f.scale,
                        "weight_on": "output", "shared_intermediate_size": f.shared_ff, "shared_gate": True})
                extra += [("feed_forward_post_norm", norm), ("feed_forward_scale", scale)]
            layers.append(LayerSpec(mixer=mixer, feed_forward=ffn, mixer_norm=norm, feed_forward_norm=norm if ffn is not None else None,
                                    arrangement="sandwich_residual", extra=tuple(extra)))
        stream_parts = ()
        if c.loop is not None:
            stream_parts = (PartSpec("add_turn_vector", {"hidden_size": c.width, "turns": c.loop.times}),)
        order = tuple(LayerCall(layer=i, cache=idx, before=0 if t is not None else None, turn=t or 0)
                      for idx, (i, t) in enumerate(c.run_order()))                 # every run of a layer has a cache of its own
        return ModelSpec(
            hidden_size=c.width, vocab_size=c.vocab, max_position=MAX_POSITION,
            embedding=PartSpec("token_embedding", {"vocab_size": c.vocab, "hidden_size": c.width}),
            layers=tuple(layers), order=order, final_norm=norm,
            head=PartSpec("lm_head", {"hidden_size": c.width, "vocab_size": c.vocab, "tied": True}),
            stream_parts=stream_parts)

    SLOTS = {"mixer_norm": "norm1", "mixer_post_norm": "norm1b", "feed_forward_norm": "norm2", "feed_forward_post_norm": "norm2b"}
    NORM_PARTS = {"weight": "", "alpha": ".alpha", "bias": ".b"}
    SCALES = {"mixer_scale": "ls1", "feed_forward_scale": "ls2"}

    def tensor_name(self, scope: tuple, local: str) -> str:
        if scope[0] == "embedding":
            return "embed"
        if scope[0] == "stream":
            return "loop.step"
        if scope[0] == "final_norm":
            return "final.norm" + self.NORM_PARTS[local]
        if scope[0] == "layer":
            i, slot = scope[1], scope[2]
            if slot == "mixer":
                return f"l{i}.mix.{local}"
            if slot == "feed_forward":
                return f"l{i}.mlp.{local}"
            if slot in self.SLOTS:
                return f"l{i}.{self.SLOTS[slot]}{self.NORM_PARTS[local]}"
            if slot in self.SCALES:
                return f"l{i}.{self.SCALES[slot]}"
        raise KeyError(scope)
