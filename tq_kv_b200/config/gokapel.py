"""Typed configuration of the Gokapel decoder and the builder that turns it
into a `ModelSpec` of parts.

A Gokapel config.json names its architecture with the key `architecture`, its
sizes with `vocab` and `width`, the number of residual streams with `streams`,
a factor on everything a sublayer writes with `residual_mult`, a factor on the
embedding's rows with `embedding.scale`, the eps of the RMS norms inside the
mixers with `norm.eps`, and lists its layers one by one: every layer gives its
`type` (which mixer it has), the mixer's sizes and constants under `mixer`, and
its feed-forward under `mlp` (null: the layer has only the mixer).  Layers of
different types may follow one another in any order.  A layer with
`weights_of: j` runs layer j once more, with its tensors and a cache or state
of its own.

A sublayer reads and writes the streams (parts/residual_streams.py) through a
norm without statistics (Dynamic Tanh); its result is multiplied by a vector
(`ls1`, `ls2`) and by a sigmoid gate of what it read (`rg1`, `rg2`).

Mixers:
  channel_delta   parts/channel_delta.py: a matrix memory per head, updated by the delta
                  rule with a decay per head and key channel
  parallel        parts/side_by_side.py: two mixers on the same input, their results added
                  with a factor each.  left: grouped softmax attention
                  (parts/softmax_attention.py) with q and k normed per head, rotated in
                  neighbouring pairs, in chunks of `mask.size` positions, with a learned sink
                  per head; right: minGRU (parts/min_gru.py)
Feed-forward:
  dense           W_down max(W_up x, 0)^2
  moe             parts/routed_experts.py with `routing: "group_router"`: softmax scores, a
                  correction that enters the choice only, `router.groups.keep` of
                  `router.groups.count` groups, the chosen experts' scores as weights;
                  experts of the dense form; a shared expert (`shared.ff`) for every token

The head is the embedding table.  Positions have no limit by design;
`max_positions` (optional, default 32,768) bounds the cache an engine plans for.
The inner widths of a channel_delta mixer's two-step projections are the
tensors' own; random weights need them given (optional keys `decay_rank` and
`gate_rank` of the mixer).
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Optional

from .model_spec import ConfigError, LayerSpec, ModelSpec, PartSpec, ScheduleEntry
from .pavisun import RotationConfig
from .zodosun import _need, _optional_int, _positive

ARCHITECTURE = "Gokapel"
MODEL_TYPE = "gokapel"
DEFAULT_MAX_POSITIONS = 32768
UNIT_EPS = 1e-6                  # fixed by the design: q and k of the delta rule are x / sqrt(sum(x^2) + this)

_MIXERS = ("channel_delta", "parallel")


@dataclass(frozen=True)
class ChannelDeltaConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int
    decay_rank: Optional[int] = None
    gate_rank: Optional[int] = None

    @classmethod
    def from_dict(cls, d: dict, where: str) -> "ChannelDeltaConfig":
        c = cls(heads=_need(d, "heads", int, where), kv_heads=_need(d, "kv_heads", int, where),
                dim=_need(d, "dim", int, where), vdim=_need(d, "vdim", int, where), conv=_need(d, "conv", int, where),
                decay_rank=_optional_int(d, "decay_rank", where), gate_rank=_optional_int(d, "gate_rank", where))
        _positive(where, heads=c.heads, kv_heads=c.kv_heads, dim=c.dim, vdim=c.vdim, conv=c.conv)
        if c.heads % c.kv_heads:
            raise ConfigError(f"config.json: {where}: {c.heads} heads cannot share {c.kv_heads} key heads")
        return c

    def to_dict(self) -> dict:
        d: dict[str, Any] = {"conv": self.conv, "dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads,
                             "vdim": self.vdim}
        if self.decay_rank is not None:
            d["decay_rank"] = self.decay_rank
        if self.gate_rank is not None:
            d["gate_rank"] = self.gate_rank
        return d


@dataclass(frozen=True)
class AttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: RotationConfig
    chunk: Optional[int] = None

    @classmethod
    def from_dict(cls, d: dict, where: str) -> "AttentionConfig":
        c = cls(heads=_need(d, "heads", int, where), kv_heads=_need(d, "kv_heads", int, where),
                dim=_need(d, "dim", int, where), vdim=_need(d, "vdim", int, where), scale=_need(d, "scale", float, where),
                rot=RotationConfig.from_dict(_need(d, "rot", dict, where), where + ".rot"),
                chunk=_optional_int(d.get("mask") or {}, "size", where + ".mask"))
        _positive(where, heads=c.heads, kv_heads=c.kv_heads, dim=c.dim, vdim=c.vdim)
        if c.heads % c.kv_heads:
            raise ConfigError(f"config.json: {where}: {c.heads} heads cannot share {c.kv_heads} key/value heads")
        if c.rot.dims > c.dim:
            raise ConfigError(f"config.json: {where}: rot.dims {c.rot.dims} exceeds the head's {c.dim} entries")
        if c.rot.scaling is not None:
            raise ConfigError(f"config.json: {where}: rot.scaling is not part of this design")
        return c

    def to_dict(self) -> dict:
        d: dict[str, Any] = {"dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads, "rot": self.rot.to_dict(),
                             "scale": self.scale, "vdim": self.vdim}
        if self.chunk is not None:
            d["mask"] = {"size": self.chunk}
        return d


@dataclass(frozen=True)
class ParallelConfig:
    left: AttentionConfig
    left_scale: float
    right_width: int
    right_scale: float

    @classmethod
    def from_dict(cls, d: dict, where: str) -> "ParallelConfig":
        right = _need(d, "right", dict, where)
        c = cls(left=AttentionConfig.from_dict(_need(d, "left", dict, where), where + ".left"),
                left_scale=_need(d, "left_scale", float, where),
                right_width=_need(right, "width", int, where + ".right"),
                right_scale=_need(d, "right_scale", float, where))
        _positive(where + ".right", width=c.right_width)
        return c

    def to_dict(self) -> dict:
        return {"left": self.left.to_dict(), "left_scale": self.left_scale, "right": {"width": self.right_width},
                "right_scale": self.right_scale}


@dataclass(frozen=True)
class FeedForwardConfig:
    """`kind` dense: `ff`.  `kind` moe: `ff` is an expert's inner width, with `experts`, `top`, the groups and the
    shared expert's inner width `shared_ff` (0: none)."""
    kind: str
    ff: int
    experts: int = 0
    top: int = 0
    groups: int = 1
    keep: int = 1
    shared_ff: int = 0

    @classmethod
    def from_dict(cls, d: dict, where: str) -> "FeedForwardConfig":
        kind = _need(d, "kind", str, where)
        if kind == "dense":
            c = cls(kind, _need(d, "ff", int, where))
            _positive(where, ff=c.ff)
            return c
        if kind != "moe":
            raise ConfigError(f"config.json: {where}: unknown kind '{kind}' (known: dense, moe)")
        router = _need(d, "router", dict, where)
        w = where + ".router"
        groups, shared = router.get("groups"), d.get("shared")
        c = cls(kind, _need(_need(d, "expert", dict, where), "ff", int, where + ".expert"),
                experts=_need(router, "experts", int, w), top=_need(router, "top", int, w),
                groups=1 if groups is None else _need(groups, "count", int, w + ".groups"),
                keep=1 if groups is None else _need(groups, "keep", int, w + ".groups"),
                shared_ff=0 if shared is None else _need(shared, "ff", int, where + ".shared"))
        _positive(where, ff=c.ff, experts=c.experts, top=c.top, count=c.groups, keep=c.keep)
        if c.experts % c.groups or c.keep > c.groups:
            raise ConfigError(f"config.json: {w}: {c.experts} experts in {c.groups} equal groups of which {c.keep} are kept")
        if c.top > c.keep * (c.experts // c.groups):
            raise ConfigError(f"config.json: {w}: a token cannot use {c.top} experts of {c.keep} groups of {c.experts // c.groups}")
        if shared is not None:
            _positive(where + ".shared", ff=c.shared_ff)
        return c

    def to_dict(self) -> dict:
        if self.kind == "dense":
            return {"ff": self.ff, "kind": "dense"}
        d: dict[str, Any] = {"expert": {"ff": self.ff}, "kind": "moe",
                             "router": {"experts": self.experts, "groups": {"count": self.groups, "keep": self.keep},
                                        "top": self.top}}
        if self.shared_ff:
            d["shared"] = {"ff": self.shared_ff}
        return d


_MIXER_CONFIGS = {"channel_delta": ChannelDeltaConfig, "parallel": ParallelConfig}


@dataclass(frozen=True)
class GokapelLayer:
    type: str
    mixer: Any
    mlp: Optional[FeedForwardConfig]
    weights_of: Optional[int] = None

    @classmethod
    def from_dict(cls, d: dict, index: int) -> "GokapelLayer":
        where = f"layers[{index}]"
        typ = _need(d, "type", str, where)
        if typ not in _MIXERS:
            raise ConfigError(f"config.json: {where}: unknown layer type '{typ}' (known: {sorted(_MIXERS)})")
        mixer = _MIXER_CONFIGS[typ].from_dict(_need(d, "mixer", dict, where), where + ".mixer")
        mlp = d.get("mlp")
        return cls(typ, mixer, None if mlp is None else FeedForwardConfig.from_dict(mlp, where + ".mlp"),
                   None if d.get("weights_of") is None else _need(d, "weights_of", int, where))

    def to_dict(self) -> dict:
        d = {"mixer": self.mixer.to_dict(), "mlp": None if self.mlp is None else self.mlp.to_dict(), "type": self.type}
        if self.weights_of is not None:
            d["weights_of"] = self.weights_of
        return d


@dataclass(frozen=True)
class GokapelConfig:
    vocab: int
    width: int
    norm_eps: float
    streams: int
    residual_mult: float
    embedding_scale: float
    layers: tuple[GokapelLayer, ...]
    max_positions: int = DEFAULT_MAX_POSITIONS
    torch_dtype: str = "bfloat16"
    stop_token_ids: tuple[int, ...] = field(default_factory=tuple)

    @classmethod
    def from_dict(cls, d: dict[str, Any]) -> "GokapelConfig":
        top = "the top level"
        layers = _need(d, "layers", list, top)
        if not layers:
            raise ConfigError("config.json: 'layers' is empty")
        cfg = cls(
            vocab=_need(d, "vocab", int, top),
            width=_need(d, "width", int, top),
            norm_eps=_need(_need(d, "norm", dict, top), "eps", float, "norm"),
            streams=_need(d, "streams", int, top),
            residual_mult=_need(d, "residual_mult", float, top),
            embedding_scale=_need(_need(d, "embedding", dict, top), "scale", float, "embedding"),
            layers=tuple(GokapelLayer.from_dict(l, i) for i, l in enumerate(layers)),
            max_positions=_optional_int(d, "max_positions", top) or DEFAULT_MAX_POSITIONS,
            torch_dtype=d.get("torch_dtype") or "bfloat16",
            stop_token_ids=tuple(int(t) for t in (d.get("stop_token_ids") or ())),
        )
        _positive(top, vocab=cfg.vocab, width=cfg.width, streams=cfg.streams)
        if not cfg.norm_eps > 0.0:
            raise ConfigError("config.json: norm.eps must be positive")
        for i, layer in enumerate(cfg.layers):
            j = layer.weights_of
            if j is None:
                continue
            if not 0 <= j < len(cfg.layers) or cfg.layers[j].weights_of is not None:
                raise ConfigError(f"config.json: layers[{i}]: weights_of {j} must name a layer with tensors of its own")
            o = cfg.layers[j]
            if (o.type, o.mixer, o.mlp) != (layer.type, layer.mixer, layer.mlp):
                raise ConfigError(f"config.json: layers[{i}] uses the tensors of layer {j} and must be like it")
        return cfg

    def to_dict(self) -> dict[str, Any]:
        d: dict[str, Any] = {
            "architecture": ARCHITECTURE,
            "embedding": {"scale": self.embedding_scale},
            "layers": [l.to_dict() for l in self.layers],
            "norm": {"eps": self.norm_eps},
            "residual_mult": self.residual_mult,
            "streams": self.streams,
            "vocab": self.vocab,
            "width": self.width,
            "torch_dtype": self.torch_dtype,
        }
        if self.max_positions != DEFAULT_MAX_POSITIONS:
            d["max_positions"] = self.max_positions
        if self.stop_token_ids:
            d["stop_token_ids"] = list(self.stop_token_ids)
        return d


def _mixer(cfg: GokapelConfig, layer: GokapelLayer, prefix: str) -> PartSpec:
    m = layer.mixer
    if layer.type == "channel_delta":
        return PartSpec("channel_delta_mixer", {
            "hidden_size": cfg.width, "heads": m.heads, "key_heads": m.kv_heads, "key_dim": m.dim, "value_dim": m.vdim,
            "taps": m.conv, "decay_rank": m.decay_rank, "gate_rank": m.gate_rank, "eps": cfg.norm_eps,
            "unit_eps": UNIT_EPS, "query_scale": m.dim ** -0.5,
            "names": {"q": "q", "k": "k", "v": "v", "q_conv": "q.conv", "k_conv": "k.conv", "v_conv": "v.conv",
                      "beta": "b", "a_log": "A_log", "decay_in": "a1", "decay_out": "a2", "dt_bias": "dt_bias",
                      "gate_in": "g1", "gate_out": "g2", "norm": "norm", "out": "o"}}, prefix)
    a = m.left
    left = PartSpec("softmax_attention", {
        "hidden_size": cfg.width, "num_heads": a.heads, "num_kv_heads": a.kv_heads, "key_dim": a.dim, "value_dim": a.vdim,
        "scale": a.scale, "values": "projected", "chunk": a.chunk, "qk_norm_eps": cfg.norm_eps, "qk_norm_weights": True,
        "sink": "learned", "result_scale": m.left_scale,
        "position": PartSpec("rotary_tables", {"rotary_dim": a.rot.dims, "theta": a.rot.base, "layout": "pairs"}),
        "names": {"q": "q", "k": "k", "v": "v", "out": "o", "q_norm": "q.norm", "k_norm": "k.norm", "sink": "sink"}},
        prefix + "left.")
    right = PartSpec("min_gru_mixer", {
        "hidden_size": cfg.width, "width": m.right_width, "result_scale": m.right_scale,
        "names": {"update": "z", "update_bias": "z.b", "candidate": "x", "candidate_bias": "x.b", "gate": "g",
                  "out": "o"}}, prefix + "right.")
    return PartSpec("side_by_side", {"width": cfg.width, "branches": [{"part": left}, {"part": right}]}, prefix)


def _feed_forward(cfg: GokapelConfig, f: FeedForwardConfig, prefix: str) -> PartSpec:
    if f.kind == "dense":
        return PartSpec("plain_feed_forward", {"hidden_size": cfg.width, "intermediate_size": f.ff,
                                               "activation": "square_relu", "names": {"up": "up", "down": "down"}}, prefix)
    return PartSpec("routed_experts", {
        "hidden_size": cfg.width, "intermediate_size": f.ff, "experts": f.experts, "top": f.top,
        "routing": "group_router", "gated": False, "groups": f.groups, "keep_groups": f.keep, "shared_size": f.shared_ff,
        "names": {"expert": "e{}.", "up": "up", "down": "down", "router": "router", "correction": "correction",
                  "shared": "shared."}}, prefix)


def build_gokapel_spec(cfg: GokapelConfig) -> ModelSpec:
    """Gokapel as parts: scaled token embedding; per layer a block on residual streams of {Dynamic Tanh norm, mixer,
    Dynamic Tanh norm, feed-forward} whose results are scaled and gated; a layer with `weights_of` is one more entry
    of the schedule that names that layer; Dynamic Tanh norm; the embedding table as head."""
    def norm(name: str) -> PartSpec:
        return PartSpec("dynamic_tanh_norm", {"width": cfg.width, "weight_name": name})

    def connection(prefix: str) -> PartSpec:
        return PartSpec("stream_connection", {"streams": cfg.streams, "residual_mult": cfg.residual_mult,
                                              "names": {"read": "in", "write": "out", "mix": "mix"}}, prefix)

    def result(prefix: str, q: int) -> PartSpec:
        return PartSpec("sublayer_result", {"width": cfg.width, "names": {"scale": f"ls{q}", "gate": f"rg{q}",
                                                                           "gate_bias": f"rg{q}.b"}}, prefix)

    layers, schedule = [], []
    own: dict[int, int] = {}                        # layer of the file -> layer of the spec
    for i, layer in enumerate(cfg.layers):
        if layer.weights_of is not None:
            continue
        p = f"l{i}."
        own[i] = len(layers)
        extra = {"mixer_streams": connection(p + "hc1."), "mixer_result": result(p, 1)}
        ffn = ffn_norm = None
        if layer.mlp is not None:
            ffn, ffn_norm = _feed_forward(cfg, layer.mlp, p + "mlp."), norm(p + "norm2")
            extra.update(feed_forward_streams=connection(p + "hc2."), feed_forward_result=result(p, 2))
        layers.append(LayerSpec(block="residual_streams", mixer=_mixer(cfg, layer, p + "mix."), feed_forward=ffn,
                                mixer_norm=norm(p + "norm1"), feed_forward_norm=ffn_norm, extra_parts=extra))
    for i, layer in enumerate(cfg.layers):
        schedule.append(ScheduleEntry(own[i if layer.weights_of is None else layer.weights_of]))
    spec = ModelSpec(
        architecture=ARCHITECTURE,
        vocab_size=cfg.vocab,
        hidden_size=cfg.width,
        max_positions=cfg.max_positions,
        embedding=PartSpec("token_embedding", {"vocab_size": cfg.vocab, "width": cfg.width, "weight_name": "embed",
                                               "scale": cfg.embedding_scale}),
        layers=tuple(layers),
        schedule=tuple(schedule),
        final_norm=norm("final.norm"),
        head=PartSpec("lm_head", {"vocab_size": cfg.vocab, "width": cfg.width, "tied_to": "embed"}),
        stop_token_ids=cfg.stop_token_ids,
        residual_streams=cfg.streams,
    )
    spec.validate()
    return spec
