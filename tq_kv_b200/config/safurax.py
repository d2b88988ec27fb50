"""Typed configuration of the Safurax decoder and the builder that turns it
into a `ModelSpec` of parts.

A Safurax config.json names its architecture with the key `architecture`, its
sizes with `vocab` and `width`, the norms' `eps` under `norm`, the factor on
the embedding's rows under `embedding`, and lists its layers one by one: every
layer gives its `type` (which mixer it has), the mixer's sizes and constants
under `mixer`, and its feed-forward under `mlp` (null: the layer has only the
mixer).  Layers of different types may follow one another in any order.

A layer is pre-norm, x <- x + mixer(norm1(x)); x <- x + ff(norm2(x)), with
layer norms (the mean taken off, a weight, no bias).

Mixers:
  latent_attention    parts/latent_attention.py without a rotated part: queries through a normed
                      latent of their own, keys and values from one cached latent per token,
                      all earlier positions, a plain softmax
  latent_attention_2  the same part with queries projected directly, a rotated key part that the
                      heads share (halves layout), a sliding window, a learned sink and a gate per
                      head.  With `kv_from: j` the layer has no latent of its own and reads what
                      layer j cached.
  attention           parts/softmax_attention.py as a difference of two maps per head over the same
                      values: grouped heads; q and k normed per head and map with one weight of the
                      head's width, rotated (halves layout) at rates divided by
                      `rot.scaling.factor`; a gate per head
Feed-forward:
  dense               W_down (silu(W_gate x) * (W_up x))
  moe                 parts/routed_experts.py with `routing: "softmax_router"`: the `top` largest
                      logits of W_router x + b, weighed by the softmax over them; a shared expert
                      (`shared.ff`) times sigmoid(w x) for every token

The head is a matrix of its own (`head`).  Positions have no limit by design;
`max_positions` (optional, default 32,768) bounds the cache an engine plans for.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Optional

from .model_spec import ConfigError, LayerSpec, ModelSpec, PartSpec, ScheduleEntry
from .zodosun import _need, _optional_int, _positive

ARCHITECTURE = "Safurax"
MODEL_TYPE = "safurax"
DEFAULT_MAX_POSITIONS = 32768


def _window(d: dict, where: str) -> Optional[int]:
    return _optional_int(d.get("mask") or {}, "size", where + ".mask")


@dataclass(frozen=True)
class LinearRotation:
    """Rotation of the first `dims` entries at the rates base^(-2i/dims) / factor."""
    base: float
    dims: int
    factor: float = 1.0

    @classmethod
    def from_dict(cls, d: dict, where: str) -> "LinearRotation":
        sc = d.get("scaling")
        c = cls(base=_need(d, "base", float, where), dims=_need(d, "dims", int, where),
                factor=1.0 if sc is None else _need(sc, "factor", float, where + ".scaling"))
        _positive(where, base=c.base, dims=c.dims, factor=c.factor)
        if c.dims % 2:
            raise ConfigError(f"config.json: {where}: dims {c.dims} must be even")
        return c

    def to_dict(self) -> dict:
        d: dict[str, Any] = {"base": self.base, "dims": self.dims}
        if self.factor != 1.0:
            d["scaling"] = {"factor": self.factor}
        return d

    def part(self) -> PartSpec:
        return PartSpec("rotary_tables", {"rotary_dim": self.dims, "theta": self.base, "layout": "halves",
                                          "rate_divisor": self.factor})


@dataclass(frozen=True)
class PlainLatentConfig:
    heads: int
    dim: int
    vdim: int
    kv_rank: int
    q_rank: int
    scale: float

    @classmethod
    def from_dict(cls, d: dict, where: str) -> "PlainLatentConfig":
        c = cls(heads=_need(d, "heads", int, where), dim=_need(d, "dim", int, where), vdim=_need(d, "vdim", int, where),
                kv_rank=_need(d, "kv_rank", int, where), q_rank=_need(d, "q_rank", int, where),
                scale=_need(d, "scale", float, where))
        _positive(where, heads=c.heads, dim=c.dim, vdim=c.vdim, kv_rank=c.kv_rank, q_rank=c.q_rank)
        return c

    def to_dict(self) -> dict:
        return {"dim": self.dim, "heads": self.heads, "kv_rank": self.kv_rank, "q_rank": self.q_rank, "scale": self.scale,
                "vdim": self.vdim}


@dataclass(frozen=True)
class WindowedLatentConfig:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    rot: LinearRotation
    window: Optional[int] = None
    kv_from: Optional[int] = None

    @classmethod
    def from_dict(cls, d: dict, where: str) -> "WindowedLatentConfig":
        c = cls(heads=_need(d, "heads", int, where), dim=_need(d, "dim", int, where),
                rot_dim=_need(d, "rot_dim", int, where), vdim=_need(d, "vdim", int, where),
                kv_rank=_need(d, "kv_rank", int, where), scale=_need(d, "scale", float, where),
                rot=LinearRotation.from_dict(_need(d, "rot", dict, where), where + ".rot"), window=_window(d, where),
                kv_from=None if d.get("kv_from") is None else _need(d, "kv_from", int, where))
        _positive(where, heads=c.heads, dim=c.dim, rot_dim=c.rot_dim, vdim=c.vdim, kv_rank=c.kv_rank)
        if c.rot.dims > c.rot_dim:
            raise ConfigError(f"config.json: {where}: rot.dims {c.rot.dims} exceeds the rotated part's {c.rot_dim} entries")
        return c

    def to_dict(self) -> dict:
        d: dict[str, Any] = {"dim": self.dim, "heads": self.heads, "kv_rank": self.kv_rank, "rot": self.rot.to_dict(),
                             "rot_dim": self.rot_dim, "scale": self.scale, "vdim": self.vdim}
        if self.kv_from is not None:
            d["kv_from"] = self.kv_from
        if self.window is not None:
            d["mask"] = {"size": self.window}
        return d


@dataclass(frozen=True)
class DifferenceConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    diff: float
    rot: LinearRotation

    @classmethod
    def from_dict(cls, d: dict, where: str) -> "DifferenceConfig":
        c = cls(heads=_need(d, "heads", int, where), kv_heads=_need(d, "kv_heads", int, where),
                dim=_need(d, "dim", int, where), vdim=_need(d, "vdim", int, where), scale=_need(d, "scale", float, where),
                diff=_need(d, "diff", float, where),
                rot=LinearRotation.from_dict(_need(d, "rot", dict, where), where + ".rot"))
        _positive(where, heads=c.heads, kv_heads=c.kv_heads, dim=c.dim, vdim=c.vdim)
        if c.heads % c.kv_heads:
            raise ConfigError(f"config.json: {where}: {c.heads} heads cannot share {c.kv_heads} key/value heads")
        if c.rot.dims > c.dim:
            raise ConfigError(f"config.json: {where}: rot.dims {c.rot.dims} exceeds the map's {c.dim} entries")
        return c

    def to_dict(self) -> dict:
        return {"diff": self.diff, "dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads,
                "rot": self.rot.to_dict(), "scale": self.scale, "vdim": self.vdim}


@dataclass(frozen=True)
class FeedForwardConfig:
    """`kind` dense: `ff`.  `kind` moe: `ff` is an expert's inner width, with `experts`, `top` and the shared expert's
    inner width `shared_ff` (0: none)."""
    kind: str
    ff: int
    experts: int = 0
    top: int = 0
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
        shared = d.get("shared")
        c = cls(kind, _need(_need(d, "expert", dict, where), "ff", int, where + ".expert"),
                experts=_need(router, "experts", int, where + ".router"), top=_need(router, "top", int, where + ".router"),
                shared_ff=0 if shared is None else _need(shared, "ff", int, where + ".shared"))
        _positive(where, ff=c.ff, experts=c.experts, top=c.top)
        if c.top > c.experts:
            raise ConfigError(f"config.json: {where}: a token cannot use {c.top} of {c.experts} experts")
        if shared is not None:
            _positive(where + ".shared", ff=c.shared_ff)
        return c

    def to_dict(self) -> dict:
        if self.kind == "dense":
            return {"ff": self.ff, "kind": "dense"}
        d: dict[str, Any] = {"expert": {"ff": self.ff}, "kind": "moe",
                             "router": {"experts": self.experts, "top": self.top}}
        if self.shared_ff:
            d["shared"] = {"ff": self.shared_ff}
        return d


_MIXER_CONFIGS = {"latent_attention": PlainLatentConfig, "latent_attention_2": WindowedLatentConfig,
                  "attention": DifferenceConfig}


@dataclass(frozen=True)
class SafuraxLayer:
    type: str
    mixer: Any
    mlp: Optional[FeedForwardConfig]

    @classmethod
    def from_dict(cls, d: dict, index: int) -> "SafuraxLayer":
        where = f"layers[{index}]"
        typ = _need(d, "type", str, where)
        if typ not in _MIXER_CONFIGS:
            raise ConfigError(f"config.json: {where}: unknown layer type '{typ}' (known: {sorted(_MIXER_CONFIGS)})")
        mixer = _MIXER_CONFIGS[typ].from_dict(_need(d, "mixer", dict, where), where + ".mixer")
        mlp = d.get("mlp")
        return cls(typ, mixer, None if mlp is None else FeedForwardConfig.from_dict(mlp, where + ".mlp"))

    @property
    def kv_from(self) -> Optional[int]:
        return self.mixer.kv_from if self.type == "latent_attention_2" else None

    def to_dict(self) -> dict:
        return {"mixer": self.mixer.to_dict(), "mlp": None if self.mlp is None else self.mlp.to_dict(),
                "type": self.type}


@dataclass(frozen=True)
class SafuraxConfig:
    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float
    layers: tuple[SafuraxLayer, ...]
    max_positions: int = DEFAULT_MAX_POSITIONS
    torch_dtype: str = "bfloat16"
    stop_token_ids: tuple[int, ...] = field(default_factory=tuple)

    @classmethod
    def from_dict(cls, d: dict[str, Any]) -> "SafuraxConfig":
        top = "the top level"
        layers = _need(d, "layers", list, top)
        if not layers:
            raise ConfigError("config.json: 'layers' is empty")
        cfg = cls(
            vocab=_need(d, "vocab", int, top),
            width=_need(d, "width", int, top),
            norm_eps=_need(_need(d, "norm", dict, top), "eps", float, "norm"),
            embedding_scale=_need(_need(d, "embedding", dict, top), "scale", float, "embedding"),
            layers=tuple(SafuraxLayer.from_dict(l, i) for i, l in enumerate(layers)),
            max_positions=_optional_int(d, "max_positions", top) or DEFAULT_MAX_POSITIONS,
            torch_dtype=d.get("torch_dtype") or "bfloat16",
            stop_token_ids=tuple(int(t) for t in (d.get("stop_token_ids") or ())),
        )
        _positive(top, vocab=cfg.vocab, width=cfg.width)
        if not cfg.norm_eps > 0.0:
            raise ConfigError("config.json: norm.eps must be positive")
        for i, layer in enumerate(cfg.layers):
            j = layer.kv_from
            if j is None:
                continue
            where = f"layers[{i}].mixer"
            if not 0 <= j < i or cfg.layers[j].type != layer.type or cfg.layers[j].kv_from is not None:
                raise ConfigError(f"config.json: {where}: kv_from {j} must name an earlier {layer.type} layer with a "
                                  f"latent of its own")
            m, o = layer.mixer, cfg.layers[j].mixer
            if (o.kv_rank, o.rot_dim, o.rot) != (m.kv_rank, m.rot_dim, m.rot):
                raise ConfigError(f"config.json: {where}: the latents of layer {j} ({o.kv_rank} + {o.rot_dim} entries, "
                                  f"rot {o.rot.to_dict()}) do not fit this layer's")
        return cfg

    def to_dict(self) -> dict[str, Any]:
        d: dict[str, Any] = {
            "architecture": ARCHITECTURE,
            "embedding": {"scale": self.embedding_scale},
            "layers": [l.to_dict() for l in self.layers],
            "norm": {"eps": self.norm_eps},
            "vocab": self.vocab,
            "width": self.width,
            "torch_dtype": self.torch_dtype,
        }
        if self.max_positions != DEFAULT_MAX_POSITIONS:
            d["max_positions"] = self.max_positions
        if self.stop_token_ids:
            d["stop_token_ids"] = list(self.stop_token_ids)
        return d


def _mixer(cfg: SafuraxConfig, index: int, prefix: str) -> PartSpec:
    layer = cfg.layers[index]
    m = layer.mixer
    if layer.type == "latent_attention":
        return PartSpec("latent_attention", {
            "hidden_size": cfg.width, "heads": m.heads, "dim": m.dim, "rot_dim": 0, "value_dim": m.vdim,
            "q_rank": m.q_rank, "kv_rank": m.kv_rank, "scale": m.scale, "eps": cfg.norm_eps,
            "names": {"q_down": "dq", "q_norm": "dq.norm", "q_up": "uq", "kv_down": "dkv", "kv_norm": "dkv.norm",
                      "k_up": "uk", "v_up": "uv", "out": "o"}}, prefix)
    if layer.type == "latent_attention_2":
        # The cache of a layer whose latents other layers read keeps the widest window among them (all if one has none).
        windows = [m.window] + [l.mixer.window for l in cfg.layers if l.kv_from == index]
        cache_window = None if any(w is None for w in windows) else max(windows)
        return PartSpec("latent_attention", {
            "hidden_size": cfg.width, "heads": m.heads, "dim": m.dim, "rot_dim": m.rot_dim, "value_dim": m.vdim,
            "q_rank": None, "kv_rank": m.kv_rank, "scale": m.scale, "eps": cfg.norm_eps, "window": m.window,
            "cache_window": cache_window, "shared_kv": m.kv_from is not None, "shares_packed": len(windows) > 1,
            "sink": True, "output_gate": "heads", "position": m.rot.part(),
            "names": {"q": "q", "kv_down": "dkv", "kv_norm": "dkv.norm", "k_up": "uk", "v_up": "uv", "out": "o",
                      "sink": "sink", "gate": "g"}}, prefix)
    return PartSpec("softmax_attention", {
        "hidden_size": cfg.width, "num_heads": m.heads, "num_kv_heads": m.kv_heads, "key_dim": m.dim,
        "value_dim": m.vdim, "scale": m.scale, "values": "projected", "qk_norm_eps": cfg.norm_eps,
        "qk_norm_weights": True, "difference": {"offset": m.diff, "eps": cfg.norm_eps}, "head_gate": True,
        "position": m.rot.part(),
        "names": {"q": "q", "k": "k", "v": "v", "out": "o", "q_norm": "q.norm", "k_norm": "k.norm", "gate": "g",
                  "lq1": "lq1", "lk1": "lk1", "lq2": "lq2", "lk2": "lk2"}}, prefix)


def _feed_forward(cfg: SafuraxConfig, f: FeedForwardConfig, prefix: str) -> PartSpec:
    if f.kind == "dense":
        return PartSpec("swiglu", {"hidden_size": cfg.width, "intermediate_size": f.ff,
                                   "names": {"gate": "gate", "up": "up", "down": "down"}, "weight_suffix": ""}, prefix)
    return PartSpec("routed_experts", {
        "hidden_size": cfg.width, "intermediate_size": f.ff, "experts": f.experts, "top": f.top,
        "routing": "softmax_router", "router_bias": True, "shared_size": f.shared_ff, "shared_gate": f.shared_ff > 0,
        "names": {"expert": "e{}.", "gate": "gate", "up": "up", "down": "down", "router": "router",
                  "router_bias": "router.b", "shared": "shared.", "shared_gate": "shared.sg"}}, prefix)


def build_safurax_spec(cfg: SafuraxConfig) -> ModelSpec:
    """Safurax as parts: token embedding times its scale; per layer a pre-norm block (layer norm, mixer, layer norm,
    feed-forward); a layer with `kv_from` reads the cache of the schedule entry of the layer it names; layer norm; a
    head of its own."""
    def norm(name: str) -> PartSpec:
        return PartSpec("layer_norm", {"width": cfg.width, "eps": cfg.norm_eps, "weight_name": name})

    layers, schedule = [], []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        ffn = ffn_norm = None
        if layer.mlp is not None:
            ffn = _feed_forward(cfg, layer.mlp, p + "mlp.")
            ffn_norm = norm(p + "norm2")
        layers.append(LayerSpec(block="prenorm_residual", mixer=_mixer(cfg, i, p + "mix."), feed_forward=ffn,
                                mixer_norm=norm(p + "norm1"), feed_forward_norm=ffn_norm))
        schedule.append(ScheduleEntry(i, layer.kv_from))
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
        head=PartSpec("lm_head", {"vocab_size": cfg.vocab, "width": cfg.width, "weight_name": "head"}),
        stop_token_ids=cfg.stop_token_ids,
    )
    spec.validate()
    return spec
