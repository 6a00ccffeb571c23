"""The Fanitar decoder: its configuration, read from the keys of its own config.json, and its description as a list of
parts.

config.json names the architecture in the string `architecture`, gives `vocab`, `width`, `norm.eps`, `embedding.scale` (the
embedded rows times a constant), `logit_scale` and lists the layers one by one: each entry gives `type` (which mixer), `mixer`
(its sizes and constants) and `mlp` (a feed-forward, or null for a layer without one).  Every sublayer has an RMS norm in
front of it and another on its result: x <- x + norm1b(mixer(norm1(x))), then x <- x + norm2b(mlp(norm2(x))).  `loop` {start,
stop, times}: the layers start .. stop-1 are passed `times` times in a row with the same weights, every pass with caches of
its own; in front of pass t the stream gets the embedded rows once more (t > 0) and the row t of the tensor `loop.step`.
Tensors of layer i are called `l<i>.*`.

Mixers.  "attention": grouped-query attention with biases whose heads come as pairs of maps over the same values (`heads`,
`kv_heads`, `dim` features per map, `vdim`, `scale`), the leading `rot.dims` features of every map rotated in halves; the
second map's result is taken off the first's times one number of the layer, made from four learned vectors and `diff`, and
the difference is normed head by head.  "latent_attention": queries from a normed row of `q_rank` features (the tensor
`mix.dq` says how many where config.json does not), keys and values from one of `kv_rank`, no positions, a sliding window of
`mask.size`, a learned sink per head, a sigmoid gate per feature of the joined heads.

Feed-forward (`mlp.kind` "dense"): a gated activation whose branches are cut off at `limit`.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Iterable, List, Mapping, Optional, Tuple

from ..config.reader import ConfigError, ConfigFields
from ..config.registry import Architecture, register_architecture
from ..parts.spec import (DifferentialAttentionSpec, EntrySpec, LatentAttentionSpec, LayerSpec, ModelSpec, NormSpec, PassStepSpec,
                          PositionSpec, Stage, SwiGLUSpec)


def _positive(f: ConfigFields, key: str) -> int:
    v = f.integer(key, required=True)
    if v <= 0:
        raise ConfigError(f"{f.origin}: {key}={v} must be positive")
    return v


def _positive_number(f: ConfigFields, key: str) -> float:
    v = f.number(key, required=True)
    if not v > 0.0:
        raise ConfigError(f"{f.origin}: {key}={v} must be positive")
    return v


@dataclass(frozen=True)
class DifferentialMixerConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    diff: float
    rot_base: float = 10000.0
    rot_dims: int = 0                      # 0: no rotation

    def to_json_dict(self) -> dict:
        out = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale,
               "diff": self.diff}
        if self.rot_dims:
            out["rot"] = {"base": self.rot_base, "dims": self.rot_dims}
        return out


@dataclass(frozen=True)
class LatentMixerConfig:
    heads: int
    dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    window: Optional[int] = None           # mask.size

    def to_json_dict(self) -> dict:
        out = {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "q_rank": self.q_rank, "kv_rank": self.kv_rank,
               "scale": self.scale}
        if self.window is not None:
            out["mask"] = {"size": self.window}
        return out


@dataclass(frozen=True)
class DenseConfig:
    ff: int
    limit: float

    def to_json_dict(self) -> dict:
        return {"kind": "dense", "ff": self.ff, "limit": self.limit}


@dataclass(frozen=True)
class FanitarLayerConfig:
    type: str                              # "attention" or "latent_attention"
    mixer: object
    mlp: Optional[DenseConfig]


@dataclass(frozen=True)
class LoopConfig:
    start: int
    stop: int
    times: int


def _differential_mixer(f: ConfigFields, shape) -> DifferentialMixerConfig:
    heads, kv_heads = _positive(f, "heads"), _positive(f, "kv_heads")
    if heads % kv_heads:
        raise ConfigError(f"{f.origin}: heads={heads} is not a multiple of kv_heads={kv_heads}")
    dim = _positive(f, "dim")
    base, dims = 10000.0, 0
    rot = f.mapping("rot")
    if rot is not None:
        dims, base = rot.integer("dims", required=True), _positive_number(rot, "base")
        if dims < 0 or dims % 2 or dims > dim:
            raise ConfigError(f"{rot.origin}: dims={dims} must be even and at most dim={dim}")
    return DifferentialMixerConfig(heads=heads, kv_heads=kv_heads, dim=dim, vdim=_positive(f, "vdim"), scale=_positive_number(f, "scale"),
                                   diff=f.number("diff", required=True), rot_base=base, rot_dims=dims)


def _latent_mixer(f: ConfigFields, shape) -> LatentMixerConfig:
    q_rank = f.integer("q_rank", None if shape is None else int(shape[0]), required=shape is None)
    if q_rank <= 0:
        raise ConfigError(f"{f.origin}: q_rank={q_rank} must be positive")
    window, mask = None, f.mapping("mask")
    if mask is not None:
        window = _positive(mask, "size")
    return LatentMixerConfig(heads=_positive(f, "heads"), dim=_positive(f, "dim"), vdim=_positive(f, "vdim"), q_rank=q_rank,
                             kv_rank=_positive(f, "kv_rank"), scale=_positive_number(f, "scale"), window=window)


_MIXERS = {"attention": _differential_mixer, "latent_attention": _latent_mixer}


def _feed_forward(f: ConfigFields) -> DenseConfig:
    kind = f.string("kind", required=True)
    if kind != "dense":
        raise ConfigError(f"{f.origin}: feed-forward kind '{kind}' is not known (dense)")
    return DenseConfig(ff=_positive(f, "ff"), limit=_positive_number(f, "limit"))


@dataclass(frozen=True)
class FanitarConfig:
    vocab: int
    width: int
    norm_eps: float
    embed_scale: float
    logit_scale: float
    layers: Tuple[FanitarLayerConfig, ...]
    loop: Optional[LoopConfig]

    architecture = "Fanitar"
    model_type = "fanitar"

    @classmethod
    def from_fields(cls, f: ConfigFields, tensor_names: Optional[Iterable[str]] = None) -> "FanitarConfig":
        """`tensor_names` may map the names to shapes: the length of a query latent is read off there where the entry does not
        give it."""
        shapes = tensor_names if isinstance(tensor_names, Mapping) else {}
        vocab, width = _positive(f, "vocab"), _positive(f, "width")
        norm = f.mapping("norm")
        if norm is None:
            raise ConfigError(f"{f.origin} missing 'norm'")
        eps = norm.number("eps", required=True)
        if not eps >= 0.0:
            raise ConfigError(f"{f.origin}: norm.eps={eps} must not be negative")
        emb = f.mapping("embedding")
        entries = f.mapping_list("layers", required=True)
        if not entries:
            raise ConfigError(f"{f.origin}: 'layers' is empty")
        layers = []
        for i, e in enumerate(entries):
            kind = e.string("type", required=True)
            if kind not in _MIXERS:
                raise ConfigError(f"{e.origin}: layer type '{kind}' is not known ({', '.join(_MIXERS)})")
            mf = e.mapping("mixer")
            if mf is None:
                raise ConfigError(f"{e.origin} missing 'mixer'")
            mlp = e.mapping("mlp")
            layers.append(FanitarLayerConfig(type=kind, mixer=_MIXERS[kind](mf, shapes.get(f"l{i}.mix.dq")),
                                             mlp=None if mlp is None else _feed_forward(mlp)))
        loop = None
        lf = f.mapping("loop")
        if lf is not None:
            loop = LoopConfig(start=lf.integer("start", required=True), stop=lf.integer("stop", required=True),
                              times=lf.integer("times", required=True))
            if not 0 <= loop.start < loop.stop <= len(layers) or loop.times < 1:
                raise ConfigError(f"{lf.origin}: start={loop.start}, stop={loop.stop}, times={loop.times} do not name a run of "
                                  f"the {len(layers)} layers passed at least once")
        return cls(vocab=vocab, width=width, norm_eps=eps, embed_scale=1.0 if emb is None else emb.number("scale", 1.0),
                   logit_scale=f.number("logit_scale", 1.0), layers=tuple(layers), loop=loop)

    def to_json_dict(self) -> dict:
        """The configuration as config.json keys (what the random-weights mode writes)."""
        out = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
               "embedding": {"scale": self.embed_scale}, "logit_scale": self.logit_scale,
               "layers": [{"type": l.type, "mixer": l.mixer.to_json_dict(),
                           "mlp": None if l.mlp is None else l.mlp.to_json_dict()} for l in self.layers]}
        if self.loop is not None:
            out["loop"] = {"start": self.loop.start, "stop": self.loop.stop, "times": self.loop.times}
        return out


def _mixer(d: int, m, eps: float, to: str):
    """(mixer spec, its tensors' checkpoint names) of a layer whose mixer's tensors begin with `to`."""
    if isinstance(m, DifferentialMixerConfig):
        position = PositionSpec(kind="none")
        if m.rot_dims:
            position = PositionSpec(kind="rope", rotary_dim=m.rot_dims, theta=m.rot_base, pairing="split_half",
                                    frequencies=tuple(m.rot_base ** (-2.0 * i / m.rot_dims) for i in range(m.rot_dims // 2)))
        spec = DifferentialAttentionSpec(hidden=d, n_heads=m.heads, n_kv_heads=m.kv_heads, dim=m.dim, vdim=m.vdim, scale=m.scale,
                                         diff=m.diff, eps=eps, position=position)
        names = {f"mixer.{x}_proj.{kind}": f"{to}{x}{end}" for x in "qkv" for kind, end in (("weight", ""), ("bias", ".b"))}
        names.update({f"mixer.{v}": to + v for v in ("lq1", "lk1", "lq2", "lk2")})
        names["mixer.o_proj.weight"] = to + "o"
        return spec, names
    spec = LatentAttentionSpec(hidden=d, n_heads=m.heads, dim=m.dim, rot_dim=0, vdim=m.vdim, q_rank=m.q_rank, kv_rank=m.kv_rank,
                               scale=m.scale, eps=eps, position=PositionSpec(kind="none"), gated=True, gate_features=True,
                               window=m.window, sink=True)
    names = {"mixer.q_down.weight": to + "dq", "mixer.q_down.norm": to + "dq.norm", "mixer.q_up.weight": to + "uq",
             "mixer.kv_down.weight": to + "dkv", "mixer.kv_down.norm": to + "dkv.norm", "mixer.k_up.weight": to + "uk",
             "mixer.v_up.weight": to + "uv", "mixer.sink": to + "sink", "mixer.gate.weight": to + "g", "mixer.o_proj.weight": to + "o"}
    return spec, names


def build_spec(cfg: FanitarConfig) -> ModelSpec:
    d, eps = cfg.width, cfg.norm_eps
    norm = NormSpec(size=d, eps=eps)
    layers: List[LayerSpec] = []
    for i, l in enumerate(cfg.layers):
        p = f"l{i}."
        mixer, names = _mixer(d, l.mixer, eps, p + "mix.")
        parts = {"mixer_norm": norm, "mixer": mixer, "mixer_out_norm": norm}
        names.update({"mixer_norm.weight": p + "norm1", "mixer_out_norm.weight": p + "norm1b"})
        if l.mlp is not None:
            parts.update({"feed_forward_norm": norm, "feed_forward_out_norm": norm,
                          "feed_forward": SwiGLUSpec(hidden=d, intermediate=l.mlp.ff, activation="glu_clamped", limit=l.mlp.limit)})
            names.update({"feed_forward_norm.weight": p + "norm2", "feed_forward_out_norm.weight": p + "norm2b",
                          "feed_forward.gate_proj.weight": p + "mlp.gate", "feed_forward.up_proj.weight": p + "mlp.up",
                          "feed_forward.down_proj.weight": p + "mlp.down"})
        layers.append(LayerSpec(parts, names, block="sandwich" if l.mlp is not None else "sandwich_mixer"))
    n = len(layers)
    order, entries = [Stage(layer=i) for i in range(n)], []
    if cfg.loop is not None:                       # every pass: caches of its own, what it begins with in front of it
        lo, hi = cfg.loop.start, cfg.loop.stop
        for t in range(cfg.loop.times):
            entries.append(EntrySpec(part=PassStepSpec(hidden=d, passes=cfg.loop.times, index=t, again=t > 0),
                                     names={"step": "loop.step"}))
        runs = [Stage(layer=i, enter=t if i == lo else None) for t in range(cfg.loop.times) for i in range(lo, hi)]
        order = order[:lo] + runs + order[hi:]
    return ModelSpec(vocab=cfg.vocab, hidden=d, layers=layers, order=order, final_norm=norm, embed_name="embed",
                     final_norm_name="final.norm", head_name="head", embed_scale=cfg.embed_scale, logit_scale=cfg.logit_scale,
                     entries=entries)


ARCHITECTURE = register_architecture(Architecture(
    name=FanitarConfig.architecture, model_type=FanitarConfig.model_type,
    config_class=FanitarConfig, build_spec=build_spec))
