"""The Dinatar decoder: its configuration, read from the keys of its own config.json, and its description as a list of
parts.

config.json names the architecture in the string `architecture`, gives `vocab`, `width`, `max_positions` (rows of the table of
learned position vectors), `norm.eps`, `embedding.scale`, `logit_scale` (on the logits of the tied head) and lists the layers
one by one: each entry gives `type` (which mixer), `mixer` (its sizes and constants) and `mlp` (a feed-forward, or null for a
layer without one).  A layer has ONE layer norm with weight and bias, whose rows both sublayers read:
x <- x + mixer(norm1(x)) + mlp(norm1(x)).  `loop` {start, stop, times}: the layers start .. stop-1 are passed `times` times in
a row with the same weights, every pass with caches and states of its own.  Tensors of layer i are called `l<i>.*`.

Mixers.  "hgrn2": linear attention whose forget gate (per head and key channel, with a learned lower bound) also decides what
is written; `heads`, `dim`, `vdim`.  "gla": linear attention with keys of their own, a decay per key channel made through a
short row of features (its length is the first size of the tensor `mix.a1`) and a tau-th root, and a SiLU gate on the result;
`heads`, `dim`, `vdim`, `tau`.  "parallel": `left`, grouped-query attention with biases, scores that fall with the distance by
a slope per head, and a sliding window of `mask.size` positions beside which the first `mask.keep_first` stay visible; `right`,
a Mamba-2 recurrence; each branch's result RMS-normed over the width, half the sum of the two.

Feed-forward: `kind` "dense", W_down relu(W_up h)^2; or "moe": `router.experts` experts with a gate branch and SiLU
(`expert.ff`), of which a token uses `router.top`, chosen by logits with a bias and weighed by a softmax over the chosen
logits; `shared`: an expert of the same form for every token.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Iterable, Mapping, Optional, Tuple

from ..config.reader import ConfigError, ConfigFields
from ..config.registry import Architecture, register_architecture
from ..parts.spec import (AttentionSpec, DenseActSpec, GatedLinearAttentionSpec, LayerSpec, Mamba2Spec, ModelSpec, NormSpec,
                          ParallelMixersSpec, PositionSpec, RoutedExpertsSpec, SharedExpertSpec, Stage)

BRANCH_SCALE = 0.5             # the two branches' normed results are averaged: fixed by the design
DECAY_RANK = 16                # length of the short row of a "gla" mixer where neither config.json nor a tensor says it


def _positive(f: ConfigFields, key: str) -> int:
    v = f.integer(key, required=True)
    if v <= 0:
        raise ConfigError(f"{f.origin}: {key}={v} must be positive")
    return v


def distance_slopes(heads: int) -> Tuple[float, ...]:
    """What the scores of head h fall by per position: 2^(-8 (h + 1) / heads)."""
    return tuple(2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads))


@dataclass(frozen=True)
class AttentionBranchConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: Optional[int] = None           # mask.size
    keep_first: int = 0                    # mask.keep_first

    def to_json_dict(self) -> dict:
        out = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale}
        if self.window is not None:
            out["mask"] = {"size": self.window, "keep_first": self.keep_first}
        return out


@dataclass(frozen=True)
class Mamba2BranchConfig:
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int
    norm_groups: int

    def to_json_dict(self) -> dict:
        return {"heads": self.heads, "vdim": self.vdim, "state": self.state, "groups": self.groups, "conv": self.conv,
                "norm_groups": self.norm_groups}


@dataclass(frozen=True)
class ParallelMixerConfig:
    left: AttentionBranchConfig
    right: Mamba2BranchConfig

    def to_json_dict(self) -> dict:
        return {"left": self.left.to_json_dict(), "right": self.right.to_json_dict()}


@dataclass(frozen=True)
class LinearMixerConfig:
    """"hgrn2" (tau and rank None) or "gla"."""
    heads: int
    dim: int
    vdim: int
    tau: Optional[float] = None
    rank: Optional[int] = None

    def to_json_dict(self) -> dict:
        out = {"heads": self.heads, "dim": self.dim, "vdim": self.vdim}
        if self.tau is not None:
            out.update(tau=self.tau, rank=self.rank)
        return out


@dataclass(frozen=True)
class DenseConfig:
    ff: int

    def to_json_dict(self) -> dict:
        return {"kind": "dense", "ff": self.ff}


@dataclass(frozen=True)
class ExpertsConfig:
    ff: int
    experts: int
    top: int
    shared_ff: Optional[int] = None        # None: no shared expert

    def to_json_dict(self) -> dict:
        out = {"kind": "moe", "expert": {"ff": self.ff}, "router": {"experts": self.experts, "top": self.top}}
        if self.shared_ff is not None:
            out["shared"] = {"ff": self.shared_ff}
        return out


@dataclass(frozen=True)
class DinatarLayerConfig:
    type: str                              # "hgrn2", "gla" or "parallel"
    mixer: object
    mlp: object                            # DenseConfig, ExpertsConfig or None


@dataclass(frozen=True)
class LoopConfig:
    start: int
    stop: int
    times: int


def _linear_mixer(f: ConfigFields, kind: str, rank: Optional[int]) -> LinearMixerConfig:
    tau = None
    if kind == "gla":
        tau = f.number("tau", required=True)
        if not tau > 0.0:
            raise ConfigError(f"{f.origin}: tau={tau} must be positive")
        if rank is None:
            rank = f.integer("rank", DECAY_RANK)
        if rank <= 0:
            raise ConfigError(f"{f.origin}: rank={rank} must be positive")
    return LinearMixerConfig(heads=_positive(f, "heads"), dim=_positive(f, "dim"), vdim=_positive(f, "vdim"), tau=tau,
                             rank=rank if kind == "gla" else None)


def _attention_branch(f: ConfigFields) -> AttentionBranchConfig:
    heads, kv_heads = _positive(f, "heads"), _positive(f, "kv_heads")
    if heads % kv_heads:
        raise ConfigError(f"{f.origin}: heads={heads} is not a multiple of kv_heads={kv_heads}")
    window, keep = None, 0
    mask = f.mapping("mask")
    if mask is not None:
        window, keep = _positive(mask, "size"), mask.integer("keep_first", 0)
        if keep < 0:
            raise ConfigError(f"{mask.origin}: keep_first={keep} must not be negative")
    scale = f.number("scale", required=True)
    if not scale > 0.0:
        raise ConfigError(f"{f.origin}: scale={scale} must be positive")
    return AttentionBranchConfig(heads=heads, kv_heads=kv_heads, dim=_positive(f, "dim"), vdim=_positive(f, "vdim"), scale=scale,
                                 window=window, keep_first=keep)


def _mamba2_branch(f: ConfigFields) -> Mamba2BranchConfig:
    c = Mamba2BranchConfig(heads=_positive(f, "heads"), vdim=_positive(f, "vdim"), state=_positive(f, "state"),
                           groups=_positive(f, "groups"), conv=_positive(f, "conv"), norm_groups=_positive(f, "norm_groups"))
    if c.heads % c.groups:
        raise ConfigError(f"{f.origin}: heads={c.heads} is not a multiple of groups={c.groups}")
    if (c.heads * c.vdim) % c.norm_groups:
        raise ConfigError(f"{f.origin}: {c.heads * c.vdim} features do not fall into norm_groups={c.norm_groups} equal parts")
    return c


def _mixer(f: ConfigFields, kind: str, rank: Optional[int]):
    if kind in ("hgrn2", "gla"):
        return _linear_mixer(f, kind, rank)
    if kind == "parallel":
        left, right = f.mapping("left"), f.mapping("right")
        if left is None or right is None:
            raise ConfigError(f"{f.origin} missing 'left' or 'right'")
        return ParallelMixerConfig(left=_attention_branch(left), right=_mamba2_branch(right))
    raise ConfigError(f"{f.origin}: layer type '{kind}' is not known (hgrn2, gla, parallel)")


def _feed_forward(f: ConfigFields):
    kind = f.string("kind", required=True)
    if kind == "dense":
        return DenseConfig(ff=_positive(f, "ff"))
    if kind != "moe":
        raise ConfigError(f"{f.origin}: feed-forward kind '{kind}' is not known (dense, moe)")
    expert, router = f.mapping("expert"), f.mapping("router")
    if expert is None or router is None:
        raise ConfigError(f"{f.origin} missing 'expert' or 'router'")
    experts, top = _positive(router, "experts"), _positive(router, "top")
    if top > experts:
        raise ConfigError(f"{router.origin}: top={top} of {experts} experts")
    shared = f.mapping("shared")
    return ExpertsConfig(ff=_positive(expert, "ff"), experts=experts, top=top, shared_ff=None if shared is None else _positive(shared, "ff"))


@dataclass(frozen=True)
class DinatarConfig:
    vocab: int
    width: int
    max_positions: int
    norm_eps: float
    embed_scale: float
    logit_scale: float
    layers: Tuple[DinatarLayerConfig, ...]
    loop: Optional[LoopConfig]

    architecture = "Dinatar"
    model_type = "dinatar"

    @classmethod
    def from_fields(cls, f: ConfigFields, tensor_names: Optional[Iterable[str]] = None) -> "DinatarConfig":
        """`tensor_names` may map the names to shapes: the length of a "gla" mixer's short row is read off there."""
        shapes = tensor_names if isinstance(tensor_names, Mapping) else {}
        vocab, width, max_positions = _positive(f, "vocab"), _positive(f, "width"), _positive(f, "max_positions")
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
            mf = e.mapping("mixer")
            if mf is None:
                raise ConfigError(f"{e.origin} missing 'mixer'")
            short = shapes.get(f"l{i}.mix.a1")
            mlp = e.mapping("mlp")
            layers.append(DinatarLayerConfig(type=kind, mixer=_mixer(mf, kind, None if short is None else int(short[0])),
                                             mlp=None if mlp is None else _feed_forward(mlp)))
        loop = None
        lf = f.mapping("loop")
        if lf is not None:
            loop = LoopConfig(start=lf.integer("start", required=True), stop=lf.integer("stop", required=True),
                              times=lf.integer("times", required=True))
            if not 0 <= loop.start <= loop.stop <= len(layers) or loop.times < 1:
                raise ConfigError(f"{lf.origin}: start={loop.start}, stop={loop.stop}, times={loop.times} do not name a run of "
                                  f"the {len(layers)} layers passed at least once")
            if loop.start == loop.stop:
                loop = None
        return cls(vocab=vocab, width=width, max_positions=max_positions, norm_eps=eps,
                   embed_scale=1.0 if emb is None else emb.number("scale", 1.0), logit_scale=f.number("logit_scale", 1.0),
                   layers=tuple(layers), loop=loop)

    def to_json_dict(self) -> dict:
        """The configuration as config.json keys (what the random-weights mode writes)."""
        out = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "max_positions": self.max_positions,
               "norm": {"eps": self.norm_eps}, "embedding": {"scale": self.embed_scale}, "logit_scale": self.logit_scale,
               "layers": [{"type": l.type, "mixer": l.mixer.to_json_dict(),
                           "mlp": None if l.mlp is None else l.mlp.to_json_dict()} for l in self.layers]}
        if self.loop is not None:
            out["loop"] = {"start": self.loop.start, "stop": self.loop.stop, "times": self.loop.times}
        return out


def _linear_spec(d: int, kind: str, m: LinearMixerConfig, eps: float, to: str):
    """(mixer spec, its tensors' checkpoint names) of a "hgrn2" or "gla" mixer whose tensors begin with `to`."""
    names = {"mixer.q_proj.weight": to + "q", "mixer.v_proj.weight": to + "v", "mixer.norm.weight": to + "norm", "mixer.o_proj.weight": to + "o"}
    if kind == "hgrn2":
        names.update({"mixer.f_proj.weight": to + "f", "mixer.f_proj.bias": to + "f.b", "mixer.lower": to + "lower"})
        return GatedLinearAttentionSpec(hidden=d, n_heads=m.heads, dim=m.dim, vdim=m.vdim, eps=eps, write="forget", query_silu=True), names
    names.update({"mixer.k_proj.weight": to + "k", "mixer.decay_in.weight": to + "a1", "mixer.decay_out.weight": to + "a2",
                  "mixer.decay_out.bias": to + "a2.b", "mixer.g_proj.weight": to + "g"})
    return GatedLinearAttentionSpec(hidden=d, n_heads=m.heads, dim=m.dim, vdim=m.vdim, eps=eps, write="key",
                                    query_scale=float(m.dim) ** -0.5, decay_rank=m.rank, decay_power=1.0 / m.tau, gated=True), names


def _parallel_spec(d: int, m: ParallelMixerConfig, eps: float, to: str):
    a, b = m.left, m.right
    left = AttentionSpec(hidden=d, n_heads=a.heads, n_kv_heads=a.kv_heads, head_dim=a.dim, qkv_bias=True,
                         position=PositionSpec(kind="none"), window=a.window, scale=a.scale, v_head_dim=a.vdim,
                         keep_first=a.keep_first if a.window is not None else 0, slopes=distance_slopes(a.heads))
    right = Mamba2Spec(hidden=d, n_heads=b.heads, vdim=b.vdim, state=b.state, groups=b.groups, conv=b.conv, norm_groups=b.norm_groups,
                       eps=eps, chunked=True)
    names = {f"mixer.left.{x}_proj.{kind}": f"{to}left.{x}{end}" for x in "qkv" for kind, end in (("weight", ""), ("bias", ".b"))}
    names.update({"mixer.left.o_proj.weight": to + "left.o", "mixer.left.out_norm.weight": to + "left.out",
                  "mixer.right.in_proj.weight": to + "right.in", "mixer.right.conv.weight": to + "right.conv",
                  "mixer.right.conv.bias": to + "right.conv.b", "mixer.right.dt_bias": to + "right.dt_bias",
                  "mixer.right.A_log": to + "right.A_log", "mixer.right.D": to + "right.D", "mixer.right.norm.weight": to + "right.norm",
                  "mixer.right.o_proj.weight": to + "right.o", "mixer.right.out_norm.weight": to + "right.out"})
    return ParallelMixersSpec(hidden=d, branches=(left, right), scales=(BRANCH_SCALE, BRANCH_SCALE), labels=("left", "right"),
                              out_norm_eps=eps), names


def _feed_forward_spec(d: int, f, to: str):
    if isinstance(f, DenseConfig):
        return DenseActSpec(hidden=d, intermediate=f.ff, activation="relu2"), \
            {"feed_forward.up.weight": to + "up", "feed_forward.down.weight": to + "down"}
    names = {"feed_forward.router.weight": to + "router", "feed_forward.router.logit_bias": to + "router.b"}
    for e in range(f.experts):
        for part in ("gate", "up", "down"):
            names[f"feed_forward.experts.{e}.{part}.weight"] = f"{to}e{e}.{part}"
    shared = None
    if f.shared_ff is not None:
        shared = SharedExpertSpec(intermediate=f.shared_ff, gated=False)
        for part in ("gate", "up", "down"):
            names[f"feed_forward.shared.{part}.weight"] = f"{to}shared.{part}"
    return RoutedExpertsSpec(hidden=d, intermediate=f.ff, experts=f.experts, top=f.top, activation="swiglu",
                             router_activation="softmax_chosen", scale_input=False, logit_bias=True, shared=shared), names


def build_spec(cfg: DinatarConfig) -> ModelSpec:
    d, eps = cfg.width, cfg.norm_eps
    norm = NormSpec(size=d, eps=eps, kind="layernorm", shift=True)
    layers = []
    for i, l in enumerate(cfg.layers):
        p = f"l{i}."
        if l.type == "parallel":
            mixer, names = _parallel_spec(d, l.mixer, eps, p + "mix.")
        else:
            mixer, names = _linear_spec(d, l.type, l.mixer, eps, p + "mix.")
        parts = {"mixer_norm": norm, "mixer": mixer}
        names.update({"mixer_norm.weight": p + "norm1", "mixer_norm.bias": p + "norm1.b"})
        if l.mlp is not None:
            parts["feed_forward"], ff_names = _feed_forward_spec(d, l.mlp, p + "mlp.")
            names.update(ff_names)
        layers.append(LayerSpec(parts, names, block="parallel_shared" if l.mlp is not None else "parallel_mixer"))
    n = len(layers)
    order = list(range(n))
    if cfg.loop is not None:                       # every pass: caches and states of its own
        lo, hi = cfg.loop.start, cfg.loop.stop
        order = order[:lo] + order[lo:hi] * cfg.loop.times + order[hi:]
    return ModelSpec(vocab=cfg.vocab, hidden=d, layers=layers, order=[Stage(layer=i) for i in order], final_norm=norm,
                     embed_name="embed", final_norm_name="final.norm", final_norm_bias_name="final.norm.b", head_name=None,
                     max_positions=cfg.max_positions, embed_scale=cfg.embed_scale, position_name="pos", logit_scale=cfg.logit_scale)


ARCHITECTURE = register_architecture(Architecture(
    name=DinatarConfig.architecture, model_type=DinatarConfig.model_type,
    config_class=DinatarConfig, build_spec=build_spec))
