"""The typed configuration of the Tomalix decoder, read from its own config.json keys.

    architecture    "Tomalix"
    vocab, width    sizes of the token table and of the residual stream
    norm            {"eps"}
    logit_softcap   logits are squashed into (-cap, cap); absent or null: they are not
    loop            {"start", "stop", "times"}: layers start .. stop - 1 run `times` times in a row; absent: no loop
    layers          a list; every entry has "type" ("attention", "attention_2" or "parallel"), "mixer" (its sizes and
                    constants) and "mlp" ({"kind": "dense", "ff"}, {"kind": "moe", "expert": {"ff"}, "router": {"experts",
                    "top"}} or null)

An "attention" mixer (two maps a head): heads, kv_heads, dim, vdim, scale, diff, rot {dims, base, scaling {factor}}.  An
"attention_2" mixer: heads, kv_heads, dim, vdim, scale, rot {dims, base, scaling {factor, original, fast, slow}}.  A
"parallel" mixer: left {heads, kv_heads, dim, vdim, scale, mask {size}, rot {dims, base}}, left_scale, right {inner, state,
conv, dt_rank}, right_scale.  A rotation without "scaling" keeps its frequencies.  Every layer carries its own sizes.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Optional, Union

from .reader import ConfigError, KeyReader
from .ridopel import LoopConfig


@dataclass(frozen=True)
class LinearScalingConfig:
    factor: float       # every frequency is divided by it


@dataclass(frozen=True)
class YarnScalingConfig:
    factor: float
    original: float     # positions the unscaled frequencies were made for
    fast: float         # lanes that turn at least this often over them keep their frequency
    slow: float         # lanes that turn at most this often have it divided by the factor


@dataclass(frozen=True)
class RotationConfig:
    dims: int           # how many of a head's first lanes turn
    base: float
    scaling: Union[LinearScalingConfig, YarnScalingConfig, None] = None


@dataclass(frozen=True)
class AttentionMixerConfig:
    heads: int
    kv_heads: int
    dim: int            # query/key lanes of a head (of each of its maps where it has two)
    vdim: int           # value lanes of a head
    scale: float
    rot: RotationConfig
    diff: Optional[float] = None     # a head has two maps and this constant in the weight of the second
    chunk: Optional[int] = None      # a position sees the positions of its own chunk of this many


@dataclass(frozen=True)
class ScanMixerConfig:
    inner: int          # channels of the scan
    state: int          # states of a channel
    conv: int           # taps of the convolution
    dt_rank: int        # lanes the step sizes are made from


@dataclass(frozen=True)
class ParallelMixerConfig:
    left: AttentionMixerConfig
    right: ScanMixerConfig
    left_scale: float
    right_scale: float


@dataclass(frozen=True)
class DenseConfig:
    ff: int


@dataclass(frozen=True)
class ExpertsConfig:
    experts: int
    top: int
    ff: int


@dataclass(frozen=True)
class TomalixLayerConfig:
    type: str
    mixer: Union[AttentionMixerConfig, ParallelMixerConfig]
    mlp: Union[DenseConfig, ExpertsConfig, None]


def _rotation(m: KeyReader, where: str, lanes: int, scaling: str) -> RotationConfig:
    rot = KeyReader(m.obj("rot"), where + "rot.")
    dims, base = rot.integer("dims", minimum=0), rot.number("base", positive=True)
    if dims % 2 or dims > lanes:
        raise ConfigError(f"config key '{where}rot.dims' ({dims}) must be even and at most {lanes}")
    found = rot.obj("scaling", default=None)
    if found is None or scaling == "none":
        if found is not None:
            raise ConfigError(f"config key '{where}rot.scaling': this mixer's rotation is not scaled")
        return RotationConfig(dims, base)
    s = KeyReader(found, where + "rot.scaling.")
    factor = s.number("factor", positive=True)
    if scaling == "linear":
        return RotationConfig(dims, base, LinearScalingConfig(factor))
    if not base > 1.0:
        raise ConfigError(f"config key '{where}rot.base' ({base}) must be above 1 where the frequencies are scaled by lanes")
    return RotationConfig(dims, base, YarnScalingConfig(factor, s.number("original", positive=True), s.number("fast", positive=True),
                                                        s.number("slow", positive=True)))


def _attention(m: KeyReader, where: str, scaling: str, diff=False, chunk=False) -> AttentionMixerConfig:
    dim = m.integer("dim", minimum=1)
    mixer = AttentionMixerConfig(
        heads=m.integer("heads", minimum=1), kv_heads=m.integer("kv_heads", minimum=1), dim=dim, vdim=m.integer("vdim", minimum=1),
        scale=m.number("scale"), rot=_rotation(m, where, dim, scaling), diff=m.number("diff") if diff else None,
        chunk=KeyReader(m.obj("mask"), where + "mask.").integer("size", minimum=1) if chunk else None)
    if mixer.heads % mixer.kv_heads:
        raise ConfigError(f"config key '{where}heads' ({mixer.heads}) must be a multiple of 'kv_heads' ({mixer.kv_heads})")
    return mixer


def _feed_forward(lr: KeyReader, where: str):
    f = lr.obj("mlp", default=None)
    if f is None:
        return None
    fr = KeyReader(f, where + "mlp.")
    kind = fr.string("kind")
    if kind == "dense":
        return DenseConfig(fr.integer("ff", minimum=1))
    if kind != "moe":
        raise ConfigError(f"config key '{where}mlp.kind' is {kind!r}; this decoder knows 'dense' and 'moe'")
    er, rr = KeyReader(fr.obj("expert"), where + "mlp.expert."), KeyReader(fr.obj("router"), where + "mlp.router.")
    mlp = ExpertsConfig(experts=rr.integer("experts", minimum=1), top=rr.integer("top", minimum=1), ff=er.integer("ff", minimum=1))
    if mlp.top > mlp.experts:
        raise ConfigError(f"config key '{where}mlp.router.top' ({mlp.top}) must be at most 'experts' ({mlp.experts})")
    return mlp


def _rotation_dict(rot: RotationConfig) -> dict:
    d = {"dims": rot.dims, "base": rot.base}
    s = rot.scaling
    if isinstance(s, LinearScalingConfig):
        d["scaling"] = {"factor": s.factor}
    elif s is not None:
        d["scaling"] = {"factor": s.factor, "original": s.original, "fast": s.fast, "slow": s.slow}
    return d


def _attention_dict(m: AttentionMixerConfig) -> dict:
    d = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale, "rot": _rotation_dict(m.rot)}
    if m.diff is not None:
        d["diff"] = m.diff
    if m.chunk is not None:
        d["mask"] = {"size": m.chunk}
    return d


@dataclass(frozen=True)
class TomalixConfig:
    vocab: int
    width: int
    eps: float
    layers: tuple
    loop: Optional[LoopConfig] = None
    logit_softcap: Optional[float] = None
    architecture: str = "Tomalix"
    torch_dtype: Optional[str] = None
    raw: dict = field(default_factory=dict, compare=False, repr=False)

    @classmethod
    def from_dict(cls, data: dict) -> "TomalixConfig":
        r = KeyReader(data)
        eps = KeyReader(r.obj("norm"), "norm.").number("eps", positive=True)
        raw_layers = data.get("layers")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise ConfigError("config key 'layers' must be a non-empty list")
        layers = []
        for i, entry in enumerate(raw_layers):
            where = f"layers[{i}]."
            if not isinstance(entry, dict):
                raise ConfigError(f"config key 'layers[{i}]' must be an object")
            lr = KeyReader(entry, where)
            kind = lr.string("type")
            mw = where + "mixer."
            m = KeyReader(lr.obj("mixer"), mw)
            if kind == "attention":
                mixer = _attention(m, mw, "linear", diff=True)
            elif kind == "attention_2":
                mixer = _attention(m, mw, "yarn")
            elif kind == "parallel":
                right = KeyReader(m.obj("right"), mw + "right.")
                mixer = ParallelMixerConfig(
                    left=_attention(KeyReader(m.obj("left"), mw + "left."), mw + "left.", "none", chunk=True),
                    right=ScanMixerConfig(inner=right.integer("inner", minimum=1), state=right.integer("state", minimum=1),
                                          conv=right.integer("conv", minimum=1), dt_rank=right.integer("dt_rank", minimum=1)),
                    left_scale=m.number("left_scale"), right_scale=m.number("right_scale"))
            else:
                raise ConfigError(f"config key '{where}type' is {kind!r}; this decoder knows 'attention', 'attention_2' and 'parallel'")
            layers.append(TomalixLayerConfig(kind, mixer, _feed_forward(lr, where)))
        loop = None
        lp = r.obj("loop", default=None)
        if lp is not None:
            lo = KeyReader(lp, "loop.")
            loop = LoopConfig(lo.integer("start", minimum=0), lo.integer("stop", minimum=0), lo.integer("times", minimum=1))
            if not loop.start <= loop.stop <= len(layers):
                raise ConfigError(f"config key 'loop': layers {loop.start} .. {loop.stop} - 1 of {len(layers)}")
        cap = r.number("logit_softcap", default=None, positive=True)
        return cls(vocab=r.integer("vocab", minimum=1), width=r.integer("width", minimum=1), eps=eps, layers=tuple(layers),
                   loop=loop, logit_softcap=cap, architecture=r.string("architecture", default="Tomalix"),
                   torch_dtype=r.string("torch_dtype", default=None) or r.string("dtype", default=None), raw=dict(data))

    def to_dict(self) -> dict:
        """The config.json content of this configuration."""
        layers = []
        for layer in self.layers:
            m, f = layer.mixer, layer.mlp
            if layer.type == "parallel":
                s = m.right
                mixer = {"left": _attention_dict(m.left), "left_scale": m.left_scale,
                         "right": {"inner": s.inner, "state": s.state, "conv": s.conv, "dt_rank": s.dt_rank}, "right_scale": m.right_scale}
            else:
                mixer = _attention_dict(m)
            mlp = None
            if isinstance(f, DenseConfig):
                mlp = {"kind": "dense", "ff": f.ff}
            elif f is not None:
                mlp = {"kind": "moe", "expert": {"ff": f.ff}, "router": {"experts": f.experts, "top": f.top}}
            layers.append({"type": layer.type, "mixer": mixer, "mlp": mlp})
        d = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps}, "layers": layers}
        if self.loop is not None:
            d["loop"] = {"start": self.loop.start, "stop": self.loop.stop, "times": self.loop.times}
        if self.logit_softcap is not None:
            d["logit_softcap"] = self.logit_softcap
        if self.torch_dtype:
            d["torch_dtype"] = self.torch_dtype
        return d
