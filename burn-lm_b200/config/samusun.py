"""The typed configuration of the Samusun decoder, read from its own config.json keys.

    architecture    "Samusun"
    vocab, width    sizes of the token table and of the residual stream
    norm            {"eps"}
    embedding       {"scale"}: what a token's row is multiplied by
    logit_scale     what the output projection is multiplied by; absent: 1
    logit_softcap   logits are squashed into (-cap, cap); absent or null: they are not
    loop            {"start", "stop", "times"}: layers start .. stop - 1 run `times` times in a row; absent: no loop
    layers          a list; every entry has "type" ("attention" or "retention"), "mixer" (its sizes and constants) and "mlp"
                    ({"kind": "dense", "ff"}, {"kind": "moe", "expert": {"ff"}, "router": {"experts", "top"}} or null)

An "attention" mixer: heads, kv_heads, dim, vdim (equal to dim: the values are the keys), scale, mask {size} (absent: every
earlier token is seen), q_temp {coef, every} (absent: queries as they are).  A "retention" mixer: heads, dim, vdim, decay (a
number per head), rot {dims, base} (absent: no rotation).  Every layer carries its own sizes.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Optional, Union

from .reader import ConfigError, KeyReader
from .ridopel import LoopConfig
from .tomalix import DenseConfig, ExpertsConfig, RotationConfig, _feed_forward, _rotation


@dataclass(frozen=True)
class TemperatureConfig:
    coef: float         # a query is multiplied by 1 + coef ln(floor((position + 1) / every) + 1)
    every: int


@dataclass(frozen=True)
class SharedAttentionConfig:
    heads: int
    kv_heads: int
    dim: int            # lanes of a head's query, key and value
    scale: float
    window: Optional[int] = None             # how many of the latest keys, its own included, a position sees
    q_temp: Optional[TemperatureConfig] = None


@dataclass(frozen=True)
class RetentionConfig:
    heads: int
    dim: int            # lanes of a head's query and key
    vdim: int           # lanes of a head's value
    decay: tuple        # a number per head
    rot: Optional[RotationConfig] = None


@dataclass(frozen=True)
class SamusunLayerConfig:
    type: str
    mixer: Union[SharedAttentionConfig, RetentionConfig]
    mlp: Union[DenseConfig, ExpertsConfig, None]


def _attention(m: KeyReader, where: str) -> SharedAttentionConfig:
    dim, vdim = m.integer("dim", minimum=1), m.integer("vdim", minimum=1)
    if vdim != dim:
        raise ConfigError(f"config key '{where}vdim' ({vdim}) must equal 'dim' ({dim}): the values are the keys")
    mask, temp, window, q_temp = m.obj("mask", default=None), m.obj("q_temp", default=None), None, None
    if mask is not None:
        window = KeyReader(mask, where + "mask.").integer("size", minimum=1)
    if temp is not None:
        t = KeyReader(temp, where + "q_temp.")
        q_temp = TemperatureConfig(t.number("coef"), t.integer("every", minimum=1))
    mixer = SharedAttentionConfig(m.integer("heads", minimum=1), m.integer("kv_heads", minimum=1), dim, m.number("scale"), window, q_temp)
    if mixer.heads % mixer.kv_heads:
        raise ConfigError(f"config key '{where}heads' ({mixer.heads}) must be a multiple of 'kv_heads' ({mixer.kv_heads})")
    return mixer


def _retention(m: KeyReader, where: str) -> RetentionConfig:
    heads, dim = m.integer("heads", minimum=1), m.integer("dim", minimum=1)
    decay = m.data.get("decay")
    if (not isinstance(decay, list) or len(decay) != heads
            or any(isinstance(d, bool) or not isinstance(d, (int, float)) or not 0.0 <= d <= 1.0 for d in decay)):
        raise ConfigError(f"config key '{where}decay' must be a list of {heads} numbers between 0 and 1")
    rot = _rotation(m, where, dim, "none") if m.obj("rot", default=None) is not None else None
    return RetentionConfig(heads, dim, m.integer("vdim", minimum=1), tuple(float(d) for d in decay), rot)


@dataclass(frozen=True)
class SamusunConfig:
    vocab: int
    width: int
    eps: float
    layers: tuple
    embedding_scale: float = 1.0
    logit_scale: float = 1.0
    logit_softcap: Optional[float] = None
    loop: Optional[LoopConfig] = None
    architecture: str = "Samusun"
    torch_dtype: Optional[str] = None
    raw: dict = field(default_factory=dict, compare=False, repr=False)

    @classmethod
    def from_dict(cls, data: dict) -> "SamusunConfig":
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
            if kind not in ("attention", "retention"):
                raise ConfigError(f"config key '{where}type' is {kind!r}; this decoder knows 'attention' and 'retention'")
            m = KeyReader(lr.obj("mixer"), where + "mixer.")
            mixer = (_attention if kind == "attention" else _retention)(m, where + "mixer.")
            layers.append(SamusunLayerConfig(kind, mixer, _feed_forward(lr, where)))
        loop = None
        lp = r.obj("loop", default=None)
        if lp is not None:
            lo = KeyReader(lp, "loop.")
            loop = LoopConfig(lo.integer("start", minimum=0), lo.integer("stop", minimum=0), lo.integer("times", minimum=1))
            if not loop.start <= loop.stop <= len(layers):
                raise ConfigError(f"config key 'loop': layers {loop.start} .. {loop.stop} - 1 of {len(layers)}")
        emb = r.obj("embedding", default=None)
        return cls(vocab=r.integer("vocab", minimum=1), width=r.integer("width", minimum=1), eps=eps, layers=tuple(layers),
                   embedding_scale=KeyReader(emb, "embedding.").number("scale", default=1.0) if emb is not None else 1.0,
                   logit_scale=r.number("logit_scale", default=1.0), logit_softcap=r.number("logit_softcap", default=None, positive=True),
                   loop=loop, architecture=r.string("architecture", default="Samusun"),
                   torch_dtype=r.string("torch_dtype", default=None) or r.string("dtype", default=None), raw=dict(data))

    def to_dict(self) -> dict:
        """The config.json content of this configuration."""
        layers = []
        for layer in self.layers:
            m, f = layer.mixer, layer.mlp
            if layer.type == "attention":
                mixer = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.dim, "scale": m.scale}
                if m.window is not None:
                    mixer["mask"] = {"size": m.window}
                if m.q_temp is not None:
                    mixer["q_temp"] = {"coef": m.q_temp.coef, "every": m.q_temp.every}
            else:
                mixer = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim, "decay": list(m.decay)}
                if m.rot is not None:
                    mixer["rot"] = {"dims": m.rot.dims, "base": m.rot.base}
            mlp = None
            if isinstance(f, DenseConfig):
                mlp = {"kind": "dense", "ff": f.ff}
            elif f is not None:
                mlp = {"kind": "moe", "expert": {"ff": f.ff}, "router": {"experts": f.experts, "top": f.top}}
            layers.append({"type": layer.type, "mixer": mixer, "mlp": mlp})
        d = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps},
             "embedding": {"scale": self.embedding_scale}, "logit_scale": self.logit_scale, "layers": layers}
        if self.logit_softcap is not None:
            d["logit_softcap"] = self.logit_softcap
        if self.loop is not None:
            d["loop"] = {"start": self.loop.start, "stop": self.loop.stop, "times": self.loop.times}
        if self.torch_dtype:
            d["torch_dtype"] = self.torch_dtype
        return d
