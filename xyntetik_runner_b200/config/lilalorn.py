"""Typed configuration of the Lilalorn decoder, read from config.json.

A Lilalorn model is a list of pre-norm layers whose sublayers' outputs are multiplied by a constant before they join the stream.  Two
mixers: "parallel" (softmax attention with rotated queries and keys beside retention, each with a scale) and "gla" (gated linear
attention: a decay per key channel and token).  The feed-forward is a mixture of ungated experts (the square of relu) with a shared
expert under a gate; or absent.  A layer may use another layer's tensors (`weights_of`), with a cache and a state of its own.  Every
size and every constant that can differ between models is a field here; the parts and kernels carry none.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple

from .base import ConfigError
from .turudra import _get

NAME = "Lilalorn"


@dataclass(frozen=True)
class WavelengthScaling:
    """Frequencies of wavelengths beyond original / low divided by `factor`, below original / high kept, blended between."""
    factor: float
    low: float
    high: float
    original: float

    @classmethod
    def from_dict(cls, d, where):
        c = cls(*(_get(d, k, float, where) for k in ("factor", "low", "high", "original")))
        if not (c.factor > 0 and c.original > 0 and c.low >= 0 and c.high > 0 and c.high >= c.low):
            raise ConfigError(f"config.json: {where}: factor, original and high must be positive, low not negative and at most high")
        return c

    def to_dict(self):
        return {"factor": self.factor, "low": self.low, "high": self.high, "original": self.original}


@dataclass(frozen=True)
class RotationConfig:
    base: float
    dims: int                          # leading elements of a query/key head that are rotated, element i with i + dims/2
    scaling: Optional[WavelengthScaling]

    @classmethod
    def from_dict(cls, d, where):
        if d is None:
            return cls(10000.0, 0, None)
        sc = d.get("scaling") if isinstance(d, Mapping) else None
        c = cls(base=_get(d, "base", float, where), dims=_get(d, "dims", int, where),
                scaling=WavelengthScaling.from_dict(sc, where + ".scaling") if sc else None)
        if c.dims % 2 or not c.base > 0:
            raise ConfigError(f"config.json: {where}: dims must be even and base positive")
        return c

    def to_dict(self):
        d = {"base": self.base, "dims": self.dims}
        if self.scaling is not None:
            d["scaling"] = self.scaling.to_dict()
        return d


@dataclass(frozen=True)
class SoftmaxSideConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: RotationConfig

    @classmethod
    def from_dict(cls, d, where):
        heads, dim = _get(d, "heads", int, where), _get(d, "dim", int, where)
        c = cls(heads=heads, kv_heads=_get(d, "kv_heads", int, where, heads), dim=dim, vdim=_get(d, "vdim", int, where, dim),
                scale=_get(d, "scale", float, where), rot=RotationConfig.from_dict(d.get("rot"), where + ".rot"))
        if min(c.heads, c.kv_heads, c.dim, c.vdim) < 1 or c.heads % c.kv_heads:
            raise ConfigError(f"config.json: {where}: sizes must be positive and heads a multiple of kv_heads")
        if c.rot.dims > c.dim:
            raise ConfigError(f"config.json: {where}.rot.dims exceeds dim")
        return c

    def to_dict(self):
        return {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale, "rot": self.rot.to_dict()}


@dataclass(frozen=True)
class RetentionConfig:
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]

    @classmethod
    def from_dict(cls, d, where):
        raw = d.get("decay") if isinstance(d, Mapping) else None
        if not isinstance(raw, list) or not all(isinstance(v, (int, float)) and not isinstance(v, bool) for v in raw):
            raise ConfigError(f"config.json: {where}.decay must be a list of numbers, one per head")
        dim = _get(d, "dim", int, where)
        c = cls(heads=_get(d, "heads", int, where), dim=dim, vdim=_get(d, "vdim", int, where, dim), decay=tuple(float(v) for v in raw))
        if min(c.heads, c.dim, c.vdim) < 1 or len(c.decay) != c.heads:
            raise ConfigError(f"config.json: {where}: sizes must be positive and decay hold one number per head")
        return c

    def to_dict(self):
        return {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "decay": list(self.decay)}


@dataclass(frozen=True)
class ParallelConfig:
    left: SoftmaxSideConfig
    right: RetentionConfig
    left_scale: float
    right_scale: float
    kind: str = "parallel"

    @classmethod
    def from_dict(cls, d, where):
        return cls(left=SoftmaxSideConfig.from_dict(_get(d, "left", dict, where), where + ".left"),
                   right=RetentionConfig.from_dict(_get(d, "right", dict, where), where + ".right"),
                   left_scale=_get(d, "left_scale", float, where, 1.0), right_scale=_get(d, "right_scale", float, where, 1.0))

    def to_dict(self):
        return {"left": self.left.to_dict(), "right": self.right.to_dict(), "left_scale": self.left_scale, "right_scale": self.right_scale}


@dataclass(frozen=True)
class GatedLinearConfig:
    heads: int
    dim: int
    vdim: int
    tau: float                         # the decay is the tau-th root of a sigmoid
    kind: str = "gla"

    @classmethod
    def from_dict(cls, d, where):
        dim = _get(d, "dim", int, where)
        c = cls(heads=_get(d, "heads", int, where), dim=dim, vdim=_get(d, "vdim", int, where, dim), tau=_get(d, "tau", float, where))
        if min(c.heads, c.dim, c.vdim) < 1 or not c.tau > 0:
            raise ConfigError(f"config.json: {where}: sizes and tau must be positive")
        return c

    def to_dict(self):
        return {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "tau": self.tau}


@dataclass(frozen=True)
class ExpertsConfig:
    experts: int
    top: int
    ff: int
    shared_ff: Optional[int]           # None: no shared expert
    kind: str = "moe"

    @classmethod
    def from_dict(cls, d, where):
        kind = _get(d, "kind", str, where, "moe")
        if kind != "moe":
            raise ConfigError(f"config.json: {where}.kind '{kind}' is not supported (known: moe)")
        r, sh = _get(d, "router", dict, where), _get(d, "shared", dict, where, None)
        c = cls(experts=_get(r, "experts", int, where + ".router"), top=_get(r, "top", int, where + ".router"),
                ff=_get(_get(d, "expert", dict, where), "ff", int, where + ".expert"),
                shared_ff=None if sh is None else _get(sh, "ff", int, where + ".shared"))
        if c.ff < 1 or (c.shared_ff is not None and c.shared_ff < 1) or not (1 <= c.top <= c.experts):
            raise ConfigError(f"config.json: {where}: expert.ff and shared.ff must be positive and 1 <= router.top <= router.experts")
        return c

    def to_dict(self):
        d = {"kind": "moe", "router": {"experts": self.experts, "top": self.top}, "expert": {"ff": self.ff}}
        if self.shared_ff is not None:
            d["shared"] = {"ff": self.shared_ff}
        return d


@dataclass(frozen=True)
class LayerConfig:
    mixer: Any                       # ParallelConfig | GatedLinearConfig
    mlp: Optional[ExpertsConfig]
    weights_of: Optional[int] = None   # the layer whose tensors this one uses


@dataclass(frozen=True)
class LilalornConfig:
    architecture: str
    vocab: int
    width: int
    layers: Tuple[LayerConfig, ...]
    norm_eps: float
    residual_mult: float
    logit_scale: float
    torch_dtype: str = "bfloat16"

    MIXERS = {"parallel": ParallelConfig, "gla": GatedLinearConfig}

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "LilalornConfig":
        top = "top level"
        raw = d.get("layers")
        if not isinstance(raw, list) or not raw:
            raise ConfigError("config.json: 'layers' must be a list with at least one layer")
        layers = []
        for i, lr in enumerate(raw):
            where = f"layers[{i}]"
            kind = _get(lr, "type", str, where)
            if kind not in cls.MIXERS:
                raise ConfigError(f"config.json: {where}.type '{kind}' is not supported (known: {', '.join(sorted(cls.MIXERS))})")
            mixer = cls.MIXERS[kind].from_dict(_get(lr, "mixer", dict, where), where + ".mixer")
            mlp = ExpertsConfig.from_dict(lr["mlp"], where + ".mlp") if lr.get("mlp") else None
            layers.append(LayerConfig(mixer, mlp, _get(lr, "weights_of", int, where, None)))
        for i, lay in enumerate(layers):
            j = lay.weights_of
            if j is None:
                continue
            if not (0 <= j < len(layers)) or j == i:
                raise ConfigError(f"config.json: layers[{i}].weights_of must name another layer")
            if (lay.mixer, lay.mlp) != (layers[j].mixer, layers[j].mlp):
                raise ConfigError(f"config.json: layers[{i}] uses the tensors of layers[{j}] but differs from it")
        cfg = cls(architecture=NAME, vocab=_get(d, "vocab", int, top), width=_get(d, "width", int, top), layers=tuple(layers),
                  norm_eps=_get(_get(d, "norm", dict, top), "eps", float, "norm"), residual_mult=_get(d, "residual_mult", float, top, 1.0),
                  logit_scale=_get(d, "logit_scale", float, top, 1.0), torch_dtype=_get(d, "torch_dtype", str, top, "bfloat16"))
        if cfg.vocab < 1 or cfg.width < 1:
            raise ConfigError("config.json: vocab and width must be positive")
        for i in range(len(layers)):
            cfg.owner(i)
        return cfg

    def owner(self, i: int) -> int:
        """The layer whose tensors layer i uses: itself, or the end of its chain of `weights_of`."""
        first, steps = i, 0
        while self.layers[i].weights_of is not None:
            i, steps = self.layers[i].weights_of, steps + 1
            if steps > len(self.layers):
                raise ConfigError(f"config.json: layers[{first}].weights_of leads back to itself")
        return i

    def to_dict(self) -> dict:
        """The config.json of this configuration."""
        layers = []
        for l in self.layers:
            e = {"type": l.mixer.kind, "mixer": l.mixer.to_dict(), "mlp": None if l.mlp is None else l.mlp.to_dict()}
            if l.weights_of is not None:
                e["weights_of"] = l.weights_of
            layers.append(e)
        return {"architecture": NAME, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps}, "residual_mult": self.residual_mult,
                "logit_scale": self.logit_scale, "layers": layers, "torch_dtype": self.torch_dtype}
