"""Typed configuration of the Semesun decoder, read from config.json.

A Semesun model is a list of pre-norm layers with two mixers: "attention" (queries and keys with a weighted norm per head, no
rotation, a learned bias by distance, a sliding window behind which the first tokens stay visible, values mixed with those of the
first mixing layer) and "mamba2" (state-space duality).  The feed-forward is dense (the square of relu), or a mixture of experts
chosen by groups from a softmax over all experts, identity experts among them; or absent.  Every size and every constant that can
differ between models is a field here; the parts and kernels carry none.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple

from .base import ConfigError
from .turudra import _get

NAME = "Semesun"


def _flag(d, key, where) -> bool:
    v = d.get(key, False)
    if v is None:
        return False
    if not isinstance(v, bool):
        raise ConfigError(f"config.json: {where}.{key} must be true or false")
    return v


@dataclass(frozen=True)
class AttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    bias_max: Optional[float]          # distance from which on the bias is constant; None: no bias
    window: Optional[int]              # None: every earlier key is visible
    keep_first: int                    # first positions of a sequence that stay visible behind the window
    v_mix: bool
    kind: str = "attention"

    @classmethod
    def from_dict(cls, d, where):
        heads = _get(d, "heads", int, where)
        mask = _get(d, "mask", dict, where, None)
        dim = _get(d, "dim", int, where)
        c = cls(heads=heads, kv_heads=_get(d, "kv_heads", int, where, heads), dim=dim, vdim=_get(d, "vdim", int, where, dim),
                scale=_get(d, "scale", float, where), bias_max=_get(d, "bias_max", float, where, None),
                window=None if mask is None else _get(mask, "size", int, where + ".mask"),
                keep_first=0 if mask is None else _get(mask, "keep_first", int, where + ".mask", 0), v_mix=_flag(d, "v_mix", where))
        if min(c.heads, c.kv_heads, c.dim, c.vdim) < 1 or c.heads % c.kv_heads:
            raise ConfigError(f"config.json: {where}: sizes must be positive and heads a multiple of kv_heads")
        if not c.scale > 0:
            raise ConfigError(f"config.json: {where}.scale must be positive")
        if c.bias_max is not None and not c.bias_max > 1:
            raise ConfigError(f"config.json: {where}.bias_max must be above one")
        if c.window is not None and c.window < 1:
            raise ConfigError(f"config.json: {where}.mask.size must be positive")
        return c

    def to_dict(self):
        d = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale, "v_mix": self.v_mix}
        if self.bias_max is not None:
            d["bias_max"] = self.bias_max
        if self.window is not None:
            d["mask"] = {"size": self.window, "keep_first": self.keep_first}
        return d


@dataclass(frozen=True)
class MambaConfig:
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int                          # taps of the convolution
    norm_groups: int
    kind: str = "mamba2"

    @classmethod
    def from_dict(cls, d, where):
        c = cls(heads=_get(d, "heads", int, where), vdim=_get(d, "vdim", int, where), state=_get(d, "state", int, where),
                groups=_get(d, "groups", int, where, 1), conv=_get(d, "conv", int, where), norm_groups=_get(d, "norm_groups", int, where, 1))
        if min(c.heads, c.vdim, c.state, c.groups, c.conv, c.norm_groups) < 1:
            raise ConfigError(f"config.json: {where}: sizes must be positive")
        if c.heads % c.groups or (c.heads * c.vdim) % c.norm_groups:
            raise ConfigError(f"config.json: {where}: groups must divide heads, and norm_groups heads times vdim")
        return c

    def to_dict(self):
        return {"heads": self.heads, "vdim": self.vdim, "state": self.state, "groups": self.groups, "conv": self.conv,
                "norm_groups": self.norm_groups}


@dataclass(frozen=True)
class DenseConfig:
    ff: int
    kind: str = "dense"

    @classmethod
    def from_dict(cls, d, where):
        c = cls(ff=_get(d, "ff", int, where))
        if c.ff < 1:
            raise ConfigError(f"config.json: {where}.ff must be positive")
        return c

    def to_dict(self):
        return {"kind": "dense", "ff": self.ff}


@dataclass(frozen=True)
class ExpertsConfig:
    experts: int
    identity: int                      # outputs of the router behind the experts whose output is the input itself
    top: int
    group_count: int
    group_keep: int
    scale: float
    ff: int
    limit: float
    kind: str = "moe"

    @classmethod
    def from_dict(cls, d, where):
        r, e = _get(d, "router", dict, where), _get(d, "expert", dict, where)
        rw = where + ".router"
        g = _get(r, "groups", dict, rw, None)
        c = cls(experts=_get(r, "experts", int, rw), identity=_get(r, "identity", int, rw, 0), top=_get(r, "top", int, rw),
                group_count=1 if g is None else _get(g, "count", int, rw + ".groups"), group_keep=1 if g is None else _get(g, "keep", int, rw + ".groups"),
                scale=_get(r, "scale", float, rw, 1.0), ff=_get(e, "ff", int, where + ".expert"), limit=_get(e, "limit", float, where + ".expert"))
        if c.ff < 1 or c.experts < 1 or not c.limit > 0:
            raise ConfigError(f"config.json: {where}: experts, expert.ff and expert.limit must be positive")
        outputs = c.experts + c.identity
        if c.group_count < 1 or outputs % c.group_count or not (1 <= c.group_keep <= c.group_count):
            raise ConfigError(f"config.json: {rw}.groups: count must divide the {outputs} outputs of the router and keep be at most count")
        if not (1 <= c.top <= c.group_keep * (outputs // c.group_count)):
            raise ConfigError(f"config.json: {rw}.top must be at least 1 and at most the outputs of the kept groups")
        return c

    def to_dict(self):
        return {"kind": "moe", "router": {"experts": self.experts, "identity": self.identity, "top": self.top, "scale": self.scale,
                                          "groups": {"count": self.group_count, "keep": self.group_keep}},
                "expert": {"ff": self.ff, "limit": self.limit}}


@dataclass(frozen=True)
class LayerConfig:
    mixer: Any                       # AttentionConfig | MambaConfig
    mlp: Any                         # DenseConfig | ExpertsConfig | None


@dataclass(frozen=True)
class SemesunConfig:
    architecture: str
    vocab: int
    width: int
    layers: Tuple[LayerConfig, ...]
    norm_eps: float
    torch_dtype: str = "bfloat16"

    MIXERS = {"attention": AttentionConfig, "mamba2": MambaConfig}
    MLPS = {"dense": DenseConfig, "moe": ExpertsConfig}

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "SemesunConfig":
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
            mlp = None
            if lr.get("mlp"):
                mk = _get(lr["mlp"], "kind", str, where + ".mlp", "dense")
                if mk not in cls.MLPS:
                    raise ConfigError(f"config.json: {where}.mlp.kind '{mk}' is not supported (known: {', '.join(sorted(cls.MLPS))})")
                mlp = cls.MLPS[mk].from_dict(lr["mlp"], where + ".mlp")
            layers.append(LayerConfig(mixer, mlp))
        cfg = cls(architecture=NAME, vocab=_get(d, "vocab", int, top), width=_get(d, "width", int, top), layers=tuple(layers),
                  norm_eps=_get(_get(d, "norm", dict, top), "eps", float, "norm"), torch_dtype=_get(d, "torch_dtype", str, top, "bfloat16"))
        if cfg.vocab < 1 or cfg.width < 1:
            raise ConfigError("config.json: vocab and width must be positive")
        mixing = [i for i, l in enumerate(layers) if l.mixer.kind == "attention" and l.mixer.v_mix]
        for i in mixing[1:]:
            a, b = layers[mixing[0]].mixer, layers[i].mixer
            if a.kv_heads * a.vdim != b.kv_heads * b.vdim:
                raise ConfigError(f"config.json: layers[{i}] mixes its values with those of layers[{mixing[0]}], which have another size")
        return cfg

    def to_dict(self) -> dict:
        """The config.json of this configuration."""
        return {"architecture": NAME, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
                "layers": [{"type": l.mixer.kind, "mixer": l.mixer.to_dict(), "mlp": None if l.mlp is None else l.mlp.to_dict()}
                           for l in self.layers],
                "torch_dtype": self.torch_dtype}
