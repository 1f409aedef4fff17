"""Typed configuration of the Sudilorn decoder, read from its own ``config.json``.

The file lists the layers one by one; each names its mixer (``type``: ``attention`` -- differential attention with a
short convolution, query/key norm and an output gate -- or ``parallel`` -- window attention beside a gated delta rule)
with the mixer's sizes and constants, and its feed-forward (``mlp``: routed experts, or null for none).  Every size and
every constant that may differ between models of the design is read from the file.

    {"architecture": "Sudilorn", "vocab": V, "width": W, "norm": {"eps": e}, "residual_mult": m,
     "layers": [{"type": "attention",
                 "mixer": {"heads", "kv_heads", "dim", "vdim", "conv" | absent, "diff", "scale", "mask": {"size"} | absent, "rot": ROT},
                 "mlp": {"kind": "moe", "expert": {"ff"}, "router": {"experts", "top", "groups": {"count", "keep"}}} | null},
                {"type": "parallel",
                 "mixer": {"left": {"heads", "kv_heads", "dim", "vdim", "scale", "mask": {"size", "keep_first"} | absent, "rot": ROT},
                           "right": {"heads", "kv_heads", "dim", "vdim", "conv"}, "left_scale", "right_scale"}, ...}, ...]}

    ROT: {"dims", "base", "scaling": {"factor", "original", "fast", "slow"} | absent} | absent
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Optional, Tuple

from .rirulix_config import _need
from .text_config import ConfigError


@dataclass(frozen=True)
class SudilornRotary:
    dims: int
    base: float
    scaling: Optional[Tuple[Tuple[str, float], ...]] = None      # (name, value) of factor, original, fast, slow

    def scaling_dict(self) -> Optional[Dict[str, Any]]:
        return None if self.scaling is None else dict(self.scaling, kind="ramp")


@dataclass(frozen=True)
class SoftmaxMixerConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: Optional[int]
    keep_first: int
    rot: Optional[SudilornRotary]
    conv: int = 0               # the differential attention's convolution (0: none) and constant
    diff: float = 0.0


@dataclass(frozen=True)
class DeltaMixerConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int


@dataclass(frozen=True)
class SudilornParallelConfig:
    left: SoftmaxMixerConfig
    right: DeltaMixerConfig
    left_scale: float
    right_scale: float


@dataclass(frozen=True)
class SudilornRoutedFf:
    experts: int
    top: int
    ff: int
    groups: int
    keep: int


@dataclass(frozen=True)
class SudilornLayerConfig:
    type: str
    mixer: Any
    mlp: Optional[SudilornRoutedFf]


def _heads(m: Dict[str, Any], where: str) -> Tuple[int, int]:
    heads = int(_need(m, "heads", where))
    kv = int(m["kv_heads"]) if m.get("kv_heads") else heads
    if heads < 1 or kv < 1 or heads % kv:
        raise ConfigError(f"config.json: {where}: {heads} heads cannot share {kv} kv_heads")
    return heads, kv


def _taps(m: Dict[str, Any], where: str, optional: bool = False) -> int:
    taps = int(m.get("conv") or 0) if optional else int(_need(m, "conv", where))
    if not (0 if optional else 1) <= taps <= 16:
        raise ConfigError(f"config.json: {where}.conv takes 1 to 16 taps, got {taps}")
    return taps


def _rotary(rot: Optional[Dict[str, Any]], dim: int, where: str) -> Optional[SudilornRotary]:
    if not rot or not rot.get("dims"):
        return None
    dims = int(rot["dims"])
    if dims < 0 or dims % 2 or dims > dim:
        raise ConfigError(f"config.json: {where}.dims must be even and at most dim {dim}, got {dims}")
    scaling = rot.get("scaling")
    if scaling is not None:
        scaling = tuple((key, float(_need(scaling, key, where + ".scaling"))) for key in ("factor", "original", "fast", "slow"))
    return SudilornRotary(dims=dims, base=float(_need(rot, "base", where)), scaling=scaling)


def _softmax(m: Dict[str, Any], where: str, differential: bool) -> SoftmaxMixerConfig:
    heads, kv = _heads(m, where)
    dim = int(_need(m, "dim", where))
    mask = m.get("mask") or {}
    window = int(mask["size"]) if mask.get("size") else None
    if window is not None and window < 1:
        raise ConfigError(f"config.json: {where}.mask.size must be at least 1, got {window}")
    keep = int(mask.get("keep_first") or 0)
    if keep < 0:
        raise ConfigError(f"config.json: {where}.mask.keep_first must not be negative, got {keep}")
    return SoftmaxMixerConfig(heads=heads, kv_heads=kv, dim=dim, vdim=int(m["vdim"]) if m.get("vdim") else dim, scale=float(_need(m, "scale", where)),
                              window=window, keep_first=keep if window else 0, rot=_rotary(m.get("rot"), dim, where + ".rot"),
                              conv=_taps(m, where, optional=True) if differential else 0, diff=float(_need(m, "diff", where)) if differential else 0.0)


def _delta(m: Dict[str, Any], where: str) -> DeltaMixerConfig:
    heads, kv = _heads(m, where)
    return DeltaMixerConfig(heads=heads, kv_heads=kv, dim=int(_need(m, "dim", where)), vdim=int(_need(m, "vdim", where)), conv=_taps(m, where))


def _mlp(mlp: Optional[Dict[str, Any]], where: str) -> Optional[SudilornRoutedFf]:
    if mlp is None:
        return None
    kind = _need(mlp, "kind", where)
    if kind != "moe":
        raise ConfigError(f"config.json: {where} has the unknown kind {kind!r}; known: moe")
    r = _need(mlp, "router", where)
    experts, top = int(_need(r, "experts", where + ".router")), int(_need(r, "top", where + ".router"))
    groups = r.get("groups") or {}
    count = int(groups.get("count") or 1)
    keep = int(groups.get("keep") or count)
    if experts < 1 or count < 1 or experts % count or not 1 <= keep <= count:
        raise ConfigError(f"config.json: {where}.router: {experts} experts do not form {count} equal groups of which {keep} are kept")
    if not 1 <= top <= keep * (experts // count):
        raise ConfigError(f"config.json: {where}.router: {top} choices cannot come from {keep} groups of {experts // count}")
    return SudilornRoutedFf(experts=experts, top=top, ff=int(_need(_need(mlp, "expert", where), "ff", where + ".expert")), groups=count, keep=keep)


@dataclass(frozen=True)
class SudilornConfig:
    vocab_size: int
    hidden_size: int
    norm_eps: float
    residual_mult: float
    layers: Tuple[SudilornLayerConfig, ...]
    eos_token_id: Optional[int] = None

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @classmethod
    def from_dict(cls, raw: Dict[str, Any]) -> "SudilornConfig":
        layers = []
        for i, entry in enumerate(_need(raw, "layers", "the model")):
            where = f"layers[{i}]"
            kind = _need(entry, "type", where)
            m = _need(entry, "mixer", where)
            if kind == "attention":
                mixer = _softmax(m, where + ".mixer", True)
            elif kind == "parallel":
                mixer = SudilornParallelConfig(_softmax(_need(m, "left", where + ".mixer"), where + ".mixer.left", False),
                                               _delta(_need(m, "right", where + ".mixer"), where + ".mixer.right"),
                                               float(m.get("left_scale", 1.0)), float(m.get("right_scale", 1.0)))
            else:
                raise ConfigError(f"config.json: {where} has the unknown type {kind!r}; known: attention, parallel")
            layers.append(SudilornLayerConfig(kind, mixer, _mlp(entry.get("mlp"), where + ".mlp")))
        eos = raw.get("eos_token_id")
        return cls(vocab_size=int(_need(raw, "vocab", "the model")), hidden_size=int(_need(raw, "width", "the model")),
                   norm_eps=float(_need(_need(raw, "norm", "the model"), "eps", "norm")), residual_mult=float(raw.get("residual_mult", 1.0)),
                   layers=tuple(layers), eos_token_id=None if eos is None else int(eos))
