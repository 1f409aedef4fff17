"""Typed configuration of the Mezinex decoder, read from its own ``config.json``.

The file lists the layers one by one; each names its mixer (``type``: ``mamba2``, ``latent_attention`` or ``rglru``) with
the mixer's sizes, and its feed-forward (``mlp``: ``dense``, or null for none).  A stretch of layers may run several
times in a row (``loop``).  The residual stream may have several rows per token (``streams``; absent: a plain residual
sum), and the embedding a table of hashed token pairs (``embedding.bigram``).  Every size and every constant that may
differ between models of the design is read from the file; nothing is filled in.

    {"architecture": "Mezinex", "vocab": V, "width": W, "norm": {"eps": e}, "streams": s, "logit_scale": c,
     "embedding": {"bigram": {"buckets": b, "mul_prev": m, "mul_cur": n} | absent},
     "loop": {"start": a, "stop": b, "times": n} | absent,
     "layers": [{"type": "mamba2", "mixer": {"heads", "vdim", "state", "groups", "norm_groups", "conv"},
                 "mlp": {"kind": "dense", "ff"} | null},
                {"type": "latent_attention",
                 "mixer": {"heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank", "scale", "rot": {"dims", "base"}}, "mlp": ...},
                {"type": "rglru", "mixer": {"width", "blocks", "conv"}, "mlp": ...}, ...]}
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Optional, Tuple

from .labolix_config import RotaryConfig, _rotary
from .mozutar_config import DenseFfConfig, LoopConfig
from .rirulix_config import _need
from .text_config import ConfigError


@dataclass(frozen=True)
class StateSpaceMixerConfig:
    heads: int
    vdim: int
    state: int
    groups: int
    norm_groups: int
    conv: int


@dataclass(frozen=True)
class GatedLatentMixerConfig:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    q_rank: int
    scale: float
    rot: Optional[RotaryConfig]


@dataclass(frozen=True)
class RecurrentMixerConfig:
    width: int
    blocks: int
    conv: int


@dataclass(frozen=True)
class PairTableConfig:
    buckets: int
    mul_prev: int
    mul_cur: int


@dataclass(frozen=True)
class MezinexLayerConfig:
    type: str
    mixer: Any
    mlp: Optional[DenseFfConfig]


def _mixer(kind: str, m: Dict[str, Any], where: str):
    need = lambda key: _need(m, key, where)
    if kind == "mamba2":
        mixer = StateSpaceMixerConfig(**{k: int(need(k)) for k in ("heads", "vdim", "state", "groups", "norm_groups", "conv")})
        if mixer.groups < 1 or mixer.heads % mixer.groups:
            raise ConfigError(f"config.json: {where}: {mixer.heads} heads cannot share {mixer.groups} groups")
        if mixer.norm_groups < 1 or mixer.heads * mixer.vdim % mixer.norm_groups:
            raise ConfigError(f"config.json: {where}: {mixer.heads * mixer.vdim} channels cannot be normed in {mixer.norm_groups} equal parts")
        return mixer
    if kind == "latent_attention":
        mixer = GatedLatentMixerConfig(scale=float(need("scale")), rot=_rotary(m, where, None),
                                       **{k: int(need(k)) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank")})
        if mixer.rot is not None and mixer.rot.dims > mixer.rot_dim:
            raise ConfigError(f"config.json: {where}.rot.dims {mixer.rot.dims} exceeds rot_dim {mixer.rot_dim}")
        return mixer
    if kind == "rglru":
        mixer = RecurrentMixerConfig(**{k: int(need(k)) for k in ("width", "blocks", "conv")})
        if mixer.blocks < 1 or mixer.width % mixer.blocks:
            raise ConfigError(f"config.json: {where}: {mixer.width} channels cannot be cut into {mixer.blocks} equal blocks")
        return mixer
    raise ConfigError(f"config.json: {where[:-len('.mixer')]} has the unknown type {kind!r}; known: latent_attention, mamba2, rglru")


@dataclass(frozen=True)
class MezinexConfig:
    vocab_size: int
    hidden_size: int
    norm_eps: float
    logit_scale: float
    layers: Tuple[MezinexLayerConfig, ...]
    streams: Optional[int] = None              # None: a plain residual sum
    pairs: Optional[PairTableConfig] = None
    loop: Optional[LoopConfig] = None
    eos_token_id: Optional[int] = None

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    def layer_runs(self):
        """The layers in the order they run."""
        n, lp = len(self.layers), self.loop
        if lp is None:
            return list(range(n))
        return list(range(lp.start)) + list(range(lp.start, lp.stop)) * lp.times + list(range(lp.stop, n))

    @classmethod
    def from_dict(cls, raw: Dict[str, Any]) -> "MezinexConfig":
        norm = _need(raw, "norm", "the model")
        layers = []
        for i, entry in enumerate(_need(raw, "layers", "the model")):
            where = f"layers[{i}]"
            kind = _need(entry, "type", where)
            mixer = _mixer(kind, _need(entry, "mixer", where), where + ".mixer")
            mlp = entry.get("mlp")
            if mlp is not None:
                if mlp.get("kind", "dense") != "dense":
                    raise ConfigError(f"config.json: {where}.mlp has the unknown kind {mlp.get('kind')!r}; known: dense")
                mlp = DenseFfConfig(ff=int(_need(mlp, "ff", where + ".mlp")))
            layers.append(MezinexLayerConfig(kind, mixer, mlp))
        loop = raw.get("loop")
        if loop is not None:
            loop = LoopConfig(int(_need(loop, "start", "loop")), int(_need(loop, "stop", "loop")), int(_need(loop, "times", "loop")))
            if not 0 <= loop.start < loop.stop <= len(layers) or loop.times < 1:
                raise ConfigError(f"config.json: loop runs layers {loop.start} .. {loop.stop - 1} {loop.times} times; the model has "
                                  f"{len(layers)} layers")
        pairs = (raw.get("embedding") or {}).get("bigram")
        if pairs is not None:
            pairs = PairTableConfig(**{k: int(_need(pairs, k, "embedding.bigram")) for k in ("buckets", "mul_prev", "mul_cur")})
            if pairs.buckets < 1:
                raise ConfigError(f"config.json: embedding.bigram.buckets must be positive, got {pairs.buckets}")
        streams, eos, scale = raw.get("streams"), raw.get("eos_token_id"), raw.get("logit_scale")
        if streams is not None and not 1 <= int(streams) <= 16:
            raise ConfigError(f"config.json: streams must be 1 to 16, got {streams}")
        return cls(vocab_size=int(_need(raw, "vocab", "the model")), hidden_size=int(_need(raw, "width", "the model")),
                   norm_eps=float(_need(norm, "eps", "norm")), logit_scale=1.0 if scale is None else float(scale), layers=tuple(layers),
                   streams=None if streams is None else int(streams), pairs=pairs, loop=loop, eos_token_id=None if eos is None else int(eos))
