"""Typed configuration of the Bifatar decoder, read from ``config.json``.

The file names the design under ``"architecture"`` and gives every size and
constant: ``layers[i]`` holds ``type`` (which mixer: ``mamba2``, ``parallel`` or
``attention``), ``mixer`` (its sizes and constants) and ``mlp`` (a dense
feed-forward, or null); ``norm.eps``, ``vocab`` and ``width`` are global.  A key
the design needs and the file lacks is an error that names its place.  What a
file may leave out, with what that means: a mixer's ``rot`` (nothing is
rotated), ``mask`` (every earlier key is visible), ``softcap`` (scores are not
capped), ``v_mix`` (false), ``conv`` (one tap), ``groups`` and ``norm_groups``
(1), a recurrence's ``kv_heads`` (as many as heads) and ``rank`` / ``gate_rank``
(the checkpoint's tensors give them), the branch scales (1), a layer's ``mlp``
(none).  A key this reader does not know changes nothing it computes; it is
kept in ``unknown_keys`` and named in one warning.
"""

from __future__ import annotations

import copy
import warnings
from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional

from .qwen2 import ConfigError


def _need(d: Dict[str, Any], key: str, where: str):
    if not isinstance(d, dict) or key not in d:
        raise ConfigError(f"config.json: {where} misses {key!r}")
    return d[key]


def _only(d: Dict[str, Any], known, where: str, unknown: List[str]) -> None:
    if not isinstance(d, dict):
        raise ConfigError(f"config.json: {where} must be an object")
    unknown.extend(f"{where}.{k}" for k in sorted(set(d) - set(known)))


def _optional(d: Dict[str, Any], key: str, kind, default=None):
    return default if d.get(key) is None else kind(d[key])


@dataclass
class RotationConfig:
    dims: int
    base: float

    @classmethod
    def from_dict(cls, r: Optional[Dict[str, Any]], dim: int, where: str, unknown: List[str]) -> Optional["RotationConfig"]:
        if r is None:
            return None
        _only(r, ("dims", "base"), where, unknown)
        c = cls(int(_need(r, "dims", where)), float(_need(r, "base", where)))
        if c.dims < 0 or c.dims % 2 or c.dims > dim or not c.base > 0:
            raise ConfigError(f"config.json: {where}: dims must be even and at most dim, base positive")
        return c if c.dims else None

    def to_dict(self) -> Dict[str, Any]:
        return {"base": self.base, "dims": self.dims}

    def key(self) -> str:
        return f"rot{self.dims}@{self.base!r}"


@dataclass
class Mamba2Config:
    """A state-space mixer with one decay per head (``layers[i].mixer`` of type ``mamba2``)."""
    heads: int
    vdim: int
    state: int
    groups: int
    norm_groups: int
    conv: int

    @classmethod
    def from_dict(cls, m: Dict[str, Any], where: str, unknown: List[str]) -> "Mamba2Config":
        _only(m, ("heads", "vdim", "state", "groups", "norm_groups", "conv"), where, unknown)
        c = cls(heads=int(_need(m, "heads", where)), vdim=int(_need(m, "vdim", where)), state=int(_need(m, "state", where)),
                groups=_optional(m, "groups", int, 1), norm_groups=_optional(m, "norm_groups", int, 1), conv=_optional(m, "conv", int, 1))
        if min(c.heads, c.vdim, c.state, c.groups, c.norm_groups, c.conv) <= 0:
            raise ConfigError(f"config.json: {where}: sizes must be positive")
        if c.heads % c.groups or (c.heads * c.vdim) % c.norm_groups:
            raise ConfigError(f"config.json: {where}: heads must be a multiple of groups, and heads * vdim of norm_groups")
        return c

    def to_dict(self) -> Dict[str, Any]:
        return {"conv": self.conv, "groups": self.groups, "heads": self.heads, "norm_groups": self.norm_groups, "state": self.state,
                "vdim": self.vdim}


@dataclass
class NormedAttentionConfig:
    """Softmax attention whose q and k are normed over their whole projections (``mixer.left``)."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: Optional[RotationConfig]

    @classmethod
    def from_dict(cls, m: Dict[str, Any], where: str, unknown: List[str]) -> "NormedAttentionConfig":
        _only(m, ("heads", "kv_heads", "dim", "vdim", "scale", "rot"), where, unknown)
        dim = int(_need(m, "dim", where))
        c = cls(heads=int(_need(m, "heads", where)), kv_heads=int(_need(m, "kv_heads", where)), dim=dim,
                vdim=_optional(m, "vdim", int, dim), scale=float(_need(m, "scale", where)),
                rot=RotationConfig.from_dict(m.get("rot"), dim, f"{where}.rot", unknown))
        if min(c.heads, c.kv_heads, c.dim, c.vdim) <= 0 or c.heads % c.kv_heads or not c.scale > 0:
            raise ConfigError(f"config.json: {where}: sizes and scale must be positive and heads a multiple of kv_heads")
        return c

    def to_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {"dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads, "scale": self.scale, "vdim": self.vdim}
        if self.rot is not None:
            d["rot"] = self.rot.to_dict()
        return d


@dataclass
class DeltaRuleConfig:
    """The gated delta rule (``mixer.right``)."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int
    rank: Optional[int] = None
    gate_rank: Optional[int] = None

    @classmethod
    def from_dict(cls, m: Dict[str, Any], where: str, unknown: List[str]) -> "DeltaRuleConfig":
        _only(m, ("heads", "kv_heads", "dim", "vdim", "conv", "rank", "gate_rank"), where, unknown)
        heads, dim, rank = int(_need(m, "heads", where)), int(_need(m, "dim", where)), _optional(m, "rank", int)
        c = cls(heads=heads, kv_heads=_optional(m, "kv_heads", int, heads), dim=dim, vdim=_optional(m, "vdim", int, dim),
                conv=_optional(m, "conv", int, 1), rank=rank, gate_rank=_optional(m, "gate_rank", int, rank))
        if min(c.heads, c.kv_heads, c.dim, c.vdim, c.conv, 1 if c.rank is None else c.rank,
               1 if c.gate_rank is None else c.gate_rank) <= 0 or c.heads % c.kv_heads:
            raise ConfigError(f"config.json: {where}: sizes must be positive and heads a multiple of kv_heads")
        return c

    def to_dict(self) -> Dict[str, Any]:
        d = {"conv": self.conv, "dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads, "vdim": self.vdim}
        if self.rank is not None:
            d["rank"] = self.rank
        if self.gate_rank is not None:
            d["gate_rank"] = self.gate_rank
        return d


@dataclass
class ParallelConfig:
    """Two mixers on the same input, their outputs added with fixed weights (type ``parallel``)."""
    left: NormedAttentionConfig
    right: DeltaRuleConfig
    left_scale: float = 1.0
    right_scale: float = 1.0

    @classmethod
    def from_dict(cls, m: Dict[str, Any], where: str, unknown: List[str]) -> "ParallelConfig":
        _only(m, ("left", "right", "left_scale", "right_scale"), where, unknown)
        return cls(NormedAttentionConfig.from_dict(_need(m, "left", where), f"{where}.left", unknown),
                   DeltaRuleConfig.from_dict(_need(m, "right", where), f"{where}.right", unknown),
                   _optional(m, "left_scale", float, 1.0), _optional(m, "right_scale", float, 1.0))

    def to_dict(self) -> Dict[str, Any]:
        return {"left": self.left.to_dict(), "left_scale": self.left_scale, "right": self.right.to_dict(),
                "right_scale": self.right_scale}


@dataclass
class CappedAttentionConfig:
    """Softmax attention with normed heads, capped scores, a window, a keyless term and mixed values (type ``attention``)."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: Optional[RotationConfig]
    softcap: Optional[float]
    window: Optional[int]
    v_mix: bool

    @classmethod
    def from_dict(cls, m: Dict[str, Any], where: str, unknown: List[str]) -> "CappedAttentionConfig":
        _only(m, ("heads", "kv_heads", "dim", "vdim", "scale", "rot", "softcap", "mask", "v_mix"), where, unknown)
        mask = m.get("mask")
        if mask is not None:
            _only(mask, ("size",), f"{where}.mask", unknown)
        dim = int(_need(m, "dim", where))
        c = cls(heads=int(_need(m, "heads", where)), kv_heads=int(_need(m, "kv_heads", where)), dim=dim,
                vdim=_optional(m, "vdim", int, dim), scale=float(_need(m, "scale", where)),
                rot=RotationConfig.from_dict(m.get("rot"), dim, f"{where}.rot", unknown), softcap=_optional(m, "softcap", float),
                window=None if mask is None else int(_need(mask, "size", f"{where}.mask")), v_mix=bool(m.get("v_mix", False)))
        if min(c.heads, c.kv_heads, c.dim, c.vdim, 1 if c.window is None else c.window) <= 0 or c.heads % c.kv_heads \
                or not c.scale > 0 or (c.softcap is not None and not c.softcap > 0):
            raise ConfigError(f"config.json: {where}: sizes, scale and the soft cap must be positive and heads a multiple of kv_heads")
        return c

    def to_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {"dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads, "scale": self.scale,
                             "v_mix": self.v_mix, "vdim": self.vdim}
        if self.softcap is not None:
            d["softcap"] = self.softcap
        if self.window is not None:
            d["mask"] = {"size": self.window}
        if self.rot is not None:
            d["rot"] = self.rot.to_dict()
        return d


@dataclass
class DenseFFConfig:
    ff: int

    @classmethod
    def from_dict(cls, m: Dict[str, Any], where: str, unknown: List[str]) -> "DenseFFConfig":
        _only(m, ("kind", "ff"), where, unknown)
        if _need(m, "kind", where) != "dense":
            raise ConfigError(f"config.json: {where}.kind {m['kind']!r}: this design's feed-forward is 'dense'")
        c = cls(int(_need(m, "ff", where)))
        if c.ff <= 0:
            raise ConfigError(f"config.json: {where}.ff must be positive")
        return c

    def to_dict(self) -> Dict[str, Any]:
        return {"ff": self.ff, "kind": "dense"}


@dataclass
class BifatarLayer:
    type: str
    mixer: Any                          # Mamba2Config, ParallelConfig or CappedAttentionConfig
    mlp: Optional[DenseFFConfig]


@dataclass
class BifatarConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: List[BifatarLayer]
    eos_token_id: Optional[Any] = None
    architecture: str = "Bifatar"
    unknown_keys: List[str] = field(default_factory=list)

    MIXERS = {"mamba2": Mamba2Config, "parallel": ParallelConfig, "attention": CappedAttentionConfig}

    @classmethod
    def from_dict(cls, cfg: Dict[str, Any]) -> "BifatarConfig":
        unknown: List[str] = []
        _only(cfg, ("architecture", "architectures", "layers", "norm", "vocab", "width", "eos_token_id"), "the top level", unknown)
        raw_layers = _need(cfg, "layers", "the top level")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers = []
        for i, L in enumerate(raw_layers):
            where = f"layers[{i}]"
            _only(L, ("type", "mixer", "mlp"), where, unknown)
            kind = _need(L, "type", where)
            if kind not in cls.MIXERS:
                raise ConfigError(f"config.json: {where}.type {kind!r}: this design's mixers are {sorted(cls.MIXERS)}")
            mixer = cls.MIXERS[kind].from_dict(_need(L, "mixer", where), f"{where}.mixer", unknown)
            mlp = L.get("mlp")
            layers.append(BifatarLayer(kind, mixer, None if mlp is None else DenseFFConfig.from_dict(mlp, f"{where}.mlp", unknown)))
        norm = _need(cfg, "norm", "the top level")
        _only(norm, ("eps",), "norm", unknown)
        out = cls(vocab=int(_need(cfg, "vocab", "the top level")), width=int(_need(cfg, "width", "the top level")),
                  norm_eps=float(_need(norm, "eps", "norm")), layers=layers, eos_token_id=cfg.get("eos_token_id"))
        if out.vocab <= 0 or out.width <= 0 or not out.norm_eps > 0:
            raise ConfigError("config.json: vocab, width and norm.eps must be positive")
        mixing = {(L.mixer.kv_heads, L.mixer.vdim) for L in layers if L.type == "attention" and L.mixer.v_mix}
        if len(mixing) > 1:
            raise ConfigError(f"config.json: layers that mix values need the same kv_heads and vdim, got {sorted(mixing)}")
        out.unknown_keys = unknown
        if unknown:
            warnings.warn(f"config.json has keys the Bifatar design does not define (ignored): {unknown}")
        return out

    def stop_token_ids(self) -> List[int]:
        if self.eos_token_id is None:
            return []
        if isinstance(self.eos_token_id, (list, tuple)):
            return [int(t) for t in self.eos_token_id]
        return [int(self.eos_token_id)]

    def to_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {
            "architecture": self.architecture,
            "layers": [{"type": L.type, "mixer": L.mixer.to_dict(), "mlp": None if L.mlp is None else L.mlp.to_dict()}
                       for L in self.layers],
            "norm": {"eps": self.norm_eps}, "vocab": self.vocab, "width": self.width,
        }
        if self.eos_token_id is not None:
            d["eos_token_id"] = copy.deepcopy(self.eos_token_id)
        return d

    def summary(self) -> str:
        kinds = ", ".join(f"{sum(L.type == k for L in self.layers)} {k}" for k in sorted(self.MIXERS))
        return f"Bifatar layers={len(self.layers)} ({kinds}) width={self.width} vocab={self.vocab} eps={self.norm_eps}"
