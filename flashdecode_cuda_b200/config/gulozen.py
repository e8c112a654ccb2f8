"""Typed configuration of the Gulozen decoder, read from ``config.json``.

The file names the design under ``"architecture"`` and gives every size and
constant: ``layers[i]`` holds ``type`` (which mixer: ``lightning`` or
``latent_attention``), ``mixer`` (its sizes and constants) and ``mlp`` (a
mixture of experts, ``kind`` ``moe``, or null); ``embedding.scale``,
``norm.eps``, ``norm.groups``, ``canon.taps``, ``vocab`` and ``width`` are
global.  A key the design needs and the file lacks is an error that names its
place.  What a file may leave out, with what that means: ``embedding.scale``
(1), ``norm.groups`` (1: a plain RMS norm), ``canon`` (one tap), a latent
mixer's ``rot.scaling`` (plain frequencies) and ``rot.dims`` (``rot_dim``), a
layer's ``mlp`` (none).  A key this reader does not know changes nothing it
computes; it is kept in ``unknown_keys`` and named in one warning.
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


_UNKNOWN: List[str] = []       # filled while a configuration is read


def _only(d: Dict[str, Any], known, where: str) -> None:
    if not isinstance(d, dict):
        raise ConfigError(f"config.json: {where} must be an object")
    _UNKNOWN.extend(f"{where}.{k}" for k in sorted(set(d) - set(known)))


SCALING_KEYS = ("factor", "original", "fast", "slow")


@dataclass
class LightningConfig:
    """Linear attention with a constant decay per head (``layers[i].mixer`` of type ``lightning``)."""
    heads: int
    dim: int
    vdim: int
    decay: List[float]

    @classmethod
    def from_dict(cls, m: Dict[str, Any], where: str) -> "LightningConfig":
        _only(m, ("heads", "dim", "vdim", "decay"), where)
        dim = int(_need(m, "dim", where))
        c = cls(int(_need(m, "heads", where)), dim, int(m.get("vdim", dim)), [float(g) for g in _need(m, "decay", where)])
        if min(c.heads, c.dim, c.vdim) <= 0:
            raise ConfigError(f"config.json: {where}: sizes must be positive")
        if len(c.decay) != c.heads:
            raise ConfigError(f"config.json: {where}.decay: {len(c.decay)} numbers for {c.heads} heads")
        return c

    def to_dict(self) -> Dict[str, Any]:
        return {"decay": list(self.decay), "dim": self.dim, "heads": self.heads, "vdim": self.vdim}


@dataclass
class LatentAttentionConfig:
    """Softmax attention over one cached latent and one rotated key part per position (``layers[i].mixer`` of type
    ``latent_attention``)."""
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot_base: float
    rot_scaling: Optional[Dict[str, float]] = None

    @classmethod
    def from_dict(cls, m: Dict[str, Any], where: str) -> "LatentAttentionConfig":
        _only(m, ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank", "scale", "rot"), where)
        dim, rot_dim = int(_need(m, "dim", where)), int(_need(m, "rot_dim", where))
        rot = _need(m, "rot", where)
        _only(rot, ("base", "dims", "scaling"), f"{where}.rot")
        sc = rot.get("scaling")
        if sc is not None:
            _only(sc, SCALING_KEYS, f"{where}.rot.scaling")
            sc = {k: float(_need(sc, k, f"{where}.rot.scaling")) for k in SCALING_KEYS}
            if not all(v > 0 for v in sc.values()):
                raise ConfigError(f"config.json: {where}.rot.scaling: every number must be positive")
        c = cls(heads=int(_need(m, "heads", where)), dim=dim, rot_dim=rot_dim, vdim=int(m.get("vdim", dim)),
                q_rank=int(_need(m, "q_rank", where)), kv_rank=int(_need(m, "kv_rank", where)),
                scale=float(_need(m, "scale", where)), rot_base=float(_need(rot, "base", f"{where}.rot")), rot_scaling=sc)
        if min(c.heads, c.dim, c.vdim, c.q_rank, c.kv_rank) <= 0:
            raise ConfigError(f"config.json: {where}: sizes must be positive")
        if rot_dim <= 0 or rot_dim % 2 or int(rot.get("dims", rot_dim)) != rot_dim:
            raise ConfigError(f"config.json: {where}: the rotated part has {rot_dim} dimensions: it must be even and "
                              f"rot.dims the same")
        if not c.rot_base > 0 or c.rot_base == 1.0:
            raise ConfigError(f"config.json: {where}.rot.base must be positive and not 1")
        return c

    def to_dict(self) -> Dict[str, Any]:
        rot: Dict[str, Any] = {"base": self.rot_base, "dims": self.rot_dim}
        if self.rot_scaling is not None:
            rot["scaling"] = dict(self.rot_scaling)
        return {"dim": self.dim, "heads": self.heads, "kv_rank": self.kv_rank, "q_rank": self.q_rank, "rot": rot,
                "rot_dim": self.rot_dim, "scale": self.scale, "vdim": self.vdim}

    def rotation_key(self) -> str:
        sc = "" if self.rot_scaling is None else "@" + ",".join(f"{k}={self.rot_scaling[k]!r}" for k in SCALING_KEYS)
        return f"rot{self.rot_dim}@{self.rot_base!r}{sc}"


@dataclass
class SoftmaxRouterConfig:
    """``mlp`` of kind ``moe``: gated experts chosen and weighted by their softmax scores."""
    experts: int
    top: int
    expert_ff: int
    kind: str = "moe"

    @classmethod
    def from_dict(cls, m: Dict[str, Any], where: str) -> "SoftmaxRouterConfig":
        _only(m, ("kind", "router", "expert"), where)
        r, e = _need(m, "router", where), _need(m, "expert", where)
        _only(r, ("experts", "top"), f"{where}.router")
        _only(e, ("ff",), f"{where}.expert")
        c = cls(experts=int(_need(r, "experts", f"{where}.router")), top=int(_need(r, "top", f"{where}.router")),
                expert_ff=int(_need(e, "ff", f"{where}.expert")))
        if c.experts <= 0 or not (0 < c.top <= c.experts) or c.expert_ff <= 0:
            raise ConfigError(f"config.json: {where}: needs 0 < top <= experts and a positive ff")
        return c

    def to_dict(self) -> Dict[str, Any]:
        return {"expert": {"ff": self.expert_ff}, "kind": "moe", "router": {"experts": self.experts, "top": self.top}}


@dataclass
class GulozenLayer:
    type: str
    mixer: Any                          # LightningConfig or LatentAttentionConfig
    mlp: Optional[SoftmaxRouterConfig]


@dataclass
class GulozenConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: List[GulozenLayer]
    norm_groups: int = 1
    taps: int = 1
    embedding_scale: float = 1.0
    eos_token_id: Optional[Any] = None
    architecture: str = "Gulozen"
    unknown_keys: List[str] = field(default_factory=list)

    MIXERS = {"lightning": LightningConfig, "latent_attention": LatentAttentionConfig}
    FEED_FORWARDS = {"moe": SoftmaxRouterConfig}

    @classmethod
    def from_dict(cls, cfg: Dict[str, Any]) -> "GulozenConfig":
        _UNKNOWN.clear()
        _only(cfg, ("architecture", "architectures", "canon", "embedding", "layers", "norm", "vocab", "width",
                    "eos_token_id"), "the top level")
        raw_layers = _need(cfg, "layers", "the top level")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers = []
        for i, L in enumerate(raw_layers):
            where = f"layers[{i}]"
            _only(L, ("type", "mixer", "mlp"), where)
            kind = _need(L, "type", where)
            if kind not in cls.MIXERS:
                raise ConfigError(f"config.json: {where}.type {kind!r}: this design's mixers are {sorted(cls.MIXERS)}")
            mixer = cls.MIXERS[kind].from_dict(_need(L, "mixer", where), f"{where}.mixer")
            mlp = L.get("mlp")
            if mlp is not None:
                fk = _need(mlp, "kind", f"{where}.mlp")
                if fk not in cls.FEED_FORWARDS:
                    raise ConfigError(f"config.json: {where}.mlp.kind {fk!r}: this design's feed-forwards are "
                                      f"{sorted(cls.FEED_FORWARDS)}")
                mlp = cls.FEED_FORWARDS[fk].from_dict(mlp, f"{where}.mlp")
            layers.append(GulozenLayer(kind, mixer, mlp))
        norm = _need(cfg, "norm", "the top level")
        _only(norm, ("eps", "groups"), "norm")
        emb, canon = cfg.get("embedding"), cfg.get("canon")
        if emb is not None:
            _only(emb, ("scale",), "embedding")
        if canon is not None:
            _only(canon, ("taps",), "canon")
        out = cls(vocab=int(_need(cfg, "vocab", "the top level")), width=int(_need(cfg, "width", "the top level")),
                  norm_eps=float(_need(norm, "eps", "norm")), layers=layers, norm_groups=int(norm.get("groups", 1)),
                  taps=1 if canon is None else int(_need(canon, "taps", "canon")),
                  embedding_scale=1.0 if emb is None else float(emb.get("scale", 1.0)), eos_token_id=cfg.get("eos_token_id"))
        if out.vocab <= 0 or out.width <= 0 or not out.norm_eps > 0:
            raise ConfigError("config.json: vocab, width and norm.eps must be positive")
        if out.norm_groups < 1 or out.width % out.norm_groups:
            raise ConfigError(f"config.json: norm.groups: {out.width} channels do not form {out.norm_groups} equal groups")
        if out.taps < 1:
            raise ConfigError("config.json: canon.taps must be positive")
        out.unknown_keys = list(_UNKNOWN)
        if out.unknown_keys:
            warnings.warn(f"config.json has keys the Gulozen design does not define (ignored): {out.unknown_keys}")
        return out

    def stop_token_ids(self) -> List[int]:
        if self.eos_token_id is None:
            return []
        if isinstance(self.eos_token_id, (list, tuple)):
            return [int(t) for t in self.eos_token_id]
        return [int(self.eos_token_id)]

    def to_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {
            "architecture": self.architecture, "canon": {"taps": self.taps}, "embedding": {"scale": self.embedding_scale},
            "layers": [{"type": L.type, "mixer": L.mixer.to_dict(), "mlp": None if L.mlp is None else L.mlp.to_dict()}
                       for L in self.layers],
            "norm": {"eps": self.norm_eps, "groups": self.norm_groups}, "vocab": self.vocab, "width": self.width,
        }
        if self.eos_token_id is not None:
            d["eos_token_id"] = copy.deepcopy(self.eos_token_id)
        return d

    def summary(self) -> str:
        kinds = ", ".join(f"{sum(L.type == k for L in self.layers)} {k}" for k in sorted(self.MIXERS))
        return (f"Gulozen layers={len(self.layers)} ({kinds}) width={self.width} vocab={self.vocab} eps={self.norm_eps} "
                f"norm groups={self.norm_groups} taps={self.taps}")
