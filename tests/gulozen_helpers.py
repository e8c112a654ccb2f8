"""Shared by the Gulozen tests: small configurations that differ from one another in every size and option, model
folders with random weights, the plain implementation as ground truth."""

from __future__ import annotations

import json
import random
from pathlib import Path
from typing import Dict, List, Optional

import torch

import flashdecode_cuda_b200 as fd
from flashdecode_cuda_b200.weights import load_checkpoint, write_model_folder
from plain import gulozen_plain as P


def lightning(heads, dim, vdim, decay=None, mlp=None):
    if decay is None:
        decay = [0.5 ** (2.0 ** -i) for i in range(heads)]            # 0.5, 0.71, 0.84, ... towards one
    return {"type": "lightning", "mixer": {"decay": decay, "dim": dim, "heads": heads, "vdim": vdim}, "mlp": mlp}


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, base=10000.0, scaling=None, mlp=None):
    rot = {"base": base, "dims": rot_dim}
    if scaling is not None:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"type": "latent_attention", "mixer": {"dim": dim, "heads": heads, "kv_rank": kv_rank, "q_rank": q_rank, "rot": rot,
                                                  "rot_dim": rot_dim, "scale": scale, "vdim": vdim}, "mlp": mlp}


def moe(experts, top, ff):
    return {"expert": {"ff": ff}, "kind": "moe", "router": {"experts": experts, "top": top}}


def model(vocab, width, eps, layers, groups=None, taps=None, emb_scale=None):
    cfg = {"architecture": "Gulozen", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}
    if groups is not None:
        cfg["norm"]["groups"] = groups
    if taps is not None:
        cfg["canon"] = {"taps": taps}
    if emb_scale is not None:
        cfg["embedding"] = {"scale": emb_scale}
    return cfg


GULOZEN: Dict[str, dict] = {
    # three norm groups, three taps; heads whose key, rotated, value, query-latent and latent sizes all differ, stretched
    # frequencies whose ramp lies inside the rotated part; a lightning layer with values wider than keys; heads of 64 + 16
    # (filled up to the tensor-core sizes); two numbers of experts and choices
    "A": model(211, 96, 1e-6, [
        latent(6, 24, 8, 40, 40, 48, 0.25, 500.0, (8.0, 64, 4.0, 1.0), moe(6, 2, 40)),
        lightning(3, 24, 40, mlp=moe(5, 3, 24)),
        latent(2, 64, 16, 64, 56, 72, 0.12, 30000.0, (5.0, 512, 16.0, 1.0), moe(7, 4, 16)),
    ], groups=3, taps=3, emb_scale=30.0),
    # one norm group, one tap (no convolution state), scale left out, plain frequencies, one head, rotated part of two
    # dimensions, every expert chosen, one choice; layers without a feed-forward; lightning heads of one size and one head
    # that never forgets
    "B": model(96, 64, 1e-5, [
        lightning(2, 32, 32, [1.0, 0.25]),
        latent(1, 16, 2, 8, 8, 8, 0.3, 100.0, None, moe(4, 1, 16)),
        lightning(4, 16, 8, mlp=moe(3, 3, 8)),
        latent(4, 64, 64, 128, 64, 128, 0.09, 10000.0),
    ]),
    # sizes that are multiples of nothing: more heads than a tile of the tensor cores has rows, ranks and head sizes that
    # are no multiples of 8, nine groups of eight channels, five taps; key heads of the recurrence wider than 128
    "C": model(160, 72, 1e-5, [
        latent(20, 12, 6, 20, 20, 36, 0.4, 1000.0, (2.0, 32, 8.0, 2.0), moe(4, 2, 20)),
        lightning(2, 136, 24, [0.9, 0.99], moe(8, 2, 40)),
        latent(3, 20, 10, 12, 12, 28, 0.35, 50.0, (16.0, 128, 2.0, 0.5), moe(9, 5, 12)),
    ], groups=9, taps=5, emb_scale=12.0),
}


def random_config(seed: int) -> dict:
    """A configuration drawn from a seed: layer orders of every kind, widths that are no power of two, all sizes of both
    mixers drawn apart, one to six taps, one to eight norm groups, with and without stretched frequencies, routed
    feed-forwards and none."""
    rng = random.Random(seed)
    groups = rng.choice([1, 2, 3, 4, 8])
    width = groups * rng.choice([12, 20, 24, 32])

    def mlp():
        if rng.random() < 0.25:
            return None
        experts = rng.choice([1, 2, 3, 5, 8, 16])
        return moe(experts, rng.randint(1, min(4, experts)), rng.choice([8, 12, 16, 40, 64]))

    def lin():
        h = rng.choice([1, 2, 3, 5])
        return lightning(h, rng.choice([8, 12, 16, 24, 40, 64, 128, 136]), rng.choice([6, 8, 16, 24, 64, 72]),
                         [rng.choice([0.0, 0.3, 0.9, 0.99, 0.9999, 1.0]) for _ in range(h)], mlp())

    def att():
        sc = None
        if rng.random() < 0.6:
            sc = (rng.choice([2.0, 4.0, 32.0]), rng.choice([16, 64, 1024]), rng.choice([4.0, 32.0]), rng.choice([0.5, 1.0]))
        return latent(rng.choice([1, 2, 3, 5, 16, 17]), rng.choice([6, 8, 12, 16, 24, 64, 128]), rng.choice([2, 4, 6, 8, 16, 32, 64]),
                      rng.choice([6, 8, 16, 20, 64, 72, 128]), rng.choice([7, 12, 16, 40, 96]), rng.choice([5, 8, 24, 50, 64, 128, 136]),
                      rng.choice([0.1, 0.2, 0.4]), rng.choice([100.0, 10000.0, 1000000.0]), sc, mlp())
    layers = [lin() if rng.random() < 0.4 else att() for _ in range(rng.randint(1, 5))]
    return model(rng.choice([50, 333, 1000]), width, rng.choice([1e-5, 1e-6]), layers, rng.choice([groups, groups] + [None] * (groups == 1)),
                 rng.choice([None, 1, 2, 3, 4, 6]), rng.choice([None, 1.0, 12.0, 40.0]))


def decisive_routers(folder: Path) -> Path:
    """Rewrite the weights so that every router's choice is decided by far more than rounding: channel 0 of the embedding
    is one constant that no sub-layer adds to, and the routers read steps of 0.8 between the experts from it and little
    else from the rest.  In bfloat16 a choice between two nearly equal scores falls either way and says nothing about
    the kernels."""
    cfg, W = raw_config(folder), weights_of(folder)
    W["embed"][:, 0] = 0.05
    x0 = [0.05 * float(cfg.get("embedding", {}).get("scale", 1.0))]          # channel 0 of X_0, X_1, ...
    x = x0[0]
    for i, L in enumerate(cfg["layers"]):
        for n in ("norm1", "norm2"):
            if f"l{i}.{n}" in W:
                W[f"l{i}.{n}"][0] = 0.0
        if L.get("mlp"):
            r = W[f"l{i}.mlp.router"].float()
            E = r.shape[0]
            g = torch.Generator().manual_seed(E + 7 * i)
            r *= 0.02
            r[:, 0] = 0.8 * torch.randperm(E, generator=g).float() / x
            W[f"l{i}.mlp.router"] = r.to(W[f"l{i}.mlp.router"].dtype)
        a = W[f"l{i}.dwa"].float()
        a[:-1] = a[:-1].abs()                                                # channel 0 stays away from zero
        W[f"l{i}.dwa"] = a.to(W[f"l{i}.dwa"].dtype)
        x0.append(x)
        x = sum(float(a[j]) * v for j, v in enumerate(x0))
    write_model_folder(folder, cfg, W)
    return folder


def write_folder(tmp: Path, name: str, seed: int = 0, decisive: bool = False) -> Path:
    folder = Path(tmp) / f"gulozen_{name}_{seed}{'_d' if decisive else ''}"
    if not (folder / "model.safetensors").exists():
        fd.write_random_model(folder, GULOZEN[name], seed)
        if decisive:
            decisive_routers(folder)
    return folder


def raw_config(folder: Path) -> dict:
    return json.loads((Path(folder) / "config.json").read_text())


def weights_of(folder: Path) -> Dict[str, torch.Tensor]:
    return {k: v.clone() for k, v in load_checkpoint(folder).items()}


_ORACLE: dict = {}

SINGLE_PRECISION_DISTANCE = 5e-7
# How near to a right angle the first token's q and k of a lightning layer may lie (over all its heads together) before
# rounding to 8 bits of mantissa decides the direction of the normed output
FIRST_TOKEN_MARGIN = 0.02
# A choice between experts that hangs on less than this much of a router logit may fall either way in float32
CHOICE_MARGIN = 1e-5
# Whole models, relative to the largest logit of the sequence, where nothing amplifies rounding.
MODEL_TOL = {"float32": 1e-4, "bfloat16": 6e-2}


class Truth:
    """The float64 logits [len, vocab] of one whole sequence from the plain implementation, and for every position how
    far rounding alone moves it: the distance of the plain model run in float32.  Where a norm divides by a root mean
    square of terms that nearly cancel - every norm here sits on what a sub-layer puts out - the roundings before it are
    magnified, in any implementation; such a position is allowed that much more."""

    def __init__(self, cfg: dict, W: Dict[str, torch.Tensor], tokens: List[int]):
        captures: list = []
        self.logits = P.forward(cfg, W, tokens, captures=captures)
        self.scale = max(float(self.logits.abs().max()), 1e-6)
        self.first_margin = 1.0
        # positions from which on a close choice between experts may have gone the other way
        n = len(tokens)
        self.close = n
        for _, kind, cap in captures:
            if kind == "lightning":
                q0, k0 = cap["q"][0], cap["k"][0]
                dots = (q0 * k0).sum(-1).abs()
                cos = float(dots.norm() / ((q0.norm(dim=-1) * k0.norm(dim=-1)).norm() + 1e-30))
                self.first_margin = min(self.first_margin, cos)
            elif kind == "moe":
                hit = (cap["margin"] < CHOICE_MARGIN).nonzero()
                if len(hit):
                    self.close = min(self.close, int(hit[0]))
        single = P.forward(cfg, W, tokens, dtype=torch.float32).double()
        self.single = (single - self.logits).abs().amax(-1) / self.scale               # [len]

    def allowed(self, dtype: str) -> torch.Tensor:
        if dtype == "float32":
            out = torch.clamp(6 * self.single, min=MODEL_TOL[dtype])
        elif self.first_margin < FIRST_TOKEN_MARGIN:
            return torch.full_like(self.single, float("inf"))
        else:
            out = MODEL_TOL[dtype] * torch.clamp(self.single / SINGLE_PRECISION_DISTANCE, min=1.0)
        out[self.close:] = float("inf")
        return out

    def excess(self, got: torch.Tensor, rows, dtype: str) -> float:
        """max over the rows of ``got`` (logits at the positions ``rows``) of distance / allowed distance: below 1
        passes."""
        rows = list(rows)
        got = got.detach().double().cpu().reshape(len(rows), -1)
        assert bool(torch.isfinite(got).all())
        d = (got - self.logits[rows]).abs().amax(-1) / self.scale
        return float((d / self.allowed(dtype)[rows]).max())


def truth(folder: Path, tokens: List[int]) -> Truth:
    key = (str(folder), tuple(tokens))
    if key not in _ORACLE:
        _ORACLE[key] = Truth(raw_config(folder), weights_of(folder), tokens)
    return _ORACLE[key]


def oracle_logits(folder: Path, tokens: List[int]) -> torch.Tensor:
    return truth(folder, tokens).logits


def plain_greedy(folder: Path, prompt: List[int], n: int) -> List[int]:
    cfg, W = raw_config(folder), weights_of(folder)
    seq, out = list(prompt), []
    for _ in range(n):
        tok = int(P.forward(cfg, W, seq)[-1].argmax())
        out.append(tok)
        seq.append(tok)
    return out
