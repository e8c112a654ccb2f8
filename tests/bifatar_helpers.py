"""Shared by the Bifatar tests: small configurations that differ from one another in every size and option, model
folders with random weights, the plain implementation as ground truth."""

from __future__ import annotations

import json
import random
from pathlib import Path
from typing import Dict, List, Optional

import torch

import flashdecode_cuda_b200 as fd
from flashdecode_cuda_b200.weights import load_checkpoint
from plain import bifatar_plain as P


def mamba2(heads, vdim, state, groups, norm_groups, conv, mlp=None):
    m = {"conv": conv, "groups": groups, "heads": heads, "norm_groups": norm_groups, "state": state, "vdim": vdim}
    return {"type": "mamba2", "mixer": m, "mlp": mlp}


def _heads(heads, kv_heads, dim, vdim, scale, rot):
    m = {"dim": dim, "heads": heads, "kv_heads": kv_heads, "scale": scale, "vdim": vdim}
    if rot is not None:
        m["rot"] = {"base": rot[1], "dims": rot[0]}
    return m


def attention(heads, kv_heads, dim, vdim, scale, rot=None, softcap=None, window=None, v_mix=False, mlp=None):
    m = dict(_heads(heads, kv_heads, dim, vdim, scale, rot), v_mix=v_mix)
    if softcap is not None:
        m["softcap"] = softcap
    if window is not None:
        m["mask"] = {"size": window}
    return {"type": "attention", "mixer": m, "mlp": mlp}


def delta(heads, kv_heads, dim, vdim, conv, rank, gate_rank=None):
    m = {"conv": conv, "dim": dim, "heads": heads, "kv_heads": kv_heads, "rank": rank, "vdim": vdim}
    if gate_rank is not None:
        m["gate_rank"] = gate_rank
    return m


def left(heads, kv_heads, dim, vdim, scale, rot=None):
    return _heads(heads, kv_heads, dim, vdim, scale, rot)


def parallel(left, right, left_scale=None, right_scale=None, mlp=None):
    m = {"left": left, "right": right}
    if left_scale is not None:
        m["left_scale"] = left_scale
    if right_scale is not None:
        m["right_scale"] = right_scale
    return {"type": "parallel", "mixer": m, "mlp": mlp}


def dense(ff):
    return {"ff": ff, "kind": "dense"}


def model(vocab, width, eps, layers):
    return {"architecture": "Bifatar", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}


BIFATAR: Dict[str, dict] = {
    # a capped layer first (the source of the mixed values), an unmixed one between it and the one that mixes; two state-space
    # heads per group; three query heads per key head; value heads wider and narrower than key heads; two delta heads
    # on one q/k head; partial rotations; windows that are no multiple of a page
    "U": model(211, 96, 1e-6, [
        attention(6, 2, 32, 40, 0.9, (16, 1000.0), softcap=6.0, window=27, v_mix=True, mlp=dense(136)),
        mamba2(4, 24, 20, 2, 3, 4, mlp=dense(72)),
        attention(2, 1, 24, 16, 0.5, (24, 10000.0), softcap=3.0, window=11, mlp=dense(56)),
        parallel(left(6, 3, 40, 24, 0.3, (20, 500.0)), delta(4, 2, 24, 40, 3, 12, 20), 0.7, 1.3, mlp=dense(104)),
        attention(6, 2, 32, 40, 1.1, (16, 1000.0), softcap=6.0, window=27, v_mix=True, mlp=dense(136)),
    ]),
    # one of everything: one state-space head, group and part, one tap, one key head for all query heads, one delta head;
    # nothing rotated, no cap, no window, nothing mixed; layers without a feed-forward; head sizes of 64
    "V": model(96, 64, 1e-5, [
        mamba2(1, 64, 64, 1, 1, 1),
        parallel(left(4, 1, 64, 64, 0.125), delta(1, 1, 64, 64, 1, 8)),
        attention(4, 1, 64, 64, 0.125, mlp=dense(64)),
        mamba2(1, 64, 64, 1, 1, 1, mlp=dense(64)),
    ]),
    # more taps than the kernels unroll, a width that is no multiple of 16, head sizes that are multiples of nothing, key sizes
    # above 128, parts of the norm that straddle heads, a window of one position, the mixing layers' constants apart
    "W": model(160, 72, 1e-5, [
        parallel(left(3, 3, 20, 12, 0.3, (6, 100.0)), delta(3, 1, 136, 9, 5, 7), 1.5, 0.25, mlp=dense(41)),
        attention(2, 2, 118, 54, 0.7, (2, 10000.0), softcap=30.0, window=1, v_mix=True, mlp=dense(40)),
        mamba2(3, 10, 136, 3, 2, 6),
        attention(4, 2, 136, 54, 0.2, (136, 50.0), softcap=2.0, window=40, v_mix=True, mlp=dense(8)),
        # (its value heads are filled up to another size than those of the layers above)
        attention(2, 2, 42, 54, 0.2, (42, 50.0), window=33, v_mix=True, mlp=dense(8)),
    ]),
}


def random_config(seed: int) -> dict:
    """A configuration drawn from a seed: layer orders of every kind, widths that are no power of two, head counts and sizes of
    all mixers drawn apart, one to six taps, nothing to everything rotated, windows from one position to longer than any
    test sequence, with and without cap, value mixing and feed-forward."""
    rng = random.Random(seed)
    width = rng.choice([48, 72, 96, 128, 200, 256])
    mix_kv, mix_vd = rng.choice([1, 2, 3]), rng.choice([8, 16, 20, 64])

    def rot(dim):
        if rng.random() < 0.15:
            return None
        dims = min(dim, rng.choice([2, 4, 8, 16, 32, dim]))
        return (dims - dims % 2, rng.choice([100.0, 10000.0, 1000000.0]))

    def mlp():
        return None if rng.random() < 0.2 else dense(rng.choice([8, 24, 41, 96, 100, 264]))

    def ssm():
        g, per = rng.choice([1, 2, 3]), rng.choice([1, 2, 4])
        h, dv = g * per, rng.choice([6, 8, 16, 24, 64])
        parts = rng.choice([p for p in (1, 2, 3, 4, 6) if (h * dv) % p == 0])
        return mamba2(h, dv, rng.choice([8, 12, 16, 40, 64, 128, 136]), g, parts, rng.choice([1, 2, 3, 4, 6]), mlp())

    def par():
        kv, g = rng.choice([1, 2, 3]), rng.choice([1, 2, 4])
        d = rng.choice([8, 12, 16, 20, 32, 40, 64, 128])
        hk, per = rng.choice([1, 2]), rng.choice([1, 2, 3])
        dd = rng.choice([8, 10, 16, 24, 48, 64, 96, 136])
        return parallel(left(kv * g, kv, d, rng.choice([d, 8, 12, 48, 64]), rng.choice([0.1, 0.125, 0.3]), rot(d)),
                        delta(hk * per, hk, dd, rng.choice([6, 8, 16, 32, 40, 64]), rng.choice([1, 2, 3, 4, 5]), rng.choice([4, 7, 24, 32]),
                              rng.choice([None, 5, 16])),
                        rng.choice([None, 0.5, 2.0]), rng.choice([None, 0.3, 1.7]), mlp())

    def att():
        mixed = rng.random() < 0.6
        kv, g = (mix_kv if mixed else rng.choice([1, 2, 3])), rng.choice([1, 2, 4])
        d = rng.choice([8, 12, 16, 20, 32, 40, 64, 128])
        return attention(kv * g, kv, d, mix_vd if mixed else rng.choice([d, 8, 16, 48]), rng.choice([0.2, 0.5, 1.0]), rot(d),
                         rng.choice([None, 1.0, 5.0, 50.0]), rng.choice([None, 1, 2, 7, 16, 33, 64, 100, 1000]), mixed, mlp())
    layers = [rng.choice([ssm, par, att])() for _ in range(rng.randint(1, 5))]
    return model(rng.choice([50, 333, 1000]), width, rng.choice([1e-5, 1e-6]), layers)


def write_folder(tmp: Path, name: str, seed: int = 0) -> Path:
    folder = Path(tmp) / f"bifatar_{name}_{seed}"
    if not (folder / "model.safetensors").exists():
        fd.write_random_model(folder, BIFATAR[name], seed)
    return folder


def raw_config(folder: Path) -> dict:
    return json.loads((Path(folder) / "config.json").read_text())


def weights_of(folder: Path) -> Dict[str, torch.Tensor]:
    return {k: v.clone() for k, v in load_checkpoint(folder).items()}


_ORACLE: dict = {}

# The plain model in float32 lies about this far (relative to the largest logit) from the plain model in float64 where nothing
# amplifies rounding.
SINGLE_PRECISION_DISTANCE = 5e-7
# Whole models, relative to the largest logit of the sequence, where nothing amplifies rounding.
MODEL_TOL = {"float32": 1e-4, "bfloat16": 5e-2}


class Truth:
    """The float64 logits [len, vocab] of one whole sequence from the plain implementation, and for every position how
    far rounding alone moves it: the distance of the plain model run in float32.  With random weights a position now
    and then divides by a root mean square of terms that nearly cancel, and every rounding before it is magnified there,
    in any implementation; such a position is allowed that much more."""

    def __init__(self, cfg: dict, W: Dict[str, torch.Tensor], tokens: List[int]):
        self.logits = P.forward(cfg, W, tokens)
        self.scale = max(float(self.logits.abs().max()), 1e-6)
        single = P.forward(cfg, W, tokens, dt=torch.float32).double()
        self.single = (single - self.logits).abs().amax(-1) / self.scale               # [len]

    def allowed(self, dtype: str) -> torch.Tensor:
        """[len]: the largest relative distance a position may have in ``dtype``."""
        if dtype == "float32":
            return torch.clamp(6 * self.single, min=MODEL_TOL[dtype])
        return MODEL_TOL[dtype] * torch.clamp(self.single / SINGLE_PRECISION_DISTANCE, min=1.0)

    def excess(self, got: torch.Tensor, rows, dtype: str) -> float:
        """max over the rows of ``got`` (logits at the positions ``rows``) of distance / allowed distance: below 1
        passes."""
        rows = list(rows)
        got = got.detach().double().cpu().reshape(len(rows), -1)
        d = (got - self.logits[rows]).abs().amax(-1) / self.scale
        return float((d / self.allowed(dtype)[rows]).max())


def truth(folder: Path, tokens: List[int]) -> Truth:
    key = (str(folder), tuple(tokens))
    if key not in _ORACLE:
        _ORACLE[key] = Truth(raw_config(folder), weights_of(folder), tokens)
    return _ORACLE[key]


def oracle_logits(folder: Path, tokens: List[int]) -> torch.Tensor:
    """float64 logits [len, vocab] of one whole sequence from the plain implementation."""
    return truth(folder, tokens).logits


def plain_greedy(folder: Path, prompt: List[int], n: int) -> List[int]:
    seq, out = list(prompt), []
    for _ in range(n):
        tok = int(P.forward(raw_config(folder), weights_of(folder), seq)[-1].argmax())
        out.append(tok)
        seq.append(tok)
    return out
