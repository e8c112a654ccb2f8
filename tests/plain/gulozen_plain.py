"""Plain, slow implementation of the Gulozen decoder: whole sequences, no cache,
one function per mechanism.  It shares no code with the product package; it
reads a raw ``config.json`` dictionary and a ``{tensor name: tensor}`` dict.

Gulozen in this file's notation.  X_0 = embed[token] * s_e, x = X_0.  Layer i:

  u = x + conv(x)                      a causal depthwise convolution over time, added to its input
  x = x + n1(mixer(u))                 the norm sits on what the sub-layer puts out
  x = x + n2(ff(x))                    (where the layer has a feed-forward)
  X_(i+1) = x;  x = sum_j a_j X_j      over j = 0 .. i + 1, with i + 2 learned numbers of the layer's own

n(y) splits y into equal groups of neighbours, divides each by its own
sqrt(mean^2 + eps) and multiplies the whole by w.  Two kinds of mixer:

* ``lightning``: linear attention with one constant decay per head,
  S_t = g S_(t-1) + k_t v_t^T, o_t = S_t^T q_t, where q, k and v have all passed
  silu; the heads side by side are RMS-normed as one vector, multiplied by
  sigmoid(W_g u) and projected.
* ``latent_attention``: q comes through a normed low-rank vector; one normed
  vector c per position gives every head its key (U_h c) and value (V_h c); a
  separate small part of the key, one for all heads, is rotated (neighbouring
  dimensions form the pairs, frequencies stretched); softmax over every earlier
  key and a learned term per head without key or value; the heads are multiplied
  by sigmoid(W_g u) and projected.

The feed-forward is a mixture of small gated (silu) experts: softmax scores over
all experts, the largest ``top`` chosen, weighted by their scores as they are.

The arithmetic dtype is a parameter (float64 by default).
"""

from __future__ import annotations

import math
from typing import Dict, Optional

import torch


def rms_norm(x: torch.Tensor, w: Optional[torch.Tensor], eps: float) -> torch.Tensor:
    y = x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)
    return y if w is None else y * w


def grouped_rms_norm(x: torch.Tensor, w: torch.Tensor, eps: float, groups: int) -> torch.Tensor:
    parts = x.view(*x.shape[:-1], groups, -1)
    return rms_norm(parts, None, eps).reshape(x.shape) * w


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def causal_conv(u: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """u [S, C], w [C, taps]: y[t] = sum_j w[:, j] u[t - (taps - 1) + j], zeros before the start."""
    S, taps = u.shape[0], w.shape[1]
    y = torch.zeros_like(u)
    for j in range(taps):
        back = taps - 1 - j
        if back < S:
            y[back:] += w[:, j] * u[:S - back]
    return y


def depth_average(history, weights: torch.Tensor) -> torch.Tensor:
    out = torch.zeros_like(history[0])
    for a, X in zip(weights, history):
        out = out + a * X
    return out


def rot_frequencies(dims: int, base: float, scaling: Optional[dict] = None):
    """(f [dims/2], factor on cos and sin).  f_i = base^(-2i/dims).  With ``scaling``: pair(t) = dims ln(original / (2
    pi t)) / (2 ln base) is the pair that turns t times within the original length; between pair(fast), rounded down,
    and pair(slow), rounded up, f_i goes over from f_i to f_i / factor along a straight line."""
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    mag = 1.0
    if scaling:
        factor, orig = float(scaling["factor"]), float(scaling["original"])

        def pair(t):
            return dims * math.log(orig / (2 * math.pi * t)) / (2 * math.log(base))
        lo = max(math.floor(pair(float(scaling["fast"]))), 0)
        hi = min(math.ceil(pair(float(scaling["slow"]))), dims - 1)
        for i in range(len(f)):
            ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
            f[i] = f[i] / factor * ramp + f[i] * (1.0 - ramp)
        mag = 0.1 * math.log(factor) + 1.0
    return torch.tensor(f, dtype=torch.float64), mag


def rotate_pairs(x: torch.Tensor, positions: torch.Tensor, freqs: torch.Tensor, mag: float) -> torch.Tensor:
    """x [S, heads, dims]: (x_2i, x_2i+1) turned by position * f_i, times mag."""
    a = positions.to(torch.float64)[:, None] * freqs[None, :]
    c, s = (torch.cos(a) * mag).to(x.dtype)[:, None, :], (torch.sin(a) * mag).to(x.dtype)[:, None, :]
    u, v = x[:, :, 0::2], x[:, :, 1::2]
    out = torch.empty_like(x)
    out[:, :, 0::2] = u * c - v * s
    out[:, :, 1::2] = v * c + u * s
    return out


def decay_recurrence(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, decay: torch.Tensor,
                     state: Optional[torch.Tensor] = None):
    """q, k [S, H, d], v [S, H, dv], decay [H]: S_t = decay S_(t-1) + k_t v_t^T, o_t = S_t^T q_t, token by token.
    Returns (o [S, H, dv], the last state)."""
    S, H, d = q.shape
    if state is None:
        state = torch.zeros((H, d, v.shape[2]), dtype=q.dtype)
    out = []
    for t in range(S):
        state = decay[:, None, None] * state + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hdv,hd->hv", state, q[t]))
    return torch.stack(out), state


def sink_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, sink: torch.Tensor) -> torch.Tensor:
    """q, k [S, H, d], v [S, H, dv], sink [H]: p_j = exp(s_j) / (exp(sink) + sum_j exp(s_j)) over j <= i."""
    S, H, _ = q.shape
    out = torch.zeros((S, H, v.shape[2]), dtype=q.dtype)
    future = torch.ones(S, S, dtype=torch.bool).triu(1)
    for h in range(H):
        s = (q[:, h] @ k[:, h].T) * scale
        s = s.masked_fill(future, -math.inf)
        m = torch.maximum(s.amax(-1), sink[h])
        e = torch.exp(s - m[:, None])
        out[:, h] = (e @ v[:, h]) / (e.sum(-1) + torch.exp(sink[h] - m))[:, None]
    return out


def lightning_mixer(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str, mc: dict, eps: float,
                    capture: Optional[dict] = None) -> torch.Tensor:
    S = h.shape[0]
    H, d, dv = mc["heads"], mc["dim"], mc["vdim"]
    q, k = silu(h @ W[f"{p}.q"].T).view(S, H, d), silu(h @ W[f"{p}.k"].T).view(S, H, d)
    v = silu(h @ W[f"{p}.v"].T).view(S, H, dv)
    o, _ = decay_recurrence(q, k, v, torch.tensor(mc["decay"], dtype=torch.float64).to(h.dtype))
    if capture is not None:
        capture.update(q=q, k=k, v=v, o=o)
    o = rms_norm(o.reshape(S, H * dv), W[f"{p}.norm"], eps)
    return (o * torch.sigmoid(h @ W[f"{p}.g"].T)) @ W[f"{p}.o"].T


def latent_mixer(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str, mc: dict, eps: float,
                 capture: Optional[dict] = None) -> torch.Tensor:
    S = h.shape[0]
    H, d, rd, dv, r = mc["heads"], mc["dim"], mc["rot_dim"], mc["vdim"], mc["kv_rank"]
    q = (rms_norm(h @ W[f"{p}.dq"].T, W[f"{p}.dq.norm"], eps) @ W[f"{p}.uq"].T).view(S, H, d + rd)
    low = h @ W[f"{p}.dkv"].T
    c = rms_norm(low[:, :r], W[f"{p}.dkv.norm"], eps)
    k = (c @ W[f"{p}.uk"].T).view(S, H, d)
    v = (c @ W[f"{p}.uv"].T).view(S, H, dv)
    f, mag = rot_frequencies(rd, float(mc["rot"]["base"]), mc["rot"].get("scaling"))
    pos = torch.arange(S)
    q_rot = rotate_pairs(q[:, :, d:], pos, f, mag)
    k_rot = rotate_pairs(low[:, None, r:], pos, f, mag)
    q = torch.cat([q[:, :, :d], q_rot], dim=-1)
    k = torch.cat([k, k_rot.expand(S, H, rd)], dim=-1)
    o = sink_attention(q, k, v, float(mc["scale"]), W[f"{p}.sink"])
    if capture is not None:
        capture.update(q=q, k=k, v=v, c=c, o=o)
    return (o.reshape(S, H * dv) * torch.sigmoid(h @ W[f"{p}.g"].T)) @ W[f"{p}.o"].T


def gated_ff(h: torch.Tensor, gate: torch.Tensor, up: torch.Tensor, down: torch.Tensor) -> torch.Tensor:
    return (silu(h @ gate.T) * (h @ up.T)) @ down.T


def route(h: torch.Tensor, router: torch.Tensor, top: int):
    """(chosen expert ids [S, top], their softmax scores [S, top], not renormalised)."""
    s = torch.softmax(h @ router.T, dim=-1)
    ids = s.topk(top, dim=-1).indices
    return ids, s.gather(1, ids)


def moe_ff(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str, fc: dict, capture: Optional[dict] = None):
    ids, w = route(h, W[f"{p}.router"], fc["router"]["top"])
    if capture is not None:
        z = (h @ W[f"{p}.router"].T).sort(dim=-1, descending=True).values
        top = fc["router"]["top"]
        capture.update(ids=ids, weights=w, margin=z[:, top - 1] - z[:, top] if top < z.shape[1] else z[:, 0] * 0 + 1e9)
    out = torch.zeros_like(h)
    for e in range(fc["router"]["experts"]):
        hit = (ids == e)
        rows = hit.any(-1).nonzero()[:, 0]
        if len(rows):
            q = f"{p}.e{e}"
            we = (w * hit).sum(-1)[rows]
            out[rows] += we[:, None] * gated_ff(h[rows], W[f"{q}.gate"], W[f"{q}.up"], W[f"{q}.down"])
    return out


MIXERS = {"lightning": lightning_mixer, "latent_attention": latent_mixer}


def forward(cfg: dict, weights: Dict[str, torch.Tensor], tokens, dtype=torch.float64, return_layers: bool = False,
            captures: Optional[list] = None):
    """Logits [S, vocab] of one whole sequence (and, on request, the stream after every layer, depth average
    included).  ``captures``: a list that receives (layer, kind, what was seen) for every mixer and feed-forward."""
    W = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in weights.items()}
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    eps, groups = float(cfg["norm"]["eps"]), int(cfg["norm"].get("groups", 1))
    x = W["embed"][tokens] * float(cfg.get("embedding", {}).get("scale", 1.0))
    history, layers = [x], []
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}"
        u = x + causal_conv(x, W[f"{p}.canon1"])
        cap = None if captures is None else {}
        x = x + grouped_rms_norm(MIXERS[L["type"]](u, W, f"{p}.mix", L["mixer"], eps, cap), W[f"{p}.norm1"], eps, groups)
        if captures is not None:
            captures.append((i, L["type"], cap))
        if L.get("mlp"):
            cap = None if captures is None else {}
            x = x + grouped_rms_norm(moe_ff(x, W, f"{p}.mlp", L["mlp"], cap), W[f"{p}.norm2"], eps, groups)
            if captures is not None:
                captures.append((i, "moe", cap))
        history.append(x)
        x = depth_average(history, W[f"{p}.dwa"])
        layers.append(x)
    logits = grouped_rms_norm(x, W["final.norm"], eps, groups) @ W["head"].T
    return (logits, torch.stack(layers)) if return_layers else logits
