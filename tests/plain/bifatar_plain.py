"""Plain, slow implementation of the Bifatar decoder: whole sequences, no cache,
one function per mechanism.  It shares no code with the product package; it
reads a raw ``config.json`` dictionary and a ``{tensor name: tensor}`` dict.

Bifatar in this file's notation.  A layer has one norm, n(x) = tanh(alpha x) * w + b
with a scalar alpha, whose output h both sub-layers read: x += mixer(h) + ff(h).
Three kinds of mixer:

* ``mamba2``: one projection gives a gate z, per-head inputs x, per-group vectors
  B and C and one step size per head.  x, B and C pass a short causal convolution
  with bias and silu.  With dt = softplus(raw + bias): S_t = exp(-exp(A) dt) S_(t-1) +
  dt B_t x_t^T, y_t = S_t^T C_t + D x_t; y * silu(z) is RMS-normed in equal parts.
* ``parallel``: the weighted sum of two branches.  The left one is grouped-head
  softmax attention with biased projections, q and k RMS-normed over the whole
  projection and then rotated (pairs i, i + dims/2).  The right one is the gated
  delta rule with a decay per key channel: q, k, v convolved and passed through
  silu, q and k made unit vectors, S_t = F + beta k (v - F^T k)^T with
  F = diag(g) S_(t-1), o = S_t^T q; each head's o RMS-normed, weighted, gated by a sigmoid.
* ``attention``: grouped-head softmax attention, rotation first, then an RMS norm
  per head without a weight, tanh-capped scores, a sliding window, one extra
  learned term per head in the softmax denominator, and values mixed with those of
  the first layer that mixes values.

The feed-forward is W_down relu(W_up h)^2.  The arithmetic dtype is a parameter
(float64 by default).
"""

from __future__ import annotations

from typing import Dict, Optional

import torch
import torch.nn.functional as F

UNIT_EPS = 1e-6          # inside the root of the delta rule's unit vectors


def dyn_tanh(x: torch.Tensor, w: torch.Tensor, b: torch.Tensor, alpha: torch.Tensor) -> torch.Tensor:
    return torch.tanh(alpha * x) * w + b


def unit_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x / sqrt(mean(x^2) + eps) over the last dimension."""
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def unit_vector(x: torch.Tensor) -> torch.Tensor:
    """x / sqrt(sum(x^2) + 1e-6) over the last dimension."""
    return x / torch.sqrt(x.pow(2).sum(-1, keepdim=True) + UNIT_EPS)


def softplus(x: torch.Tensor) -> torch.Tensor:
    return torch.logaddexp(x, torch.zeros_like(x))


def rotate_half(x: torch.Tensor, dims: int, base: float, first_pos: int = 0) -> torch.Tensor:
    """x [S, heads, d]: the first ``dims`` dimensions of each head turned by position * base^(-2i/dims), pair i being
    (i, i + dims/2): (u, v) -> (u c - v s, v c + u s)."""
    S = x.shape[0]
    half = dims // 2
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(half)], dtype=torch.float64)
    a = torch.arange(first_pos, first_pos + S, dtype=torch.float64)[:, None] * f[None, :]
    c, s = torch.cos(a).to(x.dtype)[:, None, :], torch.sin(a).to(x.dtype)[:, None, :]
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], dim=-1)


def short_conv(u: torch.Tensor, w: torch.Tensor, bias: Optional[torch.Tensor] = None) -> torch.Tensor:
    """u [S, C], w [C, taps]: y[t] = sum_j w[:, j] u[t - (taps - 1) + j] (+ bias), zeros before the start."""
    S, C = u.shape
    taps = w.shape[1]
    y = torch.zeros_like(u) if bias is None else bias[None, :].expand(S, C).clone()
    for j in range(taps):
        back = taps - 1 - j
        if back < S:
            y[back:] += w[:, j] * u[:S - back]
    return y


def ssd_recurrence(x: torch.Tensor, B: torch.Tensor, C: torch.Tensor, dt: torch.Tensor, A_log: torch.Tensor,
                   D: torch.Tensor) -> torch.Tensor:
    """x [S, H, dv], B and C [S, G, N], dt [S, H]: S_t = exp(-exp(A_log) dt) S_(t-1) + dt B_t x_t^T,
    y_t = S_t^T C_t + D x_t; head h reads group h // (H / G)."""
    S, H, dv = x.shape
    rep = H // B.shape[1]
    B, C = B.repeat_interleave(rep, dim=1), C.repeat_interleave(rep, dim=1)
    state = torch.zeros((H, B.shape[2], dv), dtype=x.dtype)
    out = []
    for t in range(S):
        decay = torch.exp(-torch.exp(A_log) * dt[t])
        state = decay[:, None, None] * state + dt[t][:, None, None] * B[t][:, :, None] * x[t][:, None, :]
        out.append(torch.einsum("hnv,hn->hv", state, C[t]) + D[:, None] * x[t])
    return torch.stack(out)


def gated_part_norm(y: torch.Tensor, z: torch.Tensor, w: torch.Tensor, parts: int, eps: float) -> torch.Tensor:
    """y, z [S, n]: y * silu(z), each of ``parts`` equal parts over its own root mean square, times w [n]."""
    S, n = y.shape
    g = y * F.silu(z)
    return unit_rms(g.view(S, parts, n // parts), eps).reshape(S, n) * w


def delta_recurrence(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, g: torch.Tensor, beta: torch.Tensor) -> torch.Tensor:
    """q, k [S, G, d], v [S, H, dv], g [S, H, d], beta [S, H]: F = diag(g_t) S_(t-1);
    S_t = F + beta_t k_t (v_t - F^T k_t)^T; o_t = S_t^T q_t; head h reads q/k head h // (H / G)."""
    S, H, dv = v.shape
    rep = H // q.shape[1]
    q, k = q.repeat_interleave(rep, dim=1), k.repeat_interleave(rep, dim=1)
    state = torch.zeros((H, q.shape[2], dv), dtype=q.dtype)
    out = []
    for t in range(S):
        state = g[t][:, :, None] * state
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", state, k[t]))
        state = state + k[t][:, :, None] * u[:, None, :]
        out.append(torch.einsum("hdv,hd->hv", state, q[t]))
    return torch.stack(out)


def attend(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, softcap: Optional[float] = None,
           window: Optional[int] = None, sink: Optional[torch.Tensor] = None) -> torch.Tensor:
    """q [S, H, d], k [S, G, d], v [S, G, dv] -> [S, H, dv].  Position i sees j with 0 <= i - j (< window); scores are
    scaled, then capped to softcap * tanh(score / softcap); the denominator of head h may also hold exp(sink[h])."""
    S, H, _ = q.shape
    per = H // k.shape[1]
    s = torch.einsum("ihd,jhd->hij", q, k.repeat_interleave(per, dim=1)) * scale
    if softcap is not None:
        s = softcap * torch.tanh(s / softcap)
    i, j = torch.arange(S)[:, None], torch.arange(S)[None, :]
    vis = j <= i
    if window is not None:
        vis = vis & (i - j < window)
    s = s.masked_fill(~vis[None], float("-inf"))
    m = s.max(-1).values
    if sink is not None:
        m = torch.maximum(m, sink[:, None])
    e = torch.exp(s - m[:, :, None])
    den = e.sum(-1)
    if sink is not None:
        den = den + torch.exp(sink[:, None] - m)
    return torch.einsum("hij,jhv->ihv", e / den[:, :, None], v.repeat_interleave(per, dim=1))


def relu_squared(z: torch.Tensor) -> torch.Tensor:
    return torch.clamp(z, min=0.0) ** 2


# ---------------------------------------------------------------------------
# mixers, feed-forward, model
# ---------------------------------------------------------------------------

def _lin(W: Dict[str, torch.Tensor], name: str, h: torch.Tensor, dt, bias: bool = False) -> torch.Tensor:
    y = h @ W[name].to(dt).t()
    if bias:
        y = y + W[name + ".b"].to(dt)
    return y


def mamba2_mixer(W, p: str, m: dict, h: torch.Tensor, eps: float, dt=torch.float64) -> torch.Tensor:
    S = h.shape[0]
    H, dv, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * dv
    z, u, raw = torch.split(_lin(W, f"{p}.in", h, dt), [inner, inner + 2 * G * N, H], dim=-1)
    u = F.silu(short_conv(u, W[f"{p}.conv"].to(dt), W[f"{p}.conv.b"].to(dt)))
    x, B, C = torch.split(u, [inner, G * N, G * N], dim=-1)
    step = softplus(raw + W[f"{p}.dt_bias"].to(dt))
    y = ssd_recurrence(x.reshape(S, H, dv), B.reshape(S, G, N), C.reshape(S, G, N), step, W[f"{p}.A_log"].to(dt),
                       W[f"{p}.D"].to(dt)).reshape(S, inner)
    y = gated_part_norm(y, z, W[f"{p}.norm"].to(dt), m["norm_groups"], eps)
    return y @ W[f"{p}.o"].to(dt).t()


def left_branch(W, p: str, m: dict, h: torch.Tensor, eps: float, dt=torch.float64) -> torch.Tensor:
    S = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (_lin(W, f"{p}.{n}", h, dt, bias=True) for n in "qkv")
    q = (unit_rms(q, eps) * W[f"{p}.q.norm"].to(dt)).view(S, H, d)
    k = (unit_rms(k, eps) * W[f"{p}.k.norm"].to(dt)).view(S, G, d)
    if m.get("rot"):
        q = rotate_half(q, m["rot"]["dims"], m["rot"]["base"])
        k = rotate_half(k, m["rot"]["dims"], m["rot"]["base"])
    a = attend(q, k, v.reshape(S, G, dv), m["scale"])
    return a.reshape(S, H * dv) @ W[f"{p}.o"].to(dt).t()


def right_branch(W, p: str, m: dict, h: torch.Tensor, eps: float, dt=torch.float64) -> torch.Tensor:
    S = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (F.silu(short_conv(_lin(W, f"{p}.{n}", h, dt), W[f"{p}.{n}.conv"].to(dt))) for n in "qkv")
    q = unit_vector(q.view(S, G, d)) * d ** -0.5
    k = unit_vector(k.view(S, G, d))
    beta = torch.sigmoid(_lin(W, f"{p}.b", h, dt))
    a = _lin(W, f"{p}.a2", _lin(W, f"{p}.a1", h, dt), dt) + W[f"{p}.dt_bias"].to(dt)
    g = torch.exp(-torch.exp(W[f"{p}.A_log"].to(dt))[None, :, None] * softplus(a).view(S, H, d))
    o = delta_recurrence(q, k, v.reshape(S, H, dv), g, beta)
    o = unit_rms(o, eps) * W[f"{p}.norm"].to(dt)
    gate = torch.sigmoid(_lin(W, f"{p}.g2", _lin(W, f"{p}.g1", h, dt), dt))
    return (o.reshape(S, H * dv) * gate) @ W[f"{p}.o"].to(dt).t()


def parallel_mixer(W, p: str, m: dict, h: torch.Tensor, eps: float, dt=torch.float64) -> torch.Tensor:
    return (m.get("left_scale", 1.0) * left_branch(W, f"{p}.left", m["left"], h, eps, dt)
            + m.get("right_scale", 1.0) * right_branch(W, f"{p}.right", m["right"], h, eps, dt))


def attention_mixer(W, p: str, m: dict, h: torch.Tensor, eps: float, shared: dict, dt=torch.float64) -> torch.Tensor:
    """``shared``: what the layers of one pass share; the first value-mixing layer leaves its values there."""
    S = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = _lin(W, f"{p}.q", h, dt).view(S, H, d)
    k = _lin(W, f"{p}.k", h, dt).view(S, G, d)
    v = _lin(W, f"{p}.v", h, dt)
    if m.get("rot"):
        q = rotate_half(q, m["rot"]["dims"], m["rot"]["base"])
        k = rotate_half(k, m["rot"]["dims"], m["rot"]["base"])
    q, k = unit_rms(q, eps), unit_rms(k, eps)
    if m.get("v_mix"):
        if "v" in shared:
            lam = W[f"{p}.vmix"].to(dt)
            v = (1.0 - lam) * v + lam * shared["v"]
        else:
            shared["v"] = v
    a = attend(q, k, v.view(S, G, dv), m["scale"], m.get("softcap"), (m.get("mask") or {}).get("size"),
               W[f"{p}.sink"].to(dt))
    return a.reshape(S, H * dv) @ W[f"{p}.o"].to(dt).t()


def dense_ff(W, p: str, h: torch.Tensor, dt=torch.float64) -> torch.Tensor:
    return relu_squared(_lin(W, f"{p}.up", h, dt)) @ W[f"{p}.down"].to(dt).t()


def forward(cfg: dict, W: Dict[str, torch.Tensor], tokens, dt=torch.float64, trace: Optional[list] = None) -> torch.Tensor:
    """Logits [S, vocab] of one sequence.  ``trace``: a list that receives the stream [S, width] after every layer."""
    eps = cfg["norm"]["eps"]
    tok = torch.as_tensor(tokens, dtype=torch.long)
    x = W["embed"].to(dt)[tok]
    shared: dict = {}

    def norm(name, x):
        return dyn_tanh(x, W[name].to(dt), W[name + ".b"].to(dt), W[name + ".alpha"].to(dt))
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}", L["mixer"]
        h = norm(f"{p}.norm1", x)
        if L["type"] == "mamba2":
            y = mamba2_mixer(W, f"{p}.mix", m, h, eps, dt)
        elif L["type"] == "parallel":
            y = parallel_mixer(W, f"{p}.mix", m, h, eps, dt)
        elif L["type"] == "attention":
            y = attention_mixer(W, f"{p}.mix", m, h, eps, shared, dt)
        else:
            raise ValueError(L["type"])
        if L.get("mlp") is not None:
            y = y + dense_ff(W, f"{p}.mlp", h, dt)
        x = x + y
        if trace is not None:
            trace.append(x.clone())
    return norm("final.norm", x) @ W["head"].to(dt).t()
