"""The gated delta rule as a mixer: linear attention whose state forgets per key channel and is corrected, not only added to."""

from __future__ import annotations

from typing import Dict, List, Optional

import torch

from .. import kernels as K
from ..cache.paged import StateSpec
from ..registry import register_part
from ..weights.spec import TensorSpec
from .base import LayerCache, Mixer, Runtime
from .linear import matmul, narrow_product

NARROW_MAX = 1024         # widest narrow vector of the decay and of the gate


@register_part("mixer", "gated_delta_rule")
class GatedDeltaRule(Mixer):
    """For the mixer's input h [T, hidden], with ``n_heads`` heads on ``n_qk_heads`` heads of q and k (head h reads q/k head
    h // (n_heads / n_qk_heads)):

        q, k, v = silu(conv(W_q h)), silu(conv(W_k h)), silu(conv(W_v h))     causal, ``taps`` taps per channel, no biases
        q, k    = x / sqrt(sum x^2 + 1e-6) per head;  q times head_dim^(-1/2)
        beta    = sigmoid(W_b h)                                              per head
        g       = exp(-exp(A_h) softplus(W_a2 (W_a1 h) + b))                  per head and key channel
        F_t     = diag(g_t) S_(t-1)                                           what the state keeps, [head_dim, v_head_dim] per head
        S_t     = F_t + k_t (beta_t (v_t - F_t^T k_t))^T;   o_t = S_t^T q_t
        out     = W_o ( concat_h o / rms(o) * w * sigmoid(W_g2 (W_g1 h)) )    rms per head over v_head_dim, w [v_head_dim]

    The state starts at zero and is carried in float32 per cache slot, and so are the last projected values (a ring of ``taps``
    places per channel, the value of position p at place p % taps).  One packed product gives q, k, v, beta's column and both
    narrow vectors.  Convolutions, unit vectors, decay, step size, state, output, norm and gate are float32 in both dtypes.
    Tensors ``<prefix>.q`` / ``.k`` / ``.v`` (+ ``.conv`` [channels, taps]), ``.b``, ``.a1``, ``.a2``, ``.dt_bias``, ``.A_log``,
    ``.g1``, ``.g2``, ``.norm``, ``.o``.  ``decay_rank`` / ``gate_rank`` (rows of W_a1, W_g1) None: the checkpoint's tensors
    give them."""

    shares_products = True

    def __init__(self, prefix: str, hidden_size: int, n_heads: int, n_qk_heads: int, head_dim: int, v_head_dim: int, taps: int,
                 eps: float, decay_rank: Optional[int] = None, gate_rank: Optional[int] = None):
        if head_dim > 256 or min(n_heads, n_qk_heads, head_dim, v_head_dim) < 1 or n_heads % n_qk_heads:
            raise ValueError(f"{prefix}: {n_heads} heads on {n_qk_heads} of {head_dim} x {v_head_dim}: the recurrence takes whole "
                             f"groups of heads and key sizes up to 256")
        if taps < 1 or any(r is not None and not 1 <= r <= NARROW_MAX for r in (decay_rank, gate_rank)):
            raise ValueError(f"{prefix}: {taps} taps, narrow vectors of {decay_rank} and {gate_rank} (1 to {NARROW_MAX})")
        self.prefix, self.hidden_size, self.eps = prefix, hidden_size, float(eps)
        self.n_heads, self.n_qk, self.d, self.dv, self.taps = n_heads, n_qk_heads, head_dim, v_head_dim, taps
        self.ranks = (decay_rank, gate_rank)
        self.nk, self.nv = n_qk_heads * head_dim, n_heads * v_head_dim
        self.n_conv = 2 * self.nk + self.nv

    def tensor_specs(self) -> List[TensorSpec]:
        p, H = self.prefix, self.hidden_size
        specs = []
        for n, c in (("q", self.nk), ("k", self.nk), ("v", self.nv)):
            specs += [TensorSpec(f"{p}.{n}", (c, H), init="unit"), TensorSpec(f"{p}.{n}.conv", (c, self.taps), "vector", init="conv")]
        ra, rg = self.ranks
        return specs + [
            TensorSpec(f"{p}.b", (self.n_heads, H), init="unit"), TensorSpec(f"{p}.A_log", (self.n_heads,), "vector", init="half"),
            TensorSpec(f"{p}.norm", (self.dv,), "vector", init="norm"),
            TensorSpec(f"{p}.a1", (ra, H), init="unit"), TensorSpec(f"{p}.a2", (self.n_heads * self.d, ra), init="unit"),
            TensorSpec(f"{p}.dt_bias", (self.n_heads * self.d,), "vector", init="step_bias"),
            TensorSpec(f"{p}.g1", (rg, H), init="unit"), TensorSpec(f"{p}.g2", (self.nv, rg), init="unit"),
            TensorSpec(f"{p}.o", (H, self.nv), init="unit")]

    def kv_request(self):
        return None

    def state_requests(self) -> List[StateSpec]:
        out = [StateSpec("state", (self.n_heads, self.d, self.dv), torch.float32)]
        if self.taps > 1:
            out.append(StateSpec("ring", (self.taps, self.n_conv), torch.float32))
        return out

    def bind(self, tensors: Dict[str, torch.Tensor], rt: Runtime) -> None:
        self.rt = rt
        p = self.prefix
        self.w_a2, self.w_g2 = tensors[f"{p}.a2"], tensors[f"{p}.g2"]
        self.ra, self.rg = self.w_a2.shape[1], self.w_g2.shape[1]
        a1, g1 = tensors.pop(f"{p}.a1"), tensors.pop(f"{p}.g1")
        for name, w, r in (("a", a1, self.ra), ("g", g1, self.rg)):
            if w.shape[0] != r or not 1 <= r <= NARROW_MAX:
                raise ValueError(f"{p}: {name}1 has {w.shape[0]} rows and {name}2 {r} columns (1 to {NARROW_MAX})")
        mats = [tensors.pop(f"{p}.{n}") for n in "qkv"] + [a1, g1, tensors.pop(f"{p}.b")]
        self.w_in = torch.cat(mats, dim=0).contiguous()                # [q | k | v | decay | gate | beta]
        self.b_in = None
        self.conv_w = torch.cat([tensors.pop(f"{p}.{n}.conv").float() for n in "qkv"], dim=0).contiguous()
        self.A_log = tensors.pop(f"{p}.A_log").float().contiguous()
        self.dt_bias = tensors.pop(f"{p}.dt_bias").float().contiguous()
        self.norm_w = tensors.pop(f"{p}.norm").float().contiguous()
        self.w_o = tensors[f"{p}.o"]

    def weight_bytes(self) -> int:
        mats = [self.w_in, self.w_a2, self.w_g2, self.conv_w] + ([self.w_o] if self.w_o is not None else [])
        return sum(w.numel() * w.element_size() for w in mats)

    def first_weights(self) -> Optional[torch.Tensor]:
        return self.w_in

    def in_proj(self):
        return self.w_in, self.b_in

    def out_proj(self) -> torch.Tensor:
        return self.w_o

    def inner(self, ctx, proj: torch.Tensor, col0: int, lc: LayerCache, act: torch.Tensor, act_col: int = 0,
              scale: float = 1.0) -> torch.Tensor:
        T, ws, rt = ctx.T, ctx.ws, self.rt
        H, Hk, d, dv = self.n_heads, self.n_qk, self.d, self.dv
        up4 = lambda n: -(-n // 4) * 4
        f32 = torch.float32
        q, k = ws.get("delta_q", (T, Hk, up4(d)), f32), ws.get("delta_k", (T, Hk, up4(d)), f32)
        v, g = ws.get("delta_v", (T, H, up4(dv)), f32), ws.get("delta_g", (T, H, up4(d)), f32)
        beta, gate_z = ws.get("delta_beta", (T, H), f32), ws.get("delta_gate", (T, H * dv), f32)
        a_col = col0 + 2 * self.nk + self.nv
        g_col = a_col + self.ra
        b_col = g_col + self.rg
        # the narrow vectors are expanded by products of their own in long bfloat16 steps, else while the rest is prepared
        z_a = narrow_product(ctx, proj, a_col, self.w_a2, "delta_za")
        wide = z_a is not None and narrow_product(ctx, proj, g_col, self.w_g2, None, out=gate_z) is not None
        ring = lc.states.get("ring")
        K.delta_prepare(proj, (col0, col0 + self.nk, col0 + 2 * self.nk, b_col, a_col, g_col), self.conv_w, ring, lc.writes,
                        self.A_log, self.dt_bias, d ** -0.5, q, k, v, g, beta, gate_z, ctx.tok_row, ctx.tok_pos, ctx.row_slot,
                        ctx.row_q_start, ctx.row_q_len, H, Hk, d, dv, a2=None if z_a is not None else self.w_a2, z_a=z_a,
                        g2=None if wide else self.w_g2)
        if ring is not None and lc.writes and ctx.max_q_len > 1:
            K.conv_ring_update(proj, col0, ring, ctx.row_slot, ctx.row_q_start, ctx.row_q_len, ctx.row_ctx_len, ctx.n_rows)
        o = ws.get("scan_out", (T, H * dv), f32)
        step = (q, k, v, g, beta, lc.states["state"], o, ctx.row_slot, ctx.row_q_start, ctx.row_q_len, ctx.n_rows, lc.writes)
        long = ctx.max_q_len > K.delta_scan_single()
        if long and proj.dtype == torch.bfloat16 and K.delta_chunks_takes(d):
            # (the rows' lengths on the host: a step with a long row is never replayed from a graph)
            if min(ctx.h_q_len, default=0) <= K.delta_scan_single():
                K.delta_scan(*step, short_only=True)
            n = K.delta_chunks_scratch_bytes(T, ctx.n_rows, H, d)
            K.delta_chunks(*step, ctx.max_q_len, ws.get("delta_chunks", (n,), torch.uint8))
        else:
            scratch = ws.get("delta_blocks", (K.delta_scan_scratch_floats(T, ctx.n_rows, H, d),), f32) if long else None
            K.delta_scan(*step, ctx.max_q_len, scratch)
        K.head_norm_gate(o, act, act_col, H, dv, self.eps, self.norm_w, None, 0, scale, sigmoid_gate=gate_z)
        return act

    def forward(self, ctx, x: torch.Tensor, lc: LayerCache) -> torch.Tensor:
        T, ws, rt = ctx.T, ctx.ws, self.rt
        proj = ws.get("rec_proj", (T, self.w_in.shape[0]), x.dtype)
        matmul(x, self.w_in, None, proj, status=rt.status)
        act = ws.get("rec_act", (T, self.nv), x.dtype)
        self.inner(ctx, proj, 0, lc, act, 0, 1.0)
        out = ws.get("mixer_out", (T, self.hidden_size), x.dtype)
        return matmul(act, self.w_o, None, out, target_ctas=4 * rt.sm_count, status=rt.status, upcoming=ctx.upcoming)
