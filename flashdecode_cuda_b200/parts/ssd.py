"""A state-space mixer with one decay per head that follows the input (Mamba-2)."""

from __future__ import annotations

from typing import Dict, List, Optional

import torch

from .. import kernels as K
from ..cache.paged import StateSpec
from ..registry import register_part
from ..weights.spec import TensorSpec
from .base import LayerCache, Runtime
from .recurrent import _StateMixer


CHUNKED_FROM = 32         # bfloat16 steps with a portion of more tokens than this take the recurrence in chunks


@register_part("mixer", "mamba2")
class Mamba2(_StateMixer):
    """For the mixer's input h [T, hidden], with ``n_heads`` heads of ``v_head_dim`` channels (together ``inner``), a state of
    ``state_size`` per channel and ``n_groups`` groups (head h reads group h // (n_heads / n_groups)):

        [z | x | B | C | raw] = W_in h          widths inner, inner, groups * state, groups * state, heads
        x, B, C = silu(conv(.) + bias)          causal, ``taps`` taps per channel, over all three side by side
        dt      = softplus(raw + b)             per head
        S_t     = exp(-exp(A_h) dt) S_(t-1) + dt B_t x_t^T;   y_t = S_t^T C_t + D_h x_t
        out     = W_o ( norm(y * silu(z)) )     RMS norm in ``norm_groups`` equal parts, weight [inner]

    The state starts at zero and is carried in float32 per cache slot, and so are the last projected values of x, B and C (a ring
    of ``taps`` places per channel).  Convolution, step size, decay, state, output, gate and norm are float32 in both dtypes.
    Tensors ``<prefix>.in``, ``.conv`` [channels, taps], ``.conv.b``, ``.dt_bias``, ``.A_log``, ``.D``, ``.norm``, ``.o``."""

    def __init__(self, prefix: str, hidden_size: int, n_heads: int, v_head_dim: int, state_size: int, n_groups: int, norm_groups: int,
                 taps: int, eps: float):
        if min(n_heads, v_head_dim, state_size, n_groups, norm_groups, taps) < 1 or state_size > 256 or n_heads % n_groups:
            raise ValueError(f"{prefix}: {n_heads} heads of {v_head_dim} in {n_groups} groups, a state of {state_size}, {taps} taps: the "
                             f"recurrence takes whole groups of heads and states up to 256")
        if (n_heads * v_head_dim) % norm_groups:
            raise ValueError(f"{prefix}: {n_heads * v_head_dim} channels do not form {norm_groups} equal parts")
        self.prefix, self.hidden_size, self.eps = prefix, hidden_size, float(eps)
        self.n_heads, self.d, self.dv = n_heads, state_size, v_head_dim
        self.groups, self.norm_groups, self.taps = n_groups, norm_groups, taps
        self.inner_size = n_heads * v_head_dim
        self.n_conv = self.inner_size + 2 * n_groups * state_size

    def tensor_specs(self) -> List[TensorSpec]:
        p, H = self.prefix, self.hidden_size
        return [TensorSpec(f"{p}.in", (self.inner_size + self.n_conv + self.n_heads, H), init="unit"),
                TensorSpec(f"{p}.conv", (self.n_conv, self.taps), "vector", init="conv"),
                TensorSpec(f"{p}.conv.b", (self.n_conv,), "vector", init="bias"),
                TensorSpec(f"{p}.dt_bias", (self.n_heads,), "vector", init="step_bias"),
                TensorSpec(f"{p}.A_log", (self.n_heads,), "vector", init="half"),
                TensorSpec(f"{p}.D", (self.n_heads,), "vector", init="norm"),
                TensorSpec(f"{p}.norm", (self.inner_size,), "vector", init="norm"),
                TensorSpec(f"{p}.o", (H, self.inner_size), init="unit")]

    def state_requests(self) -> List[StateSpec]:
        out = super().state_requests()
        if self.taps > 1:
            out.append(StateSpec("ring", (self.taps, self.n_conv), torch.float32))
        return out

    def bind(self, tensors: Dict[str, torch.Tensor], rt: Runtime) -> None:
        self.rt = rt
        p = self.prefix
        self.w_in, self.b_in = tensors[f"{p}.in"], None
        vec = lambda n: tensors.pop(f"{p}.{n}").float().contiguous()
        self.conv_w, self.conv_b, self.dt_bias, self.A_log, self.D, self.norm_w = (
            vec(n) for n in ("conv", "conv.b", "dt_bias", "A_log", "D", "norm"))
        self.w_o = tensors[f"{p}.o"]

    def inner(self, ctx, proj: torch.Tensor, col0: int, lc: LayerCache, act: torch.Tensor, act_col: int = 0,
              scale: float = 1.0) -> torch.Tensor:
        T, ws, rt = ctx.T, ctx.ws, self.rt
        xbc = ws.get("ssd_xbc", (T, self.n_conv), torch.float32)
        step = ws.get("ssd_step", (T, self.n_heads, 2), torch.float32)
        y = ws.get("scan_out", (T, self.inner_size), torch.float32)
        ring = lc.states.get("ring")
        x_col = col0 + self.inner_size
        # long portions in bfloat16: chunks on the tensor cores, from the convolved channels rounded; x itself also as floats
        chunked = proj.dtype == torch.bfloat16 and ctx.max_q_len > CHUNKED_FROM and K.ssd_chunks_takes(self.d, self.dv)
        xbc16 = ws.get("ssd_xbc16", (T, self.n_conv), torch.bfloat16) if chunked else None
        K.ssd_prepare(proj, x_col, x_col + self.n_conv, self.conv_w, self.conv_b, ring, lc.writes, self.dt_bias, self.A_log, xbc, step,
                      ctx.tok_row, ctx.tok_pos, ctx.row_slot, ctx.row_q_start, ctx.row_q_len, xbc16=xbc16,
                      float_cols=self.inner_size if chunked else None)
        if ring is not None and lc.writes and ctx.max_q_len > 1:
            K.conv_ring_update(proj, x_col, ring, ctx.row_slot, ctx.row_q_start, ctx.row_q_len, ctx.row_ctx_len, ctx.n_rows)
        b_col = self.inner_size
        if chunked:
            n = K.ssd_chunks_scratch_floats(T, ctx.n_rows, self.n_heads, self.d, self.dv)
            K.ssd_chunks(xbc16, step, self.A_log, lc.states["state"], y, self.groups, ctx.row_slot, ctx.row_q_start, ctx.row_q_len,
                         ctx.n_rows, ctx.max_q_len, lc.writes, ws.get("ssd_chunks", (n,), torch.float32))
        else:
            K.linear_scan(xbc, b_col + self.groups * self.d, b_col, 0, lc.states["state"], y, K.SCAN_STEP, ctx.row_slot,
                          ctx.row_q_start, ctx.row_q_len, ctx.row_ctx_len, ctx.n_rows, self.n_heads, self.d, self.dv, lc.writes,
                          rt.status, max_q_len=ctx.max_q_len, scratch=self.scan_scratch(ctx), step=step, qk_heads=self.groups)
        K.ssd_gate_norm(y, xbc, self.D, proj, col0, self.norm_w, act, act_col, self.norm_groups, self.eps, scale)
        return act
