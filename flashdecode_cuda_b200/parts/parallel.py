"""Mixers side by side: several mixers read the same input and their outputs are added with fixed weights."""

from __future__ import annotations

from typing import Dict, List, Optional, Sequence

import torch

from .. import kernels as K
from ..cache.paged import StateSpec
from ..registry import register_part
from ..weights.spec import TensorSpec
from .base import KVRequest, LayerCache, Mixer, Runtime
from .linear import matmul, takes_tail


@register_part("mixer", "parallel")
class ParallelMixers(Mixer):
    """out = sum_b scale_b * branch_b(h): ``branches`` are mixers (built parts), ``names`` what their share of the
    layer's state is called, ``scales`` their weights in the sum.

    Branches that can share their products (``shares_products``: an input product, inner work, an output product)
    are run as ONE input product over the stacked input matrices, each branch's inner work on its columns, and ONE
    output product over the branches' activations laid side by side with the stacked output matrices:
    sum_b scale_b W_b a_b = [W_1 | W_2 | ...] [scale_1 a_1 ; scale_2 a_2 ; ...].  The scale enters each branch's
    activations in float32 before their one rounding.  A feed-forward that reads the same input as the mixers is one more
    such branch; as the last one, its activation is taken in the input product's epilogue in steps of up to 128 tokens.  A branch's activations start at a multiple of 8 columns, and the row's length is a multiple of 32 (columns
    of zeros fill up).  Other branches run whole, and the weighted sum of the outputs is taken in float32.  At most one branch may keep keys; every branch's per-sequence state is kept under
    ``<name>.<its own name>``."""

    def __init__(self, prefix: str, branches: Sequence[Mixer], names: Sequence[str], scales: Sequence[float],
                 hidden_size: int):
        if not branches or not (len(branches) == len(names) == len(scales)) or len(set(names)) != len(names):
            raise ValueError(f"{prefix}: branches, their names and their scales must match, names differing")
        if sum(b.kv_request() is not None for b in branches) > 1:
            raise ValueError(f"{prefix}: at most one of the mixers side by side may keep keys")
        self.prefix, self.hidden_size = prefix, hidden_size
        self.branches, self.names, self.scales = list(branches), list(names), [float(s) for s in scales]
        self.fused = all(getattr(b, "shares_products", False) for b in self.branches)

    @property
    def graph_safe(self) -> bool:
        return all(getattr(b, "graph_safe", True) for b in self.branches)

    def tensor_specs(self) -> List[TensorSpec]:
        return [s for b in self.branches for s in b.tensor_specs()]

    def kv_request(self) -> Optional[KVRequest]:
        for b in self.branches:
            r = b.kv_request()
            if r is not None:
                return r
        return None

    def state_requests(self) -> List[StateSpec]:
        return [StateSpec(f"{n}.{s.name}", s.shape, s.dtype) for n, b in zip(self.names, self.branches)
                for s in b.state_requests()]

    def bind(self, tensors: Dict[str, torch.Tensor], rt: Runtime) -> None:
        self.rt = rt
        for b in self.branches:
            b.bind(tensors, rt)
        if not self.fused:
            return
        ins = [b.in_proj() for b in self.branches]
        # a feed-forward whose activation the product's epilogue can take comes last, its rows at a multiple of 16
        self.tail = len(ins) - 1 if getattr(self.branches[-1], "epilogue_act", None) == "relu2" and self.scales[-1] == 1.0 else None
        if self.tail is not None and rt.dtype == torch.bfloat16 and len(ins) > 1:
            fill = -sum(w.shape[0] for w, _ in ins[:-1]) % 16
            w, bias = ins[-2]
            if fill:
                ins[-2] = (torch.cat([w, w.new_zeros((fill, w.shape[1]))], dim=0),
                           None if bias is None else torch.cat([bias, bias.new_zeros(fill)]))
        self.w_in = torch.cat([w for w, _ in ins], dim=0).contiguous()
        self.b_in = None
        if any(bias is not None for _, bias in ins):
            self.b_in = torch.cat([bias.float() if bias is not None
                                   else torch.zeros(w.shape[0], dtype=torch.float32, device=w.device)
                                   for w, bias in ins]).contiguous()
            if rt.dtype == torch.bfloat16 and torch.equal(self.b_in.to(torch.bfloat16).float(), self.b_in):
                self.b_in = self.b_in.to(torch.bfloat16)         # as stored: the library product then adds it in its epilogue
        self.in_cols, self.act_cols, self.gaps = [], [], []
        c = a = 0
        outs = [b.out_proj() for b in self.branches]
        cols = []                                   # the stacked output matrix: the branches' columns and the zeros between
        for i, w in enumerate(outs):
            n = w.shape[1]
            unit = 32 if i + 1 == len(outs) else 8
            fill = -(a + n) % unit
            cols += [w] + ([w.new_zeros((w.shape[0], fill))] if fill else [])
            self.act_cols.append(a)
            if fill:
                self.gaps.append((a + n, a + n + fill))
            a += n + fill
        self.w_o = torch.cat(cols, dim=1).contiguous()
        self.n_act = a
        for b, (w, _) in zip(self.branches, ins):
            self.in_cols.append(c)
            # the branch keeps views of the stacked matrices instead of copies of its own (rows of w_in are
            # contiguous; its columns of w_o are not, so alone it can no longer run)
            b.w_in = self.w_in[c:c + w.shape[0]]
            c += w.shape[0]
            b.w_o = None
            tensors.pop(f"{b.prefix}.{getattr(b, 'out_name', 'o')}", None)

    def weight_bytes(self) -> int:
        if not self.fused:
            return sum(b.weight_bytes() for b in self.branches)
        return (sum(b.weight_bytes() for b in self.branches)
                + self.w_o.numel() * self.w_o.element_size())

    def first_weights(self) -> Optional[torch.Tensor]:
        return self.w_in if self.fused else self.branches[0].first_weights()

    def _sub(self, lc: LayerCache, i: int) -> LayerCache:
        pre = self.names[i] + "."
        return LayerCache(lc.group if self.branches[i].kv_request() is not None else None, lc.layer, lc.writes,
                          {k[len(pre):]: v for k, v in lc.states.items() if k.startswith(pre)})

    def forward(self, ctx, x: torch.Tensor, lc: LayerCache) -> torch.Tensor:
        T, ws, rt = ctx.T, ctx.ws, self.rt
        if self.fused:
            N, Kd = self.w_in.shape
            proj = ws.get("par_proj", (T, N), x.dtype)
            act = ws.get("par_act", (T, self.n_act), x.dtype)
            tail, branches = None, list(enumerate(self.branches))
            if self.tail is not None and takes_tail(T, N, Kd, x.dtype, self.in_cols[-1], self.n_act, self.act_cols[-1]):
                tail, branches = (self.in_cols[-1], act, self.act_cols[-1]), branches[:-1]
            matmul(x, self.w_in, self.b_in, proj, status=rt.status, tail=tail)
            for lo, hi in self.gaps:
                act[:, lo:hi].zero_()
            for i, b in branches:
                b.inner(ctx, proj, self.in_cols[i], self._sub(lc, i), act, self.act_cols[i], self.scales[i])
            out = ws.get("mixer_out", (T, self.hidden_size), x.dtype)
            return matmul(act, self.w_o, None, out, target_ctas=4 * rt.sm_count, status=rt.status, upcoming=ctx.upcoming)
        total = ws.get("par_sum", (T, self.hidden_size), torch.float32)
        for i, b in enumerate(self.branches):
            y = b.forward(ctx, x, self._sub(lc, i))
            if y.dim() == 3:
                raise ValueError(f"{self.prefix}: a branch returned partial sums it was not asked for")
            K.axpy_f32(total, y, self.scales[i], accumulate=i > 0)
        return total
