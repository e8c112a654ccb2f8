"""Layers whose norms sit on what a sub-layer puts out, with what such a layer can have around its sub-layers: a short
causal convolution over time added to the mixer's input, and a learned average over the depth of the model after the
layer.

A sub-layer's output y enters the float32 stream as x <- x + norm(y).  Like the residual add of the pre-norm layers this
is left *pending* (``PendingPost``): whoever needs the stream next - the next sub-layer, the next layer, the final norm -
completes it in the kernel that makes its own input (``K.post_norm``, ``csrc/post_norm.cu``): normed add, depth average,
then a plain copy in the model's dtype, the convolved input of a step of single tokens, or another norm."""

from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List, Optional, Union

import torch

from .. import kernels as K
from ..cache.paged import StateSpec
from ..registry import register_part
from ..weights.spec import TensorSpec
from .base import Block, LayerCache, Norm, Part, Runtime
from .moe import PendingExperts


@dataclass
class PendingPost:
    """A sub-layer's output that is not in the stream yet."""
    y: Union[torch.Tensor, PendingExperts]      # [T, H] in the model's dtype, or a routed feed-forward's unsummed rows
    norm: "GroupedRMSNorm"                      # the norm it passes on its way into the stream
    depth: Optional["DepthAverage"] = None      # the average that follows it, if it ends a layer
    history: Optional[torch.Tensor] = None      # [layers, T, H] float32: the embedding output and the layers' results


def complete(pending: Optional[PendingPost], resid: torch.Tensor, out: Optional[torch.Tensor], **how) -> None:
    """Bring ``pending`` into ``resid`` and make ``out`` from the completed stream (``how``: see ``K.post_norm``)."""
    if pending is None:
        K.post_norm(None, None, 1, 0.0, resid, out, **how)
        return
    n, d = pending.norm, pending.depth
    if d is not None:
        how.update(history=pending.history, n_history=d.index + 1, depth_weights=d.weight)
        # the layer's own result is kept for the averages of later layers
        if how.get("write_resid", True) and d.index + 1 < d.n_layers:
            how.update(put_history=d.index + 1)
    K.post_norm(pending.y, n.weight, n.groups, n.eps, resid, out, **how)


@register_part("norm", "grouped_rmsnorm")
class GroupedRMSNorm(Norm):
    """norm(y): y in ``groups`` equal parts of neighbouring channels, each over its own sqrt(mean(part^2) + eps), the whole
    times ``weight`` [size].  In a post-norm layer the block hands it to whoever completes the stream; as the final norm
    its ``forward`` completes the pending sub-layer and norms the stream at the wanted rows in one kernel.  Float32."""

    def __init__(self, prefix: str, size: int, eps: float, groups: int = 1, tensor: Optional[str] = None,
                 optional: bool = False):
        if groups < 1 or size % groups:
            raise ValueError(f"{prefix or tensor}: {size} channels do not form {groups} equal groups")
        self.name = tensor or f"{prefix}.weight"
        self.size, self.eps, self.groups, self.optional = size, float(eps), int(groups), bool(optional)

    def tensor_specs(self) -> List[TensorSpec]:
        return [TensorSpec(self.name, (self.size,), "vector", optional=self.optional, init="norm")]

    def bind(self, tensors: Dict[str, torch.Tensor], rt: Runtime) -> None:
        self.rt = rt
        w = tensors.get(self.name)
        self.weight = None if w is None else w.float().contiguous()

    def forward(self, ctx, delta: Optional[PendingPost], resid: torch.Tensor, out: torch.Tensor,
                rows: Optional[torch.Tensor] = None, n_out: Optional[int] = None, write_resid: bool = True) -> None:
        complete(delta, resid, out, rows=rows, n_out=n_out, write_resid=write_resid, out_weight=self.weight,
                 out_groups=self.groups, out_eps=self.eps)


@register_part("depth_average", "learned_average")
class DepthAverage(Part):
    """x <- sum over j = 0 .. index + 1 of a_j X_j with X_0 the embedding output and X_(j+1) the result of layer j before
    its own average; a = ``tensor`` [index + 2].  Float32."""
    kind = "depth_average"

    def __init__(self, prefix: str, index: int, n_layers: int, tensor: Optional[str] = None):
        if not 0 <= index < n_layers:
            raise ValueError(f"{prefix or tensor}: layer {index} of {n_layers}")
        self.name = tensor or f"{prefix}.weight"
        self.index, self.n_layers = index, n_layers

    def tensor_specs(self) -> List[TensorSpec]:
        return [TensorSpec(self.name, (self.index + 2,), "vector", init="depth")]

    def bind(self, tensors: Dict[str, torch.Tensor], rt: Runtime) -> None:
        self.rt = rt
        self.weight = tensors[self.name].float().contiguous()

    def history(self, ctx, width: int) -> torch.Tensor:
        return ctx.ws.get("depth_history", (self.n_layers, ctx.T, width), torch.float32)


@register_part("input_conv", "causal_conv")
class CausalConv(Part):
    """u_t = h_t + sum_j w[:, j] h_(t - taps + 1 + j): a causal convolution over time on each channel, added to its input,
    zeros before the sequence's start.  ``tensor`` [channels, taps].  The last taps - 1 inputs of a sequence are kept in
    float32 per cache slot; the sums are float32 and rounded once."""
    kind = "input_conv"

    STATE = "input_conv"

    def __init__(self, prefix: str, channels: int, taps: int, tensor: Optional[str] = None):
        if taps < 1 or channels < 1:
            raise ValueError(f"{prefix or tensor}: {taps} taps on {channels} channels")
        self.name = tensor or f"{prefix}.weight"
        self.channels, self.taps = channels, taps

    def tensor_specs(self) -> List[TensorSpec]:
        return [TensorSpec(self.name, (self.channels, self.taps), "vector", init="conv_small")]

    def state_requests(self) -> List[StateSpec]:
        return [StateSpec(self.STATE, (self.taps - 1, self.channels), torch.float32)] if self.taps > 1 else []

    def bind(self, tensors: Dict[str, torch.Tensor], rt: Runtime) -> None:
        self.rt = rt
        self.weight = tensors[self.name].float().t().contiguous()          # [taps, channels]

    def weight_bytes(self) -> int:
        return self.weight.numel() * 4

    def forward(self, ctx, resid: torch.Tensor, out: torch.Tensor, lc: LayerCache) -> None:
        """Steps with longer portions: ``out`` from the completed stream, then the state."""
        state = lc.states.get(self.STATE)
        K.stream_conv(resid, self.weight, state, out, ctx.tok_row, ctx.row_slot, ctx.row_q_start)
        if state is not None and lc.writes:
            K.conv_state_update(resid, state, ctx.row_slot, ctx.row_q_start, ctx.row_q_len, ctx.n_rows)


@register_part("block", "postnorm")
class PostNormBlock(Block):
    """u = x + conv(x) (``input_conv``, optional; u = x without);  x += norm1(mixer(u));  x += norm2(feed_forward(x)) (or no
    feed-forward; a ``norm2`` given all the same declares its tensor and never runs);  then x <- the learned average of
    the embedding output and all layers' results so far (``depth``, optional).  Takes and returns a ``PendingPost``."""

    completes_stream = True

    def __init__(self, norm1, mixer, norm2=None, feed_forward=None, input_conv=None, depth=None):
        self.norm1, self.mixer, self.norm2, self.feed_forward = norm1, mixer, norm2, feed_forward
        self.input_conv, self.depth = input_conv, depth
        if feed_forward is not None and norm2 is None:
            raise ValueError("a post-norm layer with a feed-forward needs its second norm")

    def parts(self):
        return [p for p in (self.input_conv, self.norm1, self.mixer, self.norm2, self.feed_forward, self.depth)
                if p is not None]

    def extra_state_requests(self) -> List[StateSpec]:
        return self.input_conv.state_requests() if self.input_conv is not None else []

    def first_weights(self) -> Optional[torch.Tensor]:
        return self.mixer.first_weights()

    def forward(self, ctx, resid: torch.Tensor, delta: Optional[PendingPost], lc: LayerCache) -> PendingPost:
        dt, after_block = ctx.rt.dtype, ctx.upcoming
        xin = ctx.ws.get("sublayer_in", tuple(resid.shape), dt)
        history = self.depth.history(ctx, resid.shape[1]) if self.depth is not None else None
        how = {}
        if delta is None and history is not None and self.depth.index == 0:
            how = dict(history=history, put_history=0)             # X_0, the embedding output
        if self.input_conv is None:
            complete(delta, resid, xin, **how)
        elif ctx.max_q_len == 1 and (lc.writes or self.input_conv.taps == 1):
            complete(delta, resid, xin, conv_weight=self.input_conv.weight, conv_state=lc.states.get(CausalConv.STATE),
                     tok_row=ctx.tok_row, row_slot=ctx.row_slot, **how)
        else:
            complete(delta, resid, None, **how)
            self.input_conv.forward(ctx, resid, xin, lc)
        if self.feed_forward is None:
            return PendingPost(self.mixer.forward(ctx, xin, lc), self.norm1, self.depth, history)
        ctx.upcoming = self.feed_forward.first_weights()
        y = self.mixer.forward(ctx, xin, lc)
        complete(PendingPost(y, self.norm1), resid, xin)
        ctx.upcoming = after_block
        if getattr(self.feed_forward, "offers_pairs", False):
            y = self.feed_forward.forward(ctx, xin, pairs_ok=True)
        else:
            y = self.feed_forward.forward(ctx, xin)
        return PendingPost(y, self.norm2, self.depth, history)

    def stream_state(self, resid: torch.Tensor, delta: Optional[PendingPost]) -> torch.Tensor:
        out = torch.empty_like(resid)
        complete(delta, resid, out, write_resid=False)
        return out
