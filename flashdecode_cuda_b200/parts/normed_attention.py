"""Attention mixers over normed projections: grouped-query attention whose q and k are normed over their whole
projection, with a sliding window; and latent attention, which keeps one low-rank vector (and by option one small
rotated key part) per position and makes every head's keys and values from it."""

from __future__ import annotations

from typing import Dict, List, Optional

import torch

from .. import kernels as K
from ..registry import register_part
from ..weights.spec import TensorSpec
from .attention import FP32_SPLIT_LEN, plan_splits
from .base import KVRequest, LayerCache, Mixer, Runtime
from .linear import matmul


def decode_splits(ctx, n_q: int, n_kv: int, v_dim: int, dtype: torch.dtype, rt: Runtime, head_dim: int = 0, window: int = 0):
    """(n_splits, split_len, scratch) of a step's attention: a step of single tokens cuts every sequence's keys into
    splits (float32: of a fixed length, so that where a sequence's partial sums are cut depends on its own length only;
    bfloat16: by the batch's size and, if ``window`` is given, for the keys it shows, so that the CTAs that find keys are
    about as many as the SMs); any other step does not."""
    if ctx.max_q_len != 1:
        return 1, 0, None
    if dtype == torch.float32:
        split_len = FP32_SPLIT_LEN
        n_splits = max(1, -(-ctx.kv_len_bound // split_len))
    else:
        # (the tensor-core kernel cuts a large group of query heads into several, each with CTAs of its own)
        heads = K.attention_decode_heads(n_q, n_kv, head_dim, v_dim) if head_dim else n_kv
        bound = ctx.kv_len_bound
        n_splits, split_len = plan_splits(ctx.n_rows, heads, min(bound, window + 32) if window else bound, rt.sm_count)
        n_splits = max(1, -(-bound // split_len))
        if window and n_splits > 64:                # bounded scratch memory and merge
            split_len = -(-(-(-bound // 64)) // 32) * 32
            n_splits = -(-bound // split_len)
    scratch = None
    if n_splits > 1:
        scratch = ctx.ws.get("attn_scratch", (K.attention_scratch_floats(ctx.T, n_q, v_dim, n_splits),), torch.float32)
    return n_splits, split_len, scratch


def _up8(n: int) -> int:
    return -(-n // 8) * 8


def tensor_core_sizes(head_dim: int, v_head_dim: int):
    """(key, value) head sizes as the kernels should see them: both 64 or both 128, which the tensor-core attention kernels
    take, where filling up with zeros costs at most 60 % more of the cache; else the next multiples of 8."""
    widest = max(head_dim, v_head_dim)
    size = 64 if widest <= 64 else 128
    if widest <= 128 and 2 * size <= 1.6 * (head_dim + v_head_dim):
        return size, size
    return _up8(head_dim), _up8(v_head_dim)


def _head_sizes_ok(prefix: str, **sizes: int) -> None:
    """The attention kernels take head sizes that are multiples of 8 up to 512; other sizes are padded with zeros to
    the next multiple when the weights are bound (zero rows of the projections, zero norm weights), which changes no
    score and no output."""
    for what, n in sizes.items():
        if n < 1 or _up8(n) > 512:
            raise ValueError(f"{prefix}: {what.replace('_', ' ')} {n} is not taken: the attention kernels take sizes "
                             f"from 1 to 512")


def _pad_heads(w: torch.Tensor, n_heads: int, size: int, padded: int) -> torch.Tensor:
    """w [n_heads * size, ...] -> [n_heads * padded, ...]: zero rows after every head's own."""
    if size == padded:
        return w
    out = w.new_zeros((n_heads, padded) + tuple(w.shape[1:]))
    out[:, :size] = w.view((n_heads, size) + tuple(w.shape[1:]))
    return out.view((n_heads * padded,) + tuple(w.shape[1:]))


def _pad_cols(w: torch.Tensor, size: int, padded: int) -> torch.Tensor:
    """w [N, size] -> [N, padded]: zero columns at the end."""
    if size == padded:
        return w.contiguous()
    out = w.new_zeros((w.shape[0], padded))
    out[:, :size] = w
    return out


def _pad_split_heads(w: torch.Tensor, n_heads: int, *parts) -> torch.Tensor:
    """w [n_heads * sum of sizes, ...] whose heads have several parts, each (size, padded size): zero rows after each."""
    out = w.new_zeros((n_heads, sum(p for _, p in parts)) + tuple(w.shape[1:]))
    rows = w.view((n_heads, sum(s for s, _ in parts)) + tuple(w.shape[1:]))
    a = b = 0
    for size, padded in parts:
        out[:, b:b + size] = rows[:, a:a + size]
        a, b = a + size, b + padded
    return out.view((-1,) + tuple(w.shape[1:]))


@register_part("mixer", "qk_normed_attention")
class QKNormedAttention(Mixer):
    """For the mixer's input h [T, hidden]:

        q, k, v = W_q h, W_k h, W_v h                           (``bias``: + ``.q.b``, ``.k.b``, ``.v.b``)
        q       = q / sqrt(mean(q^2) + eps) * w_q               over ALL of q's n_heads * head_dim values at once,
        k       = k / sqrt(mean(k^2) + eps) * w_k               likewise; then both are split into heads
        q, k    = rotation of every head's first ``rot_dims`` dimensions (i paired with i + rot_dims / 2), if any
        q, k    = x / sqrt(mean(x^2) + eps) per head, without a weight                  (``head_norm``)
        v       = (1 - lam) v + lam v_first                     (``value_mix``, below)
        a       = softmax over the visible keys of (q . k) * scale; query head h reads key/value head
                  h // (n_heads / n_kv_heads); value heads have ``v_head_dim`` dimensions
        out     = W_o a

    Without ``rot_dims`` positions enter through visibility alone.  Visible keys of the query at position i: j <= i,
    and with a ``window`` only i - j < window.  ``qk_norm`` False: q and k are used as projected.  ``softcap``: score <-
    softcap * tanh(score / softcap) after scaling.  ``sink``: exp(``.sink``[h]) is one more term of head h's denominator,
    without key or value.  ``value_mix``: "source" leaves the layer's values of the step's tokens for other layers,
    "mix" mixes them into its own values with lam = ``.vmix`` before they are cached; ``value_group`` names what they
    share.  One packed
    product gives q, k and v.  Tensors ``<prefix>.q`` / ``.k`` / ``.v`` / ``.o`` (stored [out, in]), ``.q.norm``,
    ``.k.norm``.  Norms, rotation, scores, softmax and mixing are float32 in both dtypes.  Other mixers, or a feed-forward,
    may share its input and output products (``parts.parallel``).
    """

    shares_products = True

    def __init__(self, prefix: str, hidden_size: int, n_heads: int, n_kv_heads: int, head_dim: int, v_head_dim: int,
                 scale: float, eps: float, window: Optional[int] = None, qk_norm: bool = True, bias: bool = False,
                 position=None, rot_dims: int = 0, head_norm: bool = False, softcap: Optional[float] = None, sink: bool = False,
                 value_mix: Optional[str] = None, value_group: str = "values"):
        _head_sizes_ok(prefix, head_size=head_dim, value_head_size=v_head_dim)
        if rot_dims < 0 or rot_dims % 2 or rot_dims > head_dim or (rot_dims and position is None):
            raise ValueError(f"{prefix}: {rot_dims} rotated dimensions of {head_dim}: they must be even and given a position part")
        if value_mix not in (None, "source", "mix") or (softcap is not None and not softcap > 0):
            raise ValueError(f"{prefix}: value mixing {value_mix!r} (None, 'source' or 'mix'), a soft cap of {softcap} (positive or None)")
        if n_kv_heads < 1 or n_heads % n_kv_heads != 0 or n_heads // n_kv_heads > 64:
            raise ValueError(f"{prefix}: {n_heads} query heads for {n_kv_heads} key/value heads: the kernels take whole "
                             f"groups of up to 64 query heads per key/value head")
        if window is not None and window < 1:
            raise ValueError(f"{prefix}: a window of {window} positions")
        self.prefix, self.hidden_size = prefix, hidden_size
        self.n_q, self.n_kv, self.d, self.dv = n_heads, n_kv_heads, head_dim, v_head_dim
        # head sizes as the kernels see them
        self.dp, self.dvp = tensor_core_sizes(head_dim, v_head_dim)
        self.scale, self.eps, self.window, self.qk_norm = float(scale), float(eps), window, qk_norm
        self.bias, self.position, self.rot_dims, self.head_norm = bool(bias), position, int(rot_dims), bool(head_norm)
        self.softcap, self.has_sink, self.value_mix, self.value_group = softcap, bool(sink), value_mix, value_group
        self.extended = bool(softcap or sink)
        # what the plain append kernel does not have
        self.turned = bool(rot_dims or head_norm or value_mix)

    def _sizes(self):
        return (("q", self.n_q * self.d), ("k", self.n_kv * self.d), ("v", self.n_kv * self.dv))

    def tensor_specs(self) -> List[TensorSpec]:
        p, H = self.prefix, self.hidden_size
        specs = [TensorSpec(f"{p}.{n}", (c, H), init="unit") for n, c in self._sizes()]
        if self.qk_norm:
            specs += [TensorSpec(f"{p}.q.norm", (self.n_q * self.d,), "vector", init="norm"),
                      TensorSpec(f"{p}.k.norm", (self.n_kv * self.d,), "vector", init="norm")]
        if self.bias:
            specs += [TensorSpec(f"{p}.{n}.b", (c,), "vector", init="bias") for n, c in self._sizes()]
        if self.has_sink:
            specs.append(TensorSpec(f"{p}.sink", (self.n_q,), "vector", init="sink"))
        if self.value_mix:          # (the source's own constant is never read)
            specs.append(TensorSpec(f"{p}.vmix", (), "vector", optional=self.value_mix == "source", init="half"))
        specs.append(TensorSpec(f"{p}.o", (H, self.n_q * self.dv), init="unit"))
        return specs

    def kv_request(self) -> KVRequest:
        return KVRequest(self.n_kv, self.dp, self.window, None, self.dvp)

    def bind(self, tensors: Dict[str, torch.Tensor], rt: Runtime) -> None:
        self.rt = rt
        p = self.prefix
        heads = {"q": (self.n_q, self.d, self.dp), "k": (self.n_kv, self.d, self.dp), "v": (self.n_kv, self.dv, self.dvp)}
        self.w_in = torch.cat([_pad_heads(tensors.pop(f"{p}.{n}"), *heads[n]) for n, _ in self._sizes()], dim=0).contiguous()
        self.b_in = None
        if self.bias:
            self.b_in = torch.cat([_pad_heads(tensors.pop(f"{p}.{n}.b"), *heads[n]) for n, _ in self._sizes()]).contiguous()
        self.sink_w = tensors.pop(f"{p}.sink").float().contiguous() if self.has_sink else None
        self.lam = tensors.pop(f"{p}.vmix").float().reshape(1).contiguous() if self.value_mix == "mix" else None
        self.q_norm = self.k_norm = None
        if self.qk_norm:
            self.q_norm = _pad_heads(tensors[f"{p}.q.norm"].float(), *heads["q"]).contiguous()
            self.k_norm = _pad_heads(tensors[f"{p}.k.norm"].float(), *heads["k"]).contiguous()
        w_o = tensors[f"{p}.o"]
        if self.dvp != self.dv:             # zero columns where the padded value dimensions arrive
            w_o = _pad_heads(w_o.t().contiguous(), self.n_q, self.dv, self.dvp).t().contiguous()
            tensors[f"{p}.o"] = w_o
        self.w_o = w_o

    def weight_bytes(self) -> int:
        return sum(w.numel() * w.element_size() for w in (self.w_in, self.w_o) if w is not None)

    def first_weights(self) -> Optional[torch.Tensor]:
        return self.w_in

    def in_proj(self):
        return self.w_in, self.b_in

    def out_proj(self) -> torch.Tensor:
        return self.w_o

    def inner(self, ctx, proj: torch.Tensor, col0: int, lc: LayerCache, act: torch.Tensor, act_col: int = 0,
              scale: float = 1.0) -> torch.Tensor:
        T, ws, rt = ctx.T, ctx.ws, self.rt
        q = ws.get("nat_q", (T, self.n_q * self.dp), proj.dtype)
        counts = dict(q_count=self.n_q * self.d, k_count=self.n_kv * self.d)
        if self.turned or col0:
            v_first = None
            if self.value_mix:
                v_first = ws.get(f"first_{self.value_group}", (T, self.n_kv * self.dv), proj.dtype)
            mode = {None: K.VALUES_PLAIN, "source": K.VALUES_SOURCE, "mix": K.VALUES_MIXED}[self.value_mix]
            rope = self.position
            K.rope_norm_append(proj, col0, q, lc.k_pool, lc.v_pool, lc.group.table, self.q_norm, self.k_norm, self.eps,
                               rope.cos if self.rot_dims else None, rope.sin if self.rot_dims else None, self.rot_dims,
                               self.head_norm, ctx.tok_row, ctx.tok_pos, ctx.row_slot, self.n_q, self.n_kv, self.dp, self.dvp,
                               lc.writes, rt.status, head_count=self.d, value_mode=mode, v_first=v_first, lam=self.lam,
                               v_count=self.dv, **counts)
        else:
            K.norm_append(proj, q, self.q_norm, self.k_norm, self.eps, ctx.tok_row, ctx.tok_pos, ctx.row_slot, lc.k_pool,
                          lc.v_pool, lc.group.table, self.n_kv, lc.writes, rt.status, **counts)
        n_splits, split_len, scratch = decode_splits(ctx, self.n_q, self.n_kv, self.dvp, proj.dtype, rt, self.dp,
                                                     (self.window or 0) if self.turned else 0)
        args = (q, lc.k_pool, lc.v_pool, act, lc.group.table, ctx.tok_row, ctx.row_slot, ctx.row_q_start, ctx.row_q_len,
                ctx.row_ctx_len, ctx.n_rows, ctx.max_q_len, self.n_q, self.n_kv, self.dp, self.scale, self.window or 0, n_splits,
                split_len, scratch, rt.status)
        if self.extended:
            K.attention_ext(*args, softcap=self.softcap or 0.0, sink=self.sink_w, out_col=act_col, out_scale=scale)
        else:
            K.attention(*args, out_col=act_col, out_scale=scale)
        return act

    def forward(self, ctx, x: torch.Tensor, lc: LayerCache) -> torch.Tensor:
        T, ws, rt = ctx.T, ctx.ws, self.rt
        proj = ws.get("nat_proj", (T, self.w_in.shape[0]), x.dtype)
        matmul(x, self.w_in, self.b_in, proj, status=rt.status)
        attn = ws.get("nat_attn", (T, self.n_q * self.dvp), x.dtype)
        self.inner(ctx, proj, 0, lc, attn)
        out = ws.get("mixer_out", (T, self.hidden_size), x.dtype)
        return matmul(attn, self.w_o, None, out, target_ctas=4 * rt.sm_count, status=rt.status)


@register_part("mixer", "latent_attention")
class LatentAttention(Mixer):
    """For the mixer's input h [T, hidden], with ``n_heads`` heads, ``head_dim`` query/key and ``v_head_dim`` value
    dimensions per head and a latent of ``kv_rank`` dimensions:

        q   = W_q h                                        or, with ``q_rank``, W_uq norm(W_dq h): through a latent of its own
        c   = (W_dkv h) / sqrt(mean((W_dkv h)^2) + eps) * w_c           the latent: cached
        k_h = U_h c,  v_h = V_h c                          (U = ``.uk`` [heads * head_dim, kv_rank], V = ``.uv``, head by head)
        a_h = softmax over the visible keys j of (q_h . k_h[j]) * scale
        out = W_o [a_1 V-values ... ]

    ``rot_dim`` > 0: a head's query has ``rot_dim`` more dimensions and W_dkv as many more rows, one key part k_r for all
    heads; both are turned at their positions (``position``: pairs 2i, 2i + 1), q_h . k_h gains q_r,h . k_r, and k_r is cached
    beside c.  ``sink``: exp(``.sink``[h]) is one more term of head h's denominator, without key or value.  ``gate``: the
    concatenated heads are multiplied by sigmoid(W_g h).

    Computed without ever expanding the cached positions: (q_h . U_h c) = (U_h^T q_h) . c, so the queries are taken
    into the latent's basis (one small product per head), attention runs over the cached rows [c ; k_r] as ONE key/value
    head that all query heads share and whose first ``kv_rank`` dimensions are the values, and V_h is applied to each
    head's attended latent afterwards.  Visible keys: j <= i, and with a ``window`` only i - j < window.

    Whole prompts in bfloat16 (a step whose sequences all start at their first token) take the other order where that
    reaches a faster attention kernel: k_h and v_h of the step's own tokens are expanded by one product, and attention runs
    over them with a key/value head per query head (``expands``); the cache still receives [c ; k_r] only.  Tensors
    ``<prefix>.q`` (or ``.dq``, ``.dq.norm``, ``.uq``), ``.dkv``, ``.dkv.norm``, ``.uk``, ``.uv``, ``.sink``, ``.g``, ``.o``.
    """

    def __init__(self, prefix: str, hidden_size: int, n_heads: int, head_dim: int, v_head_dim: int, kv_rank: int,
                 scale: float, eps: float, window: Optional[int] = None, q_rank: Optional[int] = None, rot_dim: int = 0,
                 position=None, sink: bool = False, gate: bool = False):
        _head_sizes_ok(prefix, latent_size=kv_rank)
        if n_heads < 1 or head_dim < 1 or v_head_dim < 1 or (q_rank is not None and q_rank < 1):
            raise ValueError(f"{prefix}: {n_heads} heads of {head_dim} / {v_head_dim}, query latent {q_rank}")
        if rot_dim < 0 or rot_dim % 2 or (rot_dim and position is None) or _up8(kv_rank) + _up8(rot_dim) > 640:
            raise ValueError(f"{prefix}: a rotated part of {rot_dim} dimensions beside a latent of {kv_rank}: it must be even "
                             f"and both together at most 640")
        self.prefix, self.hidden_size = prefix, hidden_size
        self.n_q, self.d, self.dv, self.r_true, self.rot = n_heads, head_dim, v_head_dim, kv_rank, rot_dim
        self.r = _up8(kv_rank)                     # the latent as the kernels see it: zero-padded to a multiple of 8
        self.rp = _up8(rot_dim)                    # ... and the rotated part
        self.q_rank, self.position, self.has_sink, self.has_gate = q_rank, position, bool(sink), bool(gate)
        self.scale, self.eps, self.window = float(scale), float(eps), window

    def tensor_specs(self) -> List[TensorSpec]:
        p, H = self.prefix, self.hidden_size
        r, nq = self.r_true, self.n_q * (self.d + self.rot)
        if self.q_rank is None:
            specs = [TensorSpec(f"{p}.q", (nq, H), init="unit")]
        else:
            specs = [TensorSpec(f"{p}.dq", (self.q_rank, H), init="unit"),
                     TensorSpec(f"{p}.dq.norm", (self.q_rank,), "vector", init="norm"),
                     TensorSpec(f"{p}.uq", (nq, self.q_rank), init="unit")]
        specs += [TensorSpec(f"{p}.dkv", (r + self.rot, H), init="unit"),
                  TensorSpec(f"{p}.dkv.norm", (r,), "vector", init="norm"),
                  TensorSpec(f"{p}.uk", (self.n_q * self.d, r), init="unit"),
                  TensorSpec(f"{p}.uv", (self.n_q * self.dv, r), init="unit")]
        if self.has_sink:
            specs.append(TensorSpec(f"{p}.sink", (self.n_q,), "vector", init="sink"))
        if self.has_gate:
            specs.append(TensorSpec(f"{p}.g", (self.n_q * self.dv, H), init="unit"))
        return specs + [TensorSpec(f"{p}.o", (H, self.n_q * self.dv), init="unit")]

    def kv_request(self) -> KVRequest:
        return KVRequest(1, self.r + self.rp, self.window, None, None, keys_only=True)

    def bind(self, tensors: Dict[str, torch.Tensor], rt: Runtime) -> None:
        self.rt = rt
        p, n = self.prefix, self.n_q
        pad = lambda w: _pad_heads(w, 1, self.r_true, self.r)            # zero rows up to the padded latent size
        # Sizes of a head's parts in the activations: as they are, or, where whole prompts run on the tcgen05 kernel over
        # plain rows, filled up with zeros to multiples of 64 (zero rows of the projections: no score and no output changes)
        self.dx, self.rx, self.vx = self.d, self.rot, self.dv
        up64 = lambda size: -(-size // 64) * 64
        dx, rx, vx = up64(self.d), up64(self.rot), up64(self.dv)
        if dx + rx == 64 and vx == 128:
            dx = 128
        expanded = 3 if K.attention_dense_takes(dx, rx, vx) else 0
        # which attention kernel the cached row itself reaches (3 tcgen05, 2 mma.sync, 1 mma.sync at wide heads, 0 others)
        latent = {128: 3, 64: 2, 192: 1, 256: 1}.get(self.r, 0) if not (self.rot or self.has_sink) else 0
        self.expands = rt.dtype == torch.bfloat16 and (expanded > latent or (expanded == latent > 0 and 2 * self.r > dx + vx))
        if self.expands:
            self.dx, self.rx, self.vx = dx, rx, vx
        self.kx = self.dx + self.rx
        w_q = tensors.pop(f"{p}.q" if self.q_rank is None else f"{p}.uq")
        dkv = tensors.pop(f"{p}.dkv")
        w_q = _pad_split_heads(w_q, n, (self.d, self.dx), (self.rot, self.rx))
        qr = self.qr = 0 if self.q_rank is None else _up8(self.q_rank)
        first = w_q if self.q_rank is None else _pad_heads(tensors.pop(f"{p}.dq"), 1, self.q_rank, qr)
        mats = [first, pad(dkv[:self.r_true]), _pad_heads(dkv[self.r_true:], 1, self.rot, self.rp)]     # [q | latent | k_r | gate]
        self.gate_col = sum(m.shape[0] for m in mats)
        if self.has_gate:
            mats.append(_pad_heads(tensors.pop(f"{p}.g"), n, self.dv, self.vx))
        self.w_in = torch.cat(mats, dim=0).contiguous()
        self.w_uq = self.q_norm = None
        if self.q_rank is not None:
            self.w_uq = _pad_cols(w_q, self.q_rank, qr)
            self.q_norm = _pad_heads(tensors[f"{p}.dq.norm"].float(), 1, self.q_rank, qr).contiguous()
        self.c_norm = pad(tensors[f"{p}.dkv.norm"].float()).contiguous()
        # per head: U_h^T [kv_rank, head_dim] takes a query into the latent's basis; V_h [v_head_dim, kv_rank]
        uk = _pad_cols(_pad_heads(tensors.pop(f"{p}.uk"), n, self.d, self.dx), self.r_true, self.r)
        uv = _pad_cols(_pad_heads(tensors.pop(f"{p}.uv"), n, self.dv, self.vx), self.r_true, self.r)
        self.w_qc = uk.view(n, self.dx, self.r).transpose(1, 2).contiguous()
        self.w_cv = uv.view(n, self.vx, self.r).contiguous()
        w_o = tensors[f"{p}.o"]
        if self.vx != self.dv:              # zero columns where the filled-up value dimensions arrive
            w_o = _pad_heads(w_o.t().contiguous(), n, self.dv, self.vx).t().contiguous()
            tensors[f"{p}.o"] = w_o
        self.w_o = w_o
        self.sink = tensors[f"{p}.sink"].float().contiguous() if self.has_sink else None
        # [heads (dx + vx), kv_rank]: head by head its key rows, then its value rows
        self.w_kv = torch.cat([uk.view(n, self.dx, self.r), uv.view(n, self.vx, self.r)], dim=1).reshape(
            n * (self.dx + self.vx), self.r).contiguous() if self.expands else None

    def weight_bytes(self) -> int:
        # (the expansion matrix is a second copy of .uk and .uv in another order: a step reads one of the two)
        mats = [self.w_in, self.w_qc, self.w_cv, self.w_o] + ([self.w_uq] if self.w_uq is not None else [])
        return sum(w.numel() * w.element_size() for w in mats)

    def first_weights(self) -> Optional[torch.Tensor]:
        return self.w_in

    def _append(self, ctx, proj: torch.Tensor, first: torch.Tensor, lc: LayerCache, **rows) -> None:
        """The query latent normed (or the queries as they are) to ``first``, [c ; k_r] to the cache."""
        rope = self.position if self.rot else None
        K.norm_append(proj, first, self.q_norm, self.c_norm, self.eps, ctx.tok_row, ctx.tok_pos, ctx.row_slot, lc.k_pool,
                      None, lc.group.table, 1, lc.writes, self.rt.status, q_count=self.q_rank or 0, k_count=self.r_true,
                      cos=rope.cos if rope else None, sin=rope.sin if rope else None, rot=self.rot, rot_places=self.rp, **rows)

    def _queries(self, ctx, first: torch.Tensor) -> torch.Tensor:
        if self.w_uq is None:
            return first
        q = ctx.ws.get("lat_q", (ctx.T, self.n_q * self.kx), first.dtype)
        return matmul(first, self.w_uq, None, q, target_ctas=4 * self.rt.sm_count, status=self.rt.status)

    def forward(self, ctx, x: torch.Tensor, lc: LayerCache) -> torch.Tensor:
        T, ws, rt, n = ctx.T, ctx.ws, self.rt, self.n_q
        proj = ws.get("lat_proj", (T, self.w_in.shape[0]), x.dtype)
        matmul(x, self.w_in, None, proj, status=rt.status)
        first = ws.get("lat_q_in", (T, self.qr or n * self.kx), x.dtype)
        out = ws.get("mixer_out", (T, self.hidden_size), x.dtype)
        if self.expands and ctx.max_q_len > 1 and not any(ctx.h_ctx_len):
            # whole prompts: expand the step's own keys and values and attend over them as they lie
            c = ws.get("lat_c", (T, self.r), x.dtype)
            kr = ws.get("lat_kr", (T, self.rx), x.dtype) if self.rot else None
            self._append(ctx, proj, first, lc, k_rows=c, r_rows=kr)
            q = self._queries(ctx, first)
            if self.rot:
                K.rope_heads(q, self.kx, self.dx, q, self.kx, self.dx, self.position.cos, self.position.sin, ctx.tok_pos, n,
                             self.rot, self.rot, rt.status)
            kv = ws.get("lat_kv", (T, self.w_kv.shape[0]), x.dtype)
            matmul(c, self.w_kv, None, kv, status=rt.status)
            av = ws.get("lat_v", (T, n * self.vx), x.dtype)
            K.attention_dense(q, kv, kr, av, ctx.row_slot, ctx.row_q_start, ctx.row_q_len, ctx.row_ctx_len, ctx.n_rows,
                              ctx.max_q_len, n, self.dx, self.vx, self.scale, self.window or 0, self.sink,
                              proj if self.has_gate else None, self.gate_col if self.has_gate else 0, rt.status)
            return matmul(av, self.w_o, None, out, target_ctas=4 * rt.sm_count, status=rt.status)
        self._append(ctx, proj, first, lc)
        q = self._queries(ctx, first)
        size = self.r + self.rp
        qc = ws.get("lat_qc", (T, n * size), x.dtype)
        rope = (self.dx, self.r, self.rot, self.rp, self.position.cos, self.position.sin, ctx.tok_pos, rt.status) if self.rot else None
        K.head_gemm(q, self.w_qc, qc, a_size=self.kx, out_size=size, rope=rope)
        ac = ws.get("lat_ac", (T, n * self.r), x.dtype)
        # the latent kernel: bfloat16 steps except those whose row size a faster kernel takes without these options
        plain = not self.rot and not self.has_sink
        tensor_rows = x.dtype == torch.bfloat16 and not (plain and (self.r in (64, 128) or ctx.max_q_len > 1))
        if tensor_rows:
            per_cta = K.LATENT_HEADS[n > K.LATENT_HEADS[0]]
            n_splits, split_len, scratch = decode_splits(ctx, n, -(-n // per_cta), self.r, x.dtype, rt)
        else:
            n_splits, split_len, scratch = decode_splits(ctx, n, 1, self.r, x.dtype, rt, size if plain else 0)
        args = (qc, lc.k_pool, lc.k_pool, ac, lc.group.table, ctx.tok_row, ctx.row_slot, ctx.row_q_start, ctx.row_q_len,
                ctx.row_ctx_len, ctx.n_rows, ctx.max_q_len, n, 1, size, self.scale, self.window or 0, n_splits, split_len,
                scratch, rt.status)
        if tensor_rows or not plain:
            K.attention_ext(*args, sink=self.sink, value_dim=self.r if self.rot else 0)
        else:
            K.attention(*args)
        v = ws.get("lat_v", (T, n * self.vx), x.dtype)
        gated = self.has_gate and (T < K.HEAD_GEMM_LIBRARY_ROWS or x.dtype != torch.bfloat16)
        K.head_gemm(ac, self.w_cv, v, gate=proj if gated else None, gate_col=self.gate_col)
        if self.has_gate and not gated:
            K.gate_mul(v, proj, self.gate_col, v)
        return matmul(v, self.w_o, None, out, target_ctas=4 * rt.sm_count, status=rt.status, upcoming=ctx.upcoming)
