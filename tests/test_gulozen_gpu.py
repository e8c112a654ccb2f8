"""Gulozen on the GPU against the plain implementation: each mechanism's kernels alone, then whole models in float32
and bfloat16 - whole prompts, token-by-token decoding, portions down to two tokens, unequal batches against each
request alone, slots and pages used again, keys far away and at page borders, long decoding, greedy generation through
the engine's entry point and scheduler, the command line and the trace runner."""

import json
import subprocess
import sys
from pathlib import Path

import pytest
import torch

import flashdecode_cuda_b200 as fd
from flashdecode_cuda_b200 import kernels as K
from flashdecode_cuda_b200.parts.moe import PendingExperts
from flashdecode_cuda_b200.parts.rope import RotaryScaled
from helpers import prompts_for, rel_err
from gulozen_helpers import (GULOZEN, MODEL_TOL as TOL, Truth, decisive_routers, oracle_logits, plain_greedy, random_config,
                             raw_config, truth, weights_of, write_folder)
import gulozen_helpers as GH
from plain import gulozen_plain as P

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parent.parent
DEV = "cuda"
NAMES = ["A", "B", "C"]
DTYPES = ["float32", "bfloat16"]
TD = {"float32": torch.float32, "bfloat16": torch.bfloat16}
KTOL = {"float32": 2e-5, "bfloat16": 2e-2}


class _Rt:
    device = torch.device(DEV)


def i32(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


def step_arrays(ctx_lens, q_lens, slots):
    """Index arrays of a step whose rows bring q_lens[i] tokens after ctx_lens[i] cached ones."""
    tok_row, tok_pos, starts = [], [], []
    for r, (c, n) in enumerate(zip(ctx_lens, q_lens)):
        starts.append(len(tok_row))
        tok_row += [r] * n
        tok_pos += list(range(c, c + n))
    return i32(tok_row), i32(tok_pos), i32(slots), i32(starts), i32(q_lens), i32(ctx_lens)


def new_status():
    return torch.zeros(1, dtype=torch.int32, device=DEV)


# ---------------------------------------------------------------- mechanisms alone
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,H,groups", [(1, 64, 1), (5, 96, 3), (3, 70, 5), (37, 1032, 2), (4, 72, 9), (3, 4096, 4), (2, 1280, 40), (2, 36, 36)])
def test_completing_a_sublayer_and_a_layer(dtype, T, H, groups):
    """x + norm(y); the result kept; the learned average over the kept ones; then a copy, or another norm on rows asked
    for in another order."""
    torch.manual_seed(T + H + groups)
    dt = TD[dtype]
    w, wf = 1 + 0.2 * torch.randn(H), 1 + 0.2 * torch.randn(H)
    y, resid = (torch.randn(T, H) * torch.rand(H) * 3).to(dt), torch.randn(T, H)
    hist = torch.randn(4, T, H)
    a = torch.randn(3)
    total = resid.double() + P.grouped_rms_norm(y.double(), w.double(), 1e-5, groups)
    avg = P.depth_average([hist[0].double(), hist[1].double(), total], a.double())
    r, out = resid.to(DEV), torch.full((T, H), float("nan"), dtype=dt, device=DEV)
    K.post_norm(y.to(DEV), w.to(DEV), groups, 1e-5, r, out)
    assert rel_err(r, total) < 1e-6 and rel_err(out, total) < KTOL[dtype]
    r, h = resid.to(DEV), hist.to(DEV)
    K.post_norm(y.to(DEV), w.to(DEV), groups, 1e-5, r, out, history=h, n_history=2, put_history=2, depth_weights=a.to(DEV))
    assert rel_err(r, avg) < 2e-6 and rel_err(out, avg) < KTOL[dtype] and rel_err(h[2], total) < 1e-6
    assert torch.equal(h[[0, 1, 3]].cpu(), hist[[0, 1, 3]])
    # the final norm: wanted rows only, nothing written back
    rows = list(range(T - 1, -1, -2))
    r, h = resid.to(DEV), hist.to(DEV)
    out2 = torch.full((len(rows), H), float("nan"), dtype=dt, device=DEV)
    for og in {groups, 1}:
        K.post_norm(y.to(DEV), w.to(DEV), groups, 1e-5, r, out2, rows=i32(rows), write_resid=False, history=h, n_history=2,
                    depth_weights=a.to(DEV), out_weight=wf.to(DEV), out_groups=og, out_eps=1e-6)
        assert rel_err(out2, P.grouped_rms_norm(avg, wf.double(), 1e-6, og)[rows]) < KTOL[dtype]
    assert torch.equal(r.cpu(), resid) and torch.equal(h.cpu(), hist)
    # nothing pending: the stream itself is kept and copied
    K.post_norm(None, None, 1, 0.0, r, out, history=h, put_history=0)
    assert torch.equal(h[0], r) and torch.equal(out, r.to(dt))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,H,top", [(5, 96, 3), (3, 50, 1), (9, 1024, 8)])
def test_completing_a_routed_sublayer_sums_the_experts_rows(dtype, T, H, top):
    torch.manual_seed(T + H)
    dt = TD[dtype]
    n = T * top + 7
    y, wts = torch.randn(n, H).to(dt), torch.rand(T, top)
    pos = torch.randperm(n)[:T * top]
    pos[1] = -1                                              # a choice that has no row
    w, resid = 1 + 0.2 * torch.randn(H), torch.randn(T, H)
    rows = y.double()[pos.clamp(min=0)] * (pos >= 0)[:, None]
    total = (rows.view(T, top, H) * wts.double()[:, :, None]).sum(1)
    want = resid.double() + P.grouped_rms_norm(total, w.double(), 1e-5, 2)
    r = resid.to(DEV)
    K.post_norm(PendingExperts(y.to(DEV), wts.to(DEV), pos.to(torch.int32).to(DEV)), w.to(DEV), 2, 1e-5, r, None)
    assert rel_err(r, want) < 1e-5


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,taps,cuts", [(64, 4, [5, 1, 1, 6, 2]), (70, 3, [2, 2, 9, 1]), (96, 1, [7, 1, 3]), (36, 6, [1, 1, 1, 10, 3, 40]),
                                         (1028, 2, [30, 1, 2, 70])])
def test_input_convolution_in_portions_and_single_tokens(dtype, H, taps, cuts):
    """Two sequences of unequal length fed in portions: longer ones through the prompt kernel, steps of single tokens
    inside the completing kernel; the state holds the last inputs."""
    torch.manual_seed(H + taps)
    dt = TD[dtype]
    S = sum(cuts)
    lens, slots = [S, S - 3], [2, 0]
    x = [torch.randn(n, H) for n in lens]
    w = torch.randn(H, taps) * 0.5
    wt = w.t().contiguous().to(DEV)
    state = torch.zeros(4, taps - 1, H, device=DEV) if taps > 1 else None
    got = [torch.zeros(n, H) for n in lens]
    done = [0, 0]
    for cut in cuts:
        rows = [r for r in range(2) if done[r] < lens[r]]
        q_lens = [min(cut, lens[r] - done[r]) for r in rows]
        resid = torch.cat([x[r][done[r]:done[r] + n] for r, n in zip(rows, q_lens)]).to(DEV).contiguous()
        tok_row, _, row_slot, q_start, q_len, _ = step_arrays([done[r] for r in rows], q_lens, [slots[r] for r in rows])
        out = torch.full(resid.shape, float("nan"), dtype=dt, device=DEV)
        if max(q_lens) == 1:
            K.post_norm(None, None, 1, 0.0, resid, out, conv_weight=wt, conv_state=state, tok_row=tok_row, row_slot=row_slot)
        else:
            K.stream_conv(resid, wt, state, out, tok_row, row_slot, q_start)
            if state is not None:
                K.conv_state_update(resid, state, row_slot, q_start, q_len, len(rows))
        at = 0
        for r, n in zip(rows, q_lens):
            got[r][done[r]:done[r] + n] = out[at:at + n].float().cpu()
            at += n
            done[r] += n
    assert done == lens
    for r in range(2):
        want = x[r].double() + P.causal_conv(x[r].double(), w.double())
        assert rel_err(got[r], want) < (1e-6 if dtype == "float32" else KTOL[dtype])
        if taps > 1 and lens[r] >= taps - 1:
            assert torch.equal(state[slots[r]].cpu(), x[r][lens[r] - (taps - 1):])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("q_rank,rank,rot,bs", [(40, 48, 8, 4), (20, 36, 6, 16), (8, 8, 2, 8), (128, 512, 64, 64), (0, 24, 10, 4)])
def test_query_latent_latent_and_rotated_part(dtype, q_rank, rank, rot, bs):
    """The query latent normed over its true size, the cached row [normed latent | rotated part] at page borders, both once
    more as plain rows; padding places hold zeros."""
    torch.manual_seed(q_rank + rank)
    dt = TD[dtype]
    up8 = lambda n: -(-n // 8) * 8
    qp, rp, tp = up8(q_rank), up8(rank), up8(rot)
    S, ctx = 3 * bs - 1, 5
    proj = torch.zeros(S, qp + rp + tp + 24)
    proj[:, :q_rank], proj[:, qp:qp + rank] = torch.randn(S, q_rank) * 3, torch.randn(S, rank)
    proj[:, qp + rp:qp + rp + rot], proj[:, qp + rp + tp:] = torch.randn(S, rot), 99.0
    proj = proj.to(dt)
    qw, cw = torch.zeros(max(qp, 1)), torch.zeros(rp)
    qw[:q_rank], cw[:rank] = 1 + 0.3 * torch.randn(q_rank), 1 + 0.3 * torch.randn(rank)
    sc = {"factor": 4.0, "original": 32, "fast": 8.0, "slow": 1.0}
    pos = RotaryScaled(rot, 100.0, sc)
    pos.prepare(256, _Rt)
    n_cols = -(-(S + ctx) // bs)
    perm = torch.randperm(n_cols + 2)[:n_cols]
    table = torch.full((3, n_cols), -1, dtype=torch.int32, device=DEV)
    table[2] = perm.to(torch.int32).to(DEV)
    pool = torch.full((n_cols + 2, 1, bs, rp + tp), 7.0, dtype=dt, device=DEV)
    q_out = torch.full((S, qp), 7.0, dtype=dt, device=DEV) if q_rank else None
    c_rows = torch.full((S, rp), 7.0, dtype=dt, device=DEV)
    r_rows = torch.full((S, tp + 16), 7.0, dtype=dt, device=DEV)
    tok_row, tok_pos, row_slot, _, _, _ = step_arrays([ctx], [S], [2])
    status = new_status()
    K.norm_append(proj.to(DEV), q_out, qw.to(DEV) if q_rank else None, cw.to(DEV), 1e-5, tok_row, tok_pos, row_slot, pool, None,
                  table, 1, True, status, k_rows=c_rows, q_count=q_rank, k_count=rank, cos=pos.cos, sin=pos.sin, rot=rot,
                  rot_places=tp, r_rows=r_rows)
    assert int(status.item()) == 0
    x = proj.double()
    c = P.rms_norm(x[:, qp:qp + rank], cw[:rank].double(), 1e-5)
    f, mag = P.rot_frequencies(rot, 100.0, sc)
    turned = P.rotate_pairs(x[:, None, qp + rp:qp + rp + rot], torch.arange(ctx, ctx + S), f, mag)[:, 0]
    if q_rank:
        assert rel_err(q_out[:, :q_rank], P.rms_norm(x[:, :q_rank], qw[:q_rank].double(), 1e-5)) < KTOL[dtype]
        assert float(q_out[:, q_rank:].float().abs().sum()) == 0.0
    rows = torch.stack([pool[perm[p // bs], 0, p % bs] for p in range(ctx, ctx + S)]).float().cpu()
    assert rel_err(rows[:, :rank], c) < KTOL[dtype] and rel_err(rows[:, rp:rp + rot], turned) < KTOL[dtype]
    assert float(rows[:, rank:rp].abs().sum()) == 0.0 and float(rows[:, rp + rot:].abs().sum()) == 0.0
    assert torch.equal(c_rows.float().cpu(), rows[:, :rp]) and torch.equal(r_rows[:, :tp].float().cpu(), rows[:, rp:])
    assert float(r_rows[:, tp:].float().abs().sum()) == 0.0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,heads,d,rot,r", [(1, 3, 24, 8, 40), (8, 16, 128, 64, 512), (13, 2, 64, 16, 72), (40, 5, 20, 6, 36), (200, 4, 32, 32, 64)])
def test_queries_into_the_latents_basis_and_back_behind_the_gate(dtype, T, heads, d, rot, r):
    torch.manual_seed(T + heads)
    dt = TD[dtype]
    tp = -(-rot // 8) * 8
    q, w = torch.randn(T, heads, d + rot).to(dt), (torch.randn(heads, r, d) / d ** 0.5).to(dt)
    out = torch.full((T, heads * (r + tp)), 7.0, dtype=dt, device=DEV)
    qd = q.reshape(T, -1).to(DEV)
    pos = RotaryScaled(rot, 1000.0, None)
    pos.prepare(512, _Rt)
    tok_pos = torch.randint(0, 400, (T,))
    status = new_status()
    K.head_gemm(qd, w.to(DEV), out, a_size=d + rot, out_size=r + tp,
                rope=(d, r, rot, tp, pos.cos, pos.sin, tok_pos.to(torch.int32).to(DEV), status))
    got = out.view(T, heads, r + tp).double().cpu()
    f, _ = P.rot_frequencies(rot, 1000.0)
    turned = P.rotate_pairs(q[:, :, d:].double(), tok_pos, f, 1.0)
    assert rel_err(got[:, :, :r], torch.einsum("thk,hnk->thn", q[:, :, :d].double(), w.double())) < KTOL[dtype]
    assert rel_err(got[:, :, r:r + rot], turned) < KTOL[dtype] and float(got[:, :, r + rot:].abs().sum()) == 0.0
    K.rope_heads(qd, d + rot, d, qd, d + rot, d, pos.cos, pos.sin, tok_pos.to(torch.int32).to(DEV), heads, rot, rot, status)
    inplace = qd.view(T, heads, d + rot).cpu()
    assert rel_err(inplace[:, :, d:], turned) < KTOL[dtype] and torch.equal(inplace[:, :, :d], q[:, :, :d])
    if T < K.HEAD_GEMM_LIBRARY_ROWS or dtype == "float32":
        v = (torch.randn(heads, 20, r) / r ** 0.5).to(dt)
        a, packed = torch.randn(T, heads, r).to(dt), torch.randn(T, 3 + heads * 20).to(dt)
        o = torch.zeros(T, heads * 20, dtype=dt, device=DEV)
        K.head_gemm(a.reshape(T, -1).to(DEV), v.to(DEV), o, gate=packed.to(DEV), gate_col=3)
        want = torch.einsum("thk,hnk->thn", a.double(), v.double()).reshape(T, -1) * torch.sigmoid(packed[:, 3:].double())
        assert rel_err(o, want) < KTOL[dtype]
    assert int(status.item()) == 0


def _standing_out(S, heads, d, seed):
    """Queries and keys in which every seventh position and one far back stand out, so that a key too many or too few, or
    a keyless term left out, changes the result by the size of a value; the second half's scores are small: there the
    keyless term is a good part of the denominator."""
    torch.manual_seed(seed)
    q, k = torch.randn(S, heads, d) * 0.3, torch.randn(S, 1, d) * 0.3
    e = torch.zeros(d)
    e[3 % d] = 1.0
    for p in {p for p in range(S) if p % 7 == 0 or p == 2}:
        k[p] += 6.0 * e
    q += 2.0 * e
    q[S // 2:] *= 0.05
    sink = torch.linspace(-1.0, 4.0, heads)
    return q, k, sink



def _plain_rows(q, k, v, scale, sink, window):
    """The plain attention with a window, position by position."""
    S, H, _ = q.shape
    out = torch.zeros(S, H, v.shape[-1], dtype=torch.float64)
    for i in range(S):
        lo = 0 if window is None else max(0, i - window + 1)
        s = torch.einsum("hd,jhd->hj", q[i], k[lo:i + 1].expand(-1, H, -1)) * scale
        m = torch.maximum(s.amax(-1), sink)
        e = torch.exp(s - m[:, None])
        out[i] = torch.einsum("hj,jhd->hd", e, v[lo:i + 1].expand(-1, H, -1)) / (e.sum(-1) + torch.exp(sink - m))[:, None]
    return out


LATENT_CASES = [  # heads, latent, rotated part (places), block size, length, window
    (6, 48, 8, 4, 150, None), (1, 8, 8, 16, 70, None), (16, 512, 64, 64, 330, None), (20, 40, 8, 8, 200, None), (3, 192, 0, 16, 200, 50),
    (33, 128, 16, 64, 140, None), (2, 72, 16, 8, 300, 33), (100, 24, 8, 16, 90, None), (32, 256, 32, 64, 200, None)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("how", ["whole", "portions", "splits"])
@pytest.mark.parametrize("case", LATENT_CASES)
def test_attention_over_cached_latents(dtype, case, how):
    """Every head's keys are the cached rows, its values their leading columns: whole prompts, portions and single tokens
    over pages in random order, single tokens with their keys cut into splits."""
    heads, r, tp, bs, S, window = case
    dt = TD[dtype]
    d = r + tp
    q, k, sink = _standing_out(S, heads, d, seed=heads + r)
    q, k = q.to(dt), k.to(dt)
    scale = 0.7
    want = _plain_rows(q.double(), k.double(), k[:, :, :r].double(), scale, sink.double(), window).reshape(S, heads * r)
    n_cols = -(-S // bs)
    perm = torch.randperm(n_cols + 3)[:n_cols]
    pool = torch.full((n_cols + 3, 1, bs, d), float("nan"), dtype=dt, device=DEV)         # what no key lies in is never used
    pool[perm[-1]] = 0.0
    table = torch.full((2, n_cols), -1, dtype=torch.int32, device=DEV)
    table[1] = perm.to(torch.int32).to(DEV)
    for p in range(S):
        pool[perm[p // bs], 0, p % bs] = k[p, 0].to(DEV)
    status = new_status()
    got = torch.zeros(S, heads * r)
    portions = [S] if how == "whole" else [5, 2, 1, 1, 17, 3] + [1] * 20 + [64] + [1] * 400
    at = 0
    for n in portions:
        n = min(n, S - at)
        if n <= 0:
            break
        tok_row, _, row_slot, q_start, q_len, ctx_len = step_arrays([at], [n], [1])
        n_splits, split_len, scratch = 1, 0, None
        if how == "splits" and n == 1 and at + 1 > 64:
            split_len = 64
            n_splits = -(-(at + 1) // split_len) + 2                    # the last two hold no key
            scratch = torch.full((K.attention_scratch_floats(1, heads, r, n_splits),), float("nan"), device=DEV)
        out = torch.full((n, heads * r), float("nan"), dtype=dt, device=DEV)
        K.attention_ext(q[at:at + n].reshape(n, heads * d).to(DEV).contiguous(), pool, pool, out, table, tok_row, row_slot,
                        q_start, q_len, ctx_len, 1, n, heads, 1, d, scale, window or 0, n_splits, split_len, scratch, status,
                        sink=sink.to(DEV), value_dim=r)
        got[at:at + n] = out.float().cpu()
        at += n
    assert at == S and int(status.item()) == 0
    err = (got.double() - want).abs().max(dim=1).values / want.abs().max()
    assert float(err.max()) < KTOL[dtype], f"first wrong position {int((~(err < KTOL[dtype])).nonzero()[0])}"


DENSE_CASES = [  # heads, own key dims, shared, value dims, lengths, window
    (2, 128, 64, 128, [700, 61, 1, 130], None), (3, 64, 64, 64, [300, 129], None), (4, 128, 0, 128, [257, 64], 100), (2, 64, 0, 64, [190], None),
    (1, 128, 64, 64, [65, 400, 2], None), (5, 64, 64, 128, [140, 33], 40), (2, 128, 0, 64, [128, 385], None), (2, 64, 128, 128, [150], None)]


@pytest.mark.parametrize("form", [0, 1, 2])
@pytest.mark.parametrize("gated", [False, True])
@pytest.mark.parametrize("case", DENSE_CASES)
def test_prompt_attention_over_plain_rows(case, gated, form):
    """Unequal prompts of one step on the tcgen05 kernel, keys and values as the product leaves them and a key part shared
    by the heads: both forms of the kernel, a far key, windows, the keyless term, the gate in the epilogue."""
    heads, dn, dr, dv, lens, window = case
    T = sum(lens)
    sink = torch.linspace(-1.0, 4.0, heads)
    kv, rot, q = torch.zeros(T, heads, dn + dv), torch.zeros(T, max(dr, 1)), torch.zeros(T, heads, dn + dr)
    at = 0
    for i, n in enumerate(lens):
        qq, kk, _ = _standing_out(n, heads, dn + dr, seed=50 + i)
        q[at:at + n] = qq
        kv[at:at + n, :, :dn] = kk[:, :, :dn] + 0.2 * torch.randn(n, heads, dn)
        if dr:
            rot[at:at + n] = kk[:, 0, dn:]
        kv[at:at + n, :, dn:] = torch.randn(n, heads, dv)
        at += n
    q, kv, rot = q.bfloat16(), kv.bfloat16(), rot.bfloat16()
    gate = torch.randn(T, 8 + heads * dv).bfloat16()
    wants, at = [], 0
    for n in lens:
        k = kv[at:at + n, :, :dn].double()
        if dr:
            k = torch.cat([k, rot[at:at + n, None].double().expand(n, heads, dr)], dim=-1)
        wants.append(_plain_rows(q[at:at + n].double(), k, kv[at:at + n, :, dn:].double(), 0.4, sink.double(), window).reshape(n, -1))
        at += n
    want = torch.cat(wants)
    if gated:
        want = want * torch.sigmoid(gate[:, 8:].double())
    out = torch.full((T, heads * dv), float("nan"), dtype=torch.bfloat16, device=DEV)
    _, _, row_slot, q_start, q_len, ctx_len = step_arrays([0] * len(lens), lens, list(range(len(lens))))
    status = new_status()
    K.attn_prefill_set_form(form)
    try:
        K.attention_dense(q.reshape(T, -1).to(DEV), kv.reshape(T, -1).to(DEV), rot.to(DEV) if dr else None, out, row_slot, q_start,
                          q_len, ctx_len, len(lens), max(lens), heads, dn, dv, 0.4, window or 0, sink.to(DEV),
                          gate.to(DEV) if gated else None, 8 if gated else 0, status)
        torch.cuda.synchronize()
    finally:
        K.attn_prefill_set_form(0)
    assert int(status.item()) == 0
    err = (out.double().cpu() - want).abs().amax(1) / want.abs().max()
    assert float(err.max()) < KTOL["bfloat16"], f"first wrong row {int((~(err < KTOL['bfloat16'])).nonzero()[0])} of {lens}"


def test_prompt_attention_over_plain_rows_reports_a_wait_that_runs_out():
    heads, dn, dr, dv, n = 2, 128, 64, 128, 200
    q, kv, rot = (torch.randn(n, c, device=DEV).bfloat16() for c in (heads * (dn + dr), heads * (dn + dv), dr))
    out = torch.zeros(n, heads * dv, dtype=torch.bfloat16, device=DEV)
    _, _, row_slot, q_start, q_len, ctx_len = step_arrays([0], [n], [0])
    args = (q, kv, rot, out, row_slot, q_start, q_len, ctx_len, 1, n, heads, dn, dv, 0.1)
    status = new_status()
    K.attention_dense(*args, status=status)
    want = out.clone()
    for form in (1, 2):
        K.attn_prefill_set_form(form)
        K.tc_test_hook(1_000_000, True)
        try:
            K.attention_dense(*args, status=status)
            torch.cuda.synchronize()
            assert int(status.item()) & K.STATUS_WAIT_TIMEOUT
        finally:
            K.tc_test_hook()
            K.attn_prefill_set_form(0)
        status.zero_()
        out.zero_()
        K.attention_dense(*args, status=status)
        assert int(status.item()) == 0 and rel_err(out, want) < 1e-2


SCAN_CASES = [(2, 16, 8), (3, 24, 40), (1, 64, 64), (2, 136, 24), (1, 12, 6), (4, 128, 128), (1, 256, 72)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("segments", [False, True])
@pytest.mark.parametrize("H,d,dv", SCAN_CASES)
def test_lightning_recurrence_in_portions_and_segments(dtype, H, d, dv, segments):
    """S_t = g S_(t-1) + silu(k_t) silu(v_t)^T, o_t = S_t^T silu(q_t) from portions of many sizes - long ones as segments
    side by side - against the plain token-by-token recurrence; decays from none at all to one."""
    torch.manual_seed(H * d + dv)
    dt = TD[dtype]
    lens, cuts = ([459, 262], [192, 129, 1, 63, 65, 3, 128]) if segments else ([90, 41], [17, 1, 1, 2, 30, 3, 1, 16, 64])
    nk, nv = H * d, H * dv
    decay = torch.tensor([1.0, 0.999, 0.5, 0.0][:H])
    xs = [torch.randn(n, 2 + 2 * nk + nv + 3).to(dt) for n in lens]
    slots = [3, 1]
    state = torch.zeros(5, H, d, dv, device=DEV)
    state[4] = 7.0
    status = new_status()
    got, done = [torch.zeros(n, nv) for n in lens], [0, 0]
    for cut in cuts:
        rows = [r for r in range(2) if done[r] < lens[r]]
        if not rows:
            break
        q_lens = [min(cut, lens[r] - done[r]) for r in rows]
        proj = torch.cat([xs[r][done[r]:done[r] + n] for r, n in zip(rows, q_lens)]).to(DEV).contiguous()
        _, _, row_slot, q_start, q_len, ctx_len = step_arrays([done[r] for r in rows], q_lens, [slots[r] for r in rows])
        out = torch.full((proj.shape[0], nv), float("nan"), device=DEV)
        kw = {}
        if segments:
            n_scr = K.linear_scan_scratch_floats(proj.shape[0], len(rows), H, d, dv)
            kw = dict(max_q_len=max(q_lens), scratch=torch.full((n_scr,), float("nan"), device=DEV))
        K.linear_scan(proj, 2, 2 + nk, 2 + 2 * nk, state, out, K.SCAN_DECAY, row_slot, q_start, q_len, ctx_len, len(rows), H, d, dv,
                      True, status, decay=decay.to(DEV), silu=True, **kw)
        at = 0
        for r, n in zip(rows, q_lens):
            got[r][done[r]:done[r] + n] = out[at:at + n].cpu()
            at += n
            done[r] += n
    assert done == lens and int(status.item()) == 0 and bool((state[4] == 7.0).all())
    for r, n in enumerate(lens):
        x = P.silu(xs[r].double())
        want, final = P.decay_recurrence(x[:, 2:2 + nk].reshape(n, H, d), x[:, 2 + nk:2 + 2 * nk].reshape(n, H, d),
                                         x[:, 2 + 2 * nk:2 + 2 * nk + nv].reshape(n, H, dv), decay.double())
        assert rel_err(got[r], want.reshape(n, nv)) < 2e-5           # the recurrence is float32 in both dtypes
        assert rel_err(state[slots[r]].cpu(), final) < 2e-5


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,n", [(1, 128), (7, 50), (3, 2048)])
def test_one_norm_over_the_heads_side_by_side_and_the_gate(dtype, T, n):
    torch.manual_seed(n)
    o, w, packed = torch.randn(T, n) * 5, 1 + 0.2 * torch.randn(n), torch.randn(T, n + 9).to(TD[dtype])
    out = torch.zeros(T, n, dtype=TD[dtype], device=DEV)
    K.row_norm_gate(o.to(DEV), w.to(DEV), packed.to(DEV), 9, out, 1e-5)
    want = P.rms_norm(o.double(), w.double(), 1e-5) * torch.sigmoid(packed[:, 9:].double())
    assert rel_err(out, want) < (2e-6 if dtype == "float32" else KTOL[dtype])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("E,top", [(8, 3), (5, 5), (1, 1), (40, 6)])
@pytest.mark.parametrize("T", [3, 70])
def test_weights_are_the_softmax_scores_themselves(dtype, E, top, T):
    torch.manual_seed(E * 10 + top)
    H = 96
    x, router = torch.randn(T, H).to(TD[dtype]), (torch.randn(E, H) / H ** 0.5 * 3).to(TD[dtype])
    want_ids, want_w = P.route(x.double(), router.double(), top)
    for given in (False, True):
        ids, wts = torch.zeros(T, top, dtype=torch.int32, device=DEV), torch.zeros(T, top, device=DEV)
        logits = (x.float() @ router.float().T).to(DEV) if given else None
        K.moe_route(x.to(DEV), router.to(DEV), None, ids, wts, logits, weight_scale=1.0)
        order, want_order = ids.long().cpu().sort(dim=1), want_ids.sort(dim=1)
        assert torch.equal(order.values, want_order.values)
        assert rel_err(wts.cpu().gather(1, order.indices), want_w.gather(1, want_order.indices)) < 1e-5


# ---------------------------------------------------------------- whole models
@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    tmp = tmp_path_factory.mktemp("gulozen")
    out = {(n, "float32"): write_folder(tmp, n, seed=31) for n in NAMES}
    # bfloat16: choices that are decided by far more than rounding
    out.update({(n, "bfloat16"): write_folder(tmp, n, seed=31, decisive=True) for n in NAMES})
    return out


@pytest.fixture(scope="module")
def engines(folders):
    return {(n, d): fd.load(folders[(n, d)], device="cuda", dtype=d) for n in NAMES for d in DTYPES}


def _vocab(name):
    return GULOZEN[name]["vocab"]


LENGTHS = [1, 2, 3, 5, 8, 9, 16, 17, 63, 64, 65, 129, 200]       # around the taps, the pages and the kernels' tiles


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
@pytest.mark.parametrize("block_size", [8, 64])
def test_whole_prompts(engines, folders, name, dtype, block_size):
    eng = engines[(name, dtype)]
    cache = eng.model.new_cache(max_tokens=320, block_size=block_size)
    for p in prompts_for(_vocab(name), LENGTHS, seed=1):
        slot = cache.admit()
        got = eng.model.step(cache, [slot], [p], "all")
        assert truth(folders[(name, dtype)], p).excess(got, range(len(p)), dtype) < 1, f"prompt of {len(p)} tokens"
        cache.release(slot)
    eng.model.check_status()
    cache.check_invariants()


def test_every_layer_in_float32(engines, folders):
    """The residual stream after every layer, its depth average included, against the plain one."""
    for name in NAMES:
        eng, folder = engines[(name, "float32")], folders[(name, "float32")]
        (p,) = prompts_for(_vocab(name), [45], seed=2)
        _, layers = P.forward(raw_config(folder), weights_of(folder), p, return_layers=True)
        cache = eng.model.new_cache(max_tokens=64)
        slot = cache.admit()
        eng.model.trace = {}
        eng.model.step(cache, [slot], [p], None)
        got, eng.model.trace = eng.model.trace, None
        assert len(layers) == len(eng.model.schedule)
        for i, want in enumerate(layers):
            assert rel_err(got[f"layer.{i}"], want) < 1e-5, f"{name}: layer {i}"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_prefill_then_token_by_token(engines, folders, name, dtype):
    """A prompt of one token, of two or of thirty, then single tokens across page borders."""
    eng = engines[(name, dtype)]
    cache = eng.model.new_cache(max_tokens=256, block_size=16)
    for head in (1, 2, 30):
        (p,) = prompts_for(_vocab(name), [head + 50], seed=3 + head)
        want = truth(folders[(name, dtype)], p)
        slot = cache.admit()
        got = eng.model.step(cache, [slot], [p[:head]], "last")
        assert want.excess(got, [head - 1], dtype) < 1
        for i in range(head, len(p)):
            got = eng.model.step(cache, [slot], [[p[i]]], "last")
            assert want.excess(got, [i], dtype) < 1, f"position {i} of a request decoded from {head}"
        cache.release(slot)
    eng.model.check_status()
    cache.check_invariants()


def test_long_decoding_in_float32(engines, folders):
    """Four hundred single tokens after a short prompt: states and pages keep what the plain model sees at once."""
    name = "A"
    eng = engines[(name, "float32")]
    (p,) = prompts_for(_vocab(name), [420], seed=9)
    want = truth(folders[(name, "float32")], p)
    cache = eng.model.new_cache(max_tokens=512, block_size=8)
    slot = cache.admit()
    eng.model.step(cache, [slot], [p[:20]], None)
    for i in range(20, len(p)):
        got = eng.model.step(cache, [slot], [[p[i]]], "last")
        if i % 50 == 0 or i > 410:
            assert want.excess(got, [i], "float32") < 1, f"position {i}"
    cache.release(slot)
    eng.model.check_status()
    cache.check_invariants()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_portions_of_several_sizes(engines, folders, name, dtype):
    """A prompt cut into portions of 2, 3, 1, 7, 33, ... tokens gives the logits of the whole prompt."""
    eng = engines[(name, dtype)]
    (p,) = prompts_for(_vocab(name), [150], seed=5)
    want = truth(folders[(name, dtype)], p)
    cache = eng.model.new_cache(max_tokens=256, block_size=8)
    slot = cache.admit()
    whole = eng.model.step(cache, [slot], [p], "all").clone()
    cache.release(slot)
    for sizes in ([2] * 75, [3, 1, 7, 33, 2, 64, 5, 1, 1, 30, 3], [149, 1], [1, 149]):
        slot = cache.admit()
        at, rows = 0, []
        for n in sizes:
            rows.append(eng.model.step(cache, [slot], [p[at:at + n]], "all").clone())
            at += n
        assert at == len(p)
        got = torch.cat(rows)
        cache.release(slot)
        assert want.excess(got, range(len(p)), dtype) < 1
        apart = (got.double().cpu() - whole.double().cpu()).abs().amax(-1) / want.scale
        bound = want.allowed(dtype) if dtype == "bfloat16" else want.allowed(dtype) * 0.1
        assert bool((apart < bound).all()), f"portions {sizes[:4]}..."
    eng.model.check_status()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_unequal_batch_equals_each_request_alone_and_slots_are_used_again(engines, folders, name, dtype):
    eng, folder = engines[(name, dtype)], folders[(name, dtype)]
    cache = eng.model.new_cache(max_tokens=64 * 8, block_size=8, max_slots=4)
    for batch_no, lengths in enumerate([[9, 80, 1, 44], [130, 3, 26], [5, 5, 62, 25]]):
        reqs = prompts_for(_vocab(name), lengths, seed=30 + batch_no)
        decode = [min(k, len(p) - 1) for k, p in zip([6, 40, 0, 9], reqs)]
        heads = [len(p) - k for p, k in zip(reqs, decode)]
        slots = [cache.admit() for _ in reqs]                 # the second and third batch get used slots, states and pages
        got = eng.model.step(cache, slots, [p[:h] for p, h in zip(reqs, heads)], "last")
        for i, (p, h) in enumerate(zip(reqs, heads)):
            assert truth(folder, p).excess(got[i], [h - 1], dtype) < 1
        live = [i for i in range(len(reqs)) if heads[i] < len(reqs[i])]
        for i in set(range(len(reqs))) - set(live):
            cache.release(slots[i])
        step = 0
        while live:
            got = eng.model.step(cache, [slots[i] for i in live], [[reqs[i][heads[i] + step]] for i in live], "last")
            for j, i in enumerate(live):
                want = truth(folder, reqs[i])
                assert want.excess(got[j], [heads[i] + step], dtype) < 1, f"batch {batch_no}, request {i}, decoded token {step}"
            step += 1
            for i in [i for i in live if heads[i] + step >= len(reqs[i])]:
                cache.release(slots[i])
                live.remove(i)
        cache.check_invariants()
        assert cache.blocks_in_use() == [0] * len(cache.groups)
    eng.model.check_status()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "C"])
def test_mixed_steps_of_prompts_portions_and_single_tokens(engines, folders, name, dtype):
    """One request decodes while another brings its prompt and a third the next part of its own."""
    eng, folder = engines[(name, dtype)], folders[(name, dtype)]
    a, b, c = prompts_for(_vocab(name), [40, 50, 70], seed=70)
    cache = eng.model.new_cache(max_tokens=512, block_size=8, max_slots=4)
    sa, sc = cache.admit(), cache.admit()
    eng.model.step(cache, [sa, sc], [a[:30], c[:20]], None)
    sb = cache.admit()
    got = eng.model.step(cache, [sa, sb, sc], [a[30:31], b[:33], c[20:57]], "last")
    for row, p, n in zip(got, (a, b, c), (31, 33, 57)):
        assert truth(folder, p).excess(row, [n - 1], dtype) < 1
    got = eng.model.step(cache, [sa, sb, sc], [a[31:32], b[33:35], c[57:58]], "last")
    for row, p, n in zip(got, (a, b, c), (32, 35, 58)):
        assert truth(folder, p).excess(row, [n - 1], dtype) < 1
    got = eng.model.step(cache, [sc, sa], [c[58:59], a[32:33]], "last")
    assert truth(folder, c).excess(got[0], [58], dtype) < 1 and truth(folder, a).excess(got[1], [32], dtype) < 1
    eng.model.check_status()


@pytest.mark.parametrize("dtype", DTYPES)
def test_two_dozen_requests_decoded_together(engines, folders, dtype):
    """More rows than the register-fed products take."""
    name = "A"
    eng, folder = engines[(name, dtype)], folders[(name, dtype)]
    reqs = prompts_for(_vocab(name), [3 + (7 * i) % 45 for i in range(24)], seed=60)
    heads = [max(1, len(p) - 4) for p in reqs]
    cache = eng.model.new_cache(max_tokens=64 * 24, block_size=16, max_slots=24)
    slots = [cache.admit() for _ in reqs]
    got = eng.model.step(cache, slots, [p[:h] for p, h in zip(reqs, heads)], "last")
    for i, (p, h) in enumerate(zip(reqs, heads)):
        assert truth(folder, p).excess(got[i], [h - 1], dtype) < 1, f"request {i}"
    for step in range(3):
        live = [i for i in range(24) if heads[i] + step < len(reqs[i])]
        got = eng.model.step(cache, [slots[i] for i in live], [[reqs[i][heads[i] + step]] for i in live], "last")
        for j, i in enumerate(live):
            assert truth(folder, reqs[i]).excess(got[j], [heads[i] + step], dtype) < 1, f"request {i}, decoded token {step}"
    eng.model.check_status()
    cache.check_invariants()


def test_batch_neighbours_change_no_bit_in_float32(engines):
    for name in NAMES:
        eng = engines[(name, "float32")]
        reqs = prompts_for(_vocab(name), [70, 3, 131], seed=40)
        cache = eng.model.new_cache(max_tokens=512, block_size=8, max_slots=4)
        alone = []
        for p in reqs:
            s = cache.admit()
            a = eng.model.step(cache, [s], [p[:-2]], "last").clone()
            b = eng.model.step(cache, [s], [[p[-2]]], "last").clone()
            alone.append((a, b))
            cache.release(s)
        slots = [cache.admit() for _ in reqs]
        a = eng.model.step(cache, slots, [p[:-2] for p in reqs], "last").clone()
        b = eng.model.step(cache, slots, [[p[-2]] for p in reqs], "last").clone()
        for i in range(len(reqs)):
            assert torch.equal(a[i], alone[i][0][0]) and torch.equal(b[i], alone[i][1][0]), f"{name}: request {i}"


def _drawn(tmp_path, seed, dtype, lengths, heads):
    cfg = random_config(seed)
    folder = fd.write_random_model(tmp_path / "m", cfg, seed)
    if dtype == "bfloat16":
        decisive_routers(folder)
    cfg, W = raw_config(folder), weights_of(folder)
    reqs = prompts_for(cfg["vocab"], lengths, seed=seed)
    want = [Truth(cfg, W, r) for r in reqs]
    eng = fd.load(folder, device="cuda", dtype=dtype)
    cache = eng.model.new_cache(max_tokens=256, max_slots=4, slack_blocks=4, block_size=16)
    for r, w in zip(reqs, want):
        s = cache.admit()
        assert w.excess(eng.model.step(cache, [s], [r], "all"), range(len(r)), dtype) < 1, cfg
        cache.release(s)
    slots = [cache.admit() for _ in reqs]
    got = eng.model.step(cache, slots, [r[:h] for r, h in zip(reqs, heads)], "last")
    for i in range(len(reqs)):
        assert want[i].excess(got[i], [heads[i] - 1], dtype) < 1, cfg
    for step in range(7):
        live = [i for i in range(len(reqs)) if heads[i] + step < len(reqs[i])]
        got = eng.model.step(cache, [slots[i] for i in live], [[reqs[i][heads[i] + step]] for i in live], "last")
        for j, i in enumerate(live):
            assert want[i].excess(got[j], [heads[i] + step], dtype) < 1, (cfg, i, step)
    eng.model.check_status()
    cache.check_invariants()


@pytest.mark.parametrize("seed", range(100, 130))
def test_configurations_drawn_at_random_in_float32(tmp_path, seed):
    """Sizes and layer orders nobody chose: whole prompts, then a batch of unequal prompts decoded together."""
    _drawn(tmp_path, seed, "float32", [2, 37, 131], [1, 30, 124])


@pytest.mark.parametrize("seed", range(200, 212))
def test_configurations_drawn_at_random_in_bfloat16(tmp_path, seed):
    _drawn(tmp_path, seed, "bfloat16", [20, 150], [13, 143])


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_prompts_at_sizes_of_the_tensor_core_kernels(tmp_path, dtype):
    """Heads of 128 + 64 over a latent of 128 + 64, heads of 64 + 64, experts wide enough for the grouped tcgen05 products,
    prompts of several hundred tokens: many segments of the recurrence, many key tiles; each prompt alone, then the two
    together and decoded on."""
    cfg = GH.model(333, 256, 1e-5, [
        GH.latent(2, 128, 64, 128, 96, 128, 0.06, 40000.0, (4.0, 256, 32.0, 1.0), GH.moe(8, 2, 128)),
        GH.lightning(2, 64, 64, [0.9, 0.995]),
        GH.latent(18, 64, 64, 64, 64, 192, 0.09, 10000.0, None, GH.moe(4, 3, 128)),
        GH.lightning(1, 128, 128, [0.98], GH.moe(6, 2, 256))], groups=4, taps=4, emb_scale=20.0)
    folder = fd.write_random_model(tmp_path / "m", cfg, 7)
    if dtype == "bfloat16":
        decisive_routers(folder)
    W = weights_of(folder)
    cfg = raw_config(folder)
    reqs = prompts_for(cfg["vocab"], [610, 333], seed=7)
    want = [Truth(cfg, W, r) for r in reqs]
    eng = fd.load(folder, device="cuda", dtype=dtype)
    cache = eng.model.new_cache(max_tokens=1024, max_slots=4, slack_blocks=4, block_size=64)
    for r, w in zip(reqs, want):
        s = cache.admit()
        assert w.excess(eng.model.step(cache, [s], [r], "all"), range(len(r)), dtype) < 1, f"prompt of {len(r)} tokens"
        cache.release(s)
    slots = [cache.admit() for _ in reqs]
    heads = [600, 325]
    got = eng.model.step(cache, slots, [r[:h] for r, h in zip(reqs, heads)], "last")
    for i in range(2):
        assert want[i].excess(got[i], [heads[i] - 1], dtype) < 1
    for step in range(8):
        got = eng.model.step(cache, slots, [[reqs[i][heads[i] + step]] for i in range(2)], "last")
        for i in range(2):
            assert want[i].excess(got[i], [heads[i] + step], dtype) < 1, (i, step)
    eng.model.check_status()
    cache.check_invariants()


@pytest.mark.parametrize("dtype", DTYPES)
def test_first_tokens_see_zeros_not_an_earlier_sequence(engines, folders, dtype):
    """A slot whose convolution and recurrence states an earlier sequence left full starts a new one from zeros."""
    name = "A"
    eng, folder = engines[(name, dtype)], folders[(name, dtype)]
    cache = eng.model.new_cache(max_tokens=128, block_size=8, max_slots=1)
    old, new = prompts_for(_vocab(name), [60, 12], seed=80)
    s = cache.admit()
    eng.model.step(cache, [s], [old], None)
    cache.release(s)
    s = cache.admit()
    want = truth(folder, new)
    for i, t in enumerate(new):
        assert want.excess(eng.model.step(cache, [s], [[t]], "last"), [i], dtype) < 1, f"token {i}"


@pytest.mark.parametrize("name", NAMES)
def test_greedy_generation_through_the_engine(folders, name):
    """``Engine.generate``: the scheduler admits five requests three at a time, decode steps replay captured graphs."""
    folder = folders[(name, "float32")]
    eng = fd.load(folder, device="cuda", dtype="float32")
    prompts = prompts_for(_vocab(name), [3, 30, 1, 70, 9], seed=50)
    got = eng.generate(prompts, 30, max_batch=3)
    for p, r in zip(prompts, got):
        assert r.tokens == plain_greedy(folder, p, 30)
    eng.model.check_status()


@pytest.mark.parametrize("name", ["A", "C"])
def test_greedy_generation_in_bfloat16_picks_a_best_token(folders, name):
    folder = folders[(name, "bfloat16")]
    eng = fd.load(folder, device="cuda", dtype="bfloat16")
    prompts = prompts_for(_vocab(name), [5, 50, 2], seed=51)
    got = eng.generate(prompts, 30)
    for p, r in zip(prompts, got):
        full = p + r.tokens
        ref = oracle_logits(folder, full[:-1])
        scale = float(ref.abs().max())
        for i, tok in enumerate(r.tokens):
            row = ref[len(p) - 1 + i]
            assert float(row.max() - row[tok]) <= 2 * TOL["bfloat16"] * scale, f"token {i}"
    eng.model.check_status()


def test_command_line_generates(folders):
    folder = folders[("B", "float32")]
    p = prompts_for(_vocab("B"), [12], seed=52)[0]
    cmd = [sys.executable, "-m", "flashdecode_cuda_b200", "generate", "--model", str(folder), "--dtype", "float32",
           "--prompt-ids", ",".join(map(str, p)), "--max-new-tokens", "8"]
    r = subprocess.run(cmd, cwd=ROOT, capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert json.loads(r.stdout.strip().splitlines()[-1])["tokens"] == plain_greedy(folder, p, 8)


@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_runner_replays_a_schedule(folders, tmp_path, dtype):
    """Prompts of unequal lengths in one step, then one token each, the shorter request ending earlier; the same
    request again afterwards in the freed slot."""
    name = "A"
    folder = folders[(name, dtype)]
    a, b = prompts_for(_vocab(name), [40, 9], seed=53)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:30], "want": [0, 23, 24, 29]},
                                     {"id": "b", "tokens": b[:7], "want": [6]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": [a[30]], "want": [0]}, {"id": "b", "tokens": [b[7]], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": [a[31]], "want": [0]}, {"id": "b", "tokens": [b[8]], "want": [0]}], "end": ["b"]}]
    steps += [{"step": 3 + i, "entries": [{"id": "a", "tokens": [a[32 + i]], "want": [0]}], "end": ["a"] if i == 7 else []}
              for i in range(8)]
    steps.append({"step": 11, "entries": [{"id": "c", "tokens": b, "want": [8]}], "end": ["c"]})
    out = tmp_path / "out"
    r = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(folder), "--dtype", dtype, "--out", str(out),
                        "--max-tokens", "128"], input="\n".join(json.dumps(s) for s in steps) + "\n", cwd=ROOT,
                       capture_output=True, text=True, timeout=900)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(12)]
    V = _vocab(name)
    wa, wb = truth(folder, a), truth(folder, b)

    def read(i):
        return torch.frombuffer(bytearray((out / f"{i}.f32").read_bytes()), dtype=torch.float32).view(-1, V)
    assert wa.excess(read(0)[:4], [0, 23, 24, 29], dtype) < 1 and wb.excess(read(0)[4:], [6], dtype) < 1
    assert wa.excess(read(1), [30], dtype) < 1
    assert wa.excess(read(2)[:1], [31], dtype) < 1 and wb.excess(read(2)[1:], [8], dtype) < 1
    for i in range(8):
        assert wa.excess(read(3 + i), [32 + i], dtype) < 1
    assert wb.excess(read(11), [8], dtype) < 1
