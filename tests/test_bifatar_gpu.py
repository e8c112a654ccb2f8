"""Bifatar on the GPU against the plain implementation: each mechanism's kernels alone, then whole models in float32
and bfloat16 - whole prompts, token-by-token decoding, portions down to two tokens, unequal batches against each
request alone, slots and pages used again, keys far away, at page borders and at the window's edges, long decoding, greedy
generation through the engine's entry point and scheduler, the command line and the trace runner."""

import json
import subprocess
import sys
from pathlib import Path

import pytest
import torch
import torch.nn.functional as F

import flashdecode_cuda_b200 as fd
from flashdecode_cuda_b200 import kernels as K
from flashdecode_cuda_b200.parts.rope import RotaryScaled
from helpers import prompts_for, rel_err
from bifatar_helpers import (BIFATAR, MODEL_TOL as TOL, Truth, oracle_logits, plain_greedy, random_config, raw_config, truth,
                             weights_of, write_folder)
from plain import bifatar_plain as P

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parent.parent
DEV = "cuda"
NAMES = ["U", "V", "W"]
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


def portions(lens, cuts):
    """Steps that feed sequences of ``lens`` tokens in portions of ``cuts``: (rows, tokens before, tokens of the step)."""
    done = [0] * len(lens)
    for cut in cuts:
        rows = [r for r in range(len(lens)) if done[r] < lens[r]]
        if not rows:
            return
        n = [min(cut, lens[r] - done[r]) for r in rows]
        yield rows, [done[r] for r in rows], n
        for r, k in zip(rows, n):
            done[r] += k
    assert done == list(lens)


def f32(*shape):
    return torch.full(shape, float("nan"), device=DEV)


def new_status():
    return torch.zeros(1, dtype=torch.int32, device=DEV)


# ---------------------------------------------------------------- norm, rotation, mixing, append
ROPE_CASES = [  # n_q, n_kv, d_true, d, dv, rot, whole norm, head norm
    (4, 2, 32, 32, 24, 32, True, False), (6, 3, 40, 40, 80, 16, True, False), (3, 1, 18, 24, 16, 6, True, False),
    (4, 4, 64, 64, 64, 64, False, True), (2, 1, 128, 128, 40, 96, False, True), (5, 1, 20, 64, 64, 20, False, True),
    (2, 2, 136, 136, 8, 136, True, True), (3, 3, 48, 48, 48, 0, False, True), (1, 1, 16, 16, 16, 2, True, True),
    (16, 4, 128, 128, 128, 64, True, False)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", ROPE_CASES)
@pytest.mark.parametrize("mix", ["", "source", "mix"])
def test_norms_rotation_value_mixing_and_append(dtype, case, mix):
    """Two sequences in portions, their columns at an offset of a wider projection, pages of 4 tokens: q and the cached keys
    are the whole-projection norm, the rotation of pairs (i, i + rot/2) and the unit norm per head, the cached values those of
    the token or mixed with the first layer's; the means run over the true sizes of padded heads."""
    n_q, n_kv, dt_true, d, dv, rot, whole, unit = case
    torch.manual_seed(sum(case))
    dt, bs, col0, eps = TD[dtype], 4, 8, 1e-5
    lens, cuts = [13, 9], [5, 1, 1, 6]
    C = (n_q + n_kv) * d + n_kv * dv
    u = [torch.randn(n, col0 + C + 4).to(dt) for n in lens]
    for x in u:
        for h in range(n_q + n_kv):                         # padded dimensions arrive as zeros
            x[:, col0 + h * d + dt_true:col0 + (h + 1) * d] = 0
    dv_true = dv - 4 if dv % 8 == 0 and dv > 16 else dv     # value heads may be padded too
    for x in u:
        for h in range(n_kv):
            at = col0 + (n_q + n_kv) * d + h * dv
            x[:, at + dv_true:at + dv] = 0
    first = [torch.randn(n, n_kv * dv_true).to(dt) for n in lens]
    lam = torch.tensor([0.3])
    wq, wk = 1 + 0.2 * torch.randn(n_q, d), 1 + 0.2 * torch.randn(n_kv, d)
    wq[:, dt_true:] = 0
    wk[:, dt_true:] = 0
    k_pool = torch.zeros(16, n_kv, bs, d, dtype=dt, device=DEV)
    v_pool = torch.zeros(16, n_kv, bs, dv, dtype=dt, device=DEV)
    table = torch.full((4, 8), -1, dtype=torch.int32, device=DEV)
    slots = [2, 0]
    table[2, :4], table[0, :4] = i32([5, 1, 7, 3]), i32([0, 9, 2, 11])
    pos = None
    if rot:
        pos = RotaryScaled(rot, 1000.0)
        pos.prepare(64, _Rt)
    status = new_status()
    q_got = [torch.zeros(n, n_q * d) for n in lens]
    left = [torch.zeros(n, n_kv * dv_true) for n in lens]
    for rows, ctx, n in portions(lens, cuts):
        proj = torch.cat([u[r][c:c + k] for r, c, k in zip(rows, ctx, n)]).to(DEV).contiguous()
        tok_row, tok_pos, row_slot, *_ = step_arrays(ctx, n, [slots[r] for r in rows])
        q = torch.zeros(sum(n), n_q * d, dtype=dt, device=DEV)
        vf = torch.cat([first[r][c:c + k] for r, c, k in zip(rows, ctx, n)]).to(DEV).contiguous() if mix == "mix" else \
            torch.zeros(sum(n), n_kv * dv_true, dtype=dt, device=DEV)
        mode = {"": K.VALUES_PLAIN, "source": K.VALUES_SOURCE, "mix": K.VALUES_MIXED}[mix]
        K.rope_norm_append(proj, col0, q, k_pool, v_pool, table, wq.reshape(-1).to(DEV) if whole else None,
                           wk.reshape(-1).to(DEV) if whole else None, eps, pos.cos if rot else None, pos.sin if rot else None, rot,
                           unit, tok_row, tok_pos, row_slot, n_q, n_kv, d, dv, True, status, q_count=n_q * dt_true,
                           k_count=n_kv * dt_true, head_count=dt_true, value_mode=mode, v_first=vf if mix else None,
                           lam=lam.to(DEV) if mix == "mix" else None, v_count=dv_true)
        at = 0
        for r, c, k in zip(rows, ctx, n):
            q_got[r][c:c + k] = q[at:at + k].float().cpu()
            left[r][c:c + k] = vf[at:at + k].float().cpu()
            at += k
    assert int(status) == 0
    for r, S in enumerate(lens):
        x = u[r][:, col0:].double()
        want = {}
        for name, c0, heads, w in (("q", 0, n_q, wq), ("k", n_q * d, n_kv, wk)):
            y = x[:, c0:c0 + heads * d].view(S, heads, d)[..., :dt_true]
            if whole:
                y = (P.unit_rms(y.reshape(S, -1), eps)).view(S, heads, dt_true) * w[:, :dt_true].double()
            if rot:
                y = P.rotate_half(y, rot, 1000.0)
            want[name] = P.unit_rms(y, eps) if unit else y
        v = x[:, (n_q + n_kv) * d:(n_q + n_kv) * d + n_kv * dv].view(S, n_kv, dv)[..., :dv_true].reshape(S, -1)
        if mix == "source":
            assert torch.equal(left[r].double(), v)
        if mix == "mix":
            v = 0.7 * v + 0.3 * first[r].double()
        assert rel_err(q_got[r].view(S, n_q, d)[..., :dt_true], want["q"]) < KTOL[dtype] * 0.5
        assert bool((q_got[r].view(S, n_q, d)[..., dt_true:] == 0).all())
        for t in range(S):
            blk = int(table[slots[r], t // bs])
            assert rel_err(k_pool[blk, :, t % bs, :dt_true], want["k"][t]) < KTOL[dtype] * 0.5
            assert rel_err(v_pool[blk, :, t % bs, :dv_true].reshape(-1), v[t]) < KTOL[dtype] * 0.5
            assert bool((v_pool[blk, :, t % bs, dv_true:] == 0).all())


def test_append_reports_a_missing_page_and_a_position_beyond_the_table():
    dt, d = torch.float32, 16
    proj = torch.randn(2, 3 * d, device=DEV)
    pool = torch.zeros(2, 1, 4, d, device=DEV)
    table = torch.full((1, 2), -1, dtype=torch.int32, device=DEV)
    pos = RotaryScaled(16, 100.0)
    pos.MIN_TABLE = 4
    pos.prepare(4, _Rt)
    for start, bit in ((0, K.STATUS_BAD_BLOCK), (5, K.STATUS_BAD_POSITION)):
        table[0, :] = -1 if bit == K.STATUS_BAD_BLOCK else 1
        status = new_status()
        tok_row, tok_pos, row_slot, *_ = step_arrays([start], [2], [0])
        K.rope_norm_append(proj, 0, torch.zeros(2, d, device=DEV), pool, pool.clone(), table, None, None, 1e-5, pos.cos, pos.sin, 16,
                           True, tok_row, tok_pos, row_slot, 1, 1, d, d, True, status)
        assert int(status) == bit


# ---------------------------------------------------------------- the gated delta rule
DELTA_CASES = [  # heads, q/k heads, dim, vdim, taps, decay rank, gate rank
    (2, 2, 16, 24, 4, 8, 8), (4, 2, 40, 10, 3, 7, 12), (3, 1, 64, 64, 1, 24, 5), (6, 3, 10, 33, 2, 16, 16), (2, 1, 128, 40, 5, 64, 80),
    (1, 1, 136, 17, 6, 3, 100), (2, 2, 128, 128, 4, 128, 128)]
DELTA_CUTS = [2, 2, 19, 1, 1, 1, 3, 41, 99, 40]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", DELTA_CASES)
@pytest.mark.parametrize("form", ["tokens", "blocks", "chunks"])
def test_gated_delta_rule_in_portions(dtype, case, form):
    """What enters the recurrence and the recurrence itself, in portions down to one token with ring and state carried, from
    columns at an offset: heads that share q and k, channels that forget nearly everything or nothing at once, step sizes
    of nearly zero and one, a key that comes back hundreds of tokens later, slots that held other sequences before.
    ``form``: long portions token by token, in blocks of four or in chunks of sixteen on the tensor cores; in the last, the
    narrow vectors come expanded, as long prompts have them."""
    H, Hk, d, dv, taps, ra, rg = case
    products = form == "chunks"
    if products and not K.delta_chunks_takes(d):
        pytest.skip("key size")
    torch.manual_seed(sum(case))
    dt, col0 = TD[dtype], 5
    lens, slots = [209, 120], [2, 0]
    nk, nv = Hk * d, H * dv
    C = 2 * nk + nv
    cols = [col0, col0 + nk, col0 + 2 * nk, col0 + C + ra + rg, col0 + C, col0 + C + ra]
    u = [torch.randn(n, col0 + C + ra + rg + H + 3).to(dt) for n in lens]
    for x in u:
        x[::7, cols[3]] = 8.0                               # step sizes near one, and near zero
        x[3::7, cols[3]] = -9.0
    u[0][-1, col0 + nk:col0 + 2 * nk] = u[0][4, col0 + nk:col0 + 2 * nk]
    conv_w = torch.randn(C, taps) * 0.5
    A_log, dt_bias = torch.randn(H) * 0.5, torch.randn(H * d) - 2
    dt_bias[0], dt_bias[-1] = 6.0, -12.0                    # a channel that forgets at once and one that forgets nothing
    a2, g2 = (torch.randn(H * d, ra) / ra ** 0.5).to(dt), (torch.randn(nv, rg) / rg ** 0.5).to(dt)
    ring = torch.full((4, taps, C), 7.0, device=DEV)        # another sequence's values
    state = torch.zeros(4, H, d, dv, device=DEV)
    up4 = lambda n: -(-n // 4) * 4
    o_got, z_got = [torch.zeros(n, nv) for n in lens], [torch.zeros(n, nv) for n in lens]
    for rows, ctx, n in portions(lens, DELTA_CUTS):
        proj = torch.cat([u[r][c:c + k] for r, c, k in zip(rows, ctx, n)]).to(DEV).contiguous()
        T = sum(n)
        tok_row, tok_pos, row_slot, q_start, q_len, ctx_len = step_arrays(ctx, n, [slots[r] for r in rows])
        q, k = f32(T, Hk, up4(d)), f32(T, Hk, up4(d))
        v, g, beta, gz = f32(T, H, up4(dv)), f32(T, H, up4(d)), f32(T, H), f32(T, nv)
        za = None
        if products:
            za = (proj[:, cols[4]:cols[4] + ra].float() @ a2.to(DEV).float().t()).contiguous()
            gz = (proj[:, cols[5]:cols[5] + rg].float() @ g2.to(DEV).float().t()).contiguous()
        K.delta_prepare(proj, cols, conv_w.to(DEV), ring, True, A_log.to(DEV), dt_bias.to(DEV), d ** -0.5, q, k, v, g, beta, gz,
                        tok_row, tok_pos, row_slot, q_start, q_len, H, Hk, d, dv, a2=None if products else a2.to(DEV), z_a=za,
                        g2=None if products else g2.to(DEV))
        if max(n) > 1 and taps > 1:
            K.conv_ring_update(proj, col0, ring, row_slot, q_start, q_len, ctx_len, len(rows))
        o = f32(T, nv)
        step = (q, k, v, g, beta, state, o, row_slot, q_start, q_len, len(rows), True)
        if form == "tokens" or max(n) <= K.delta_scan_single():
            K.delta_scan(*step)
        elif form == "blocks":
            K.delta_scan(*step, max(n), f32(K.delta_scan_scratch_floats(T, len(rows), H, d)))
        else:
            K.delta_scan(*step, short_only=True)
            K.delta_chunks(*step, max(n), torch.zeros(K.delta_chunks_scratch_bytes(T, len(rows), H, d), dtype=torch.uint8, device=DEV))
        at = 0
        for r, c, m in zip(rows, ctx, n):
            o_got[r][c:c + m], z_got[r][c:c + m] = o[at:at + m].cpu(), gz[at:at + m].cpu()
            at += m
    for r, S in enumerate(lens):
        x = u[r].double()
        conv = F.silu(P.short_conv(x[:, col0:col0 + C], conv_w.double()))
        q = P.unit_vector(conv[:, :nk].view(S, Hk, d)) * d ** -0.5
        k = P.unit_vector(conv[:, nk:2 * nk].view(S, Hk, d))
        v = conv[:, 2 * nk:].reshape(S, H, dv)
        beta = torch.sigmoid(x[:, cols[3]:cols[3] + H])
        z = x[:, cols[4]:cols[4] + ra] @ a2.double().t() + dt_bias.double()
        g = torch.exp(-torch.exp(A_log.double())[None, :, None] * P.softplus(z).view(S, H, d))
        assert rel_err(o_got[r], P.delta_recurrence(q, k, v, g, beta).reshape(S, nv)) < (2e-4 if form == "chunks" else 3e-5)
        assert rel_err(z_got[r], x[:, cols[5]:cols[5] + rg] @ g2.double().t()) < 1e-5


@pytest.mark.parametrize("dtype", DTYPES)
def test_delta_rule_reads_back_what_it_wrote(dtype):
    """With decays of one and a step size of one, writing v under a unit key k leaves S^T k = v exactly, whatever was
    there: the same key written twice with different values reads back the second."""
    T, d, dv = 40, 32, 16
    torch.manual_seed(3)
    k = P.unit_vector(torch.randn(T, 1, d))
    k[30] = k[2]
    v = torch.randn(T, 1, dv)
    q = torch.zeros(T, 1, d)
    q[35], q[3] = k[30], k[2]
    state, o = torch.zeros(1, 1, d, dv, device=DEV), f32(T, dv)
    K.delta_scan(q.to(DEV), k.to(DEV), v.to(DEV), torch.zeros(T, 1, d, device=DEV), torch.ones(T, 1, device=DEV), state, o, i32([0]), i32([0]),
                 i32([T]), 1, True)
    want = P.delta_recurrence(q.double(), k.double(), v.double(), torch.ones(T, 1, d).double(), torch.ones(T, 1).double()).reshape(T, dv)
    assert rel_err(o, want) < 1e-5
    o1 = f32(3, dv)                                          # right after the write the value is there
    K.delta_scan(k[:3].to(DEV), k[:3].contiguous().to(DEV), v[:3].to(DEV), torch.zeros(3, 1, d, device=DEV), torch.ones(3, 1, device=DEV),
                 torch.zeros_like(state), o1, i32([0]), i32([0]), i32([3]), 1, True)
    assert rel_err(o1, v[:3, 0].double()) < 1e-5


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,dv", [(3, 40), (1, 128), (5, 6)])
def test_norm_per_head_with_a_sigmoid_gate(dtype, H, dv):
    torch.manual_seed(H + dv)
    T, eps, col = 9, 1e-5, 3
    o, z, w = torch.randn(T, H * dv), torch.randn(T, H * dv) * 3, 1 + 0.1 * torch.randn(dv)
    out = torch.zeros(T, col + H * dv + 2, dtype=TD[dtype], device=DEV)
    K.head_norm_gate(o.to(DEV), out, col, H, dv, eps, w.to(DEV), None, 0, 1.7, sigmoid_gate=z.to(DEV))
    want = 1.7 * P.unit_rms(o.double().view(T, H, dv), eps) * w.double() * torch.sigmoid(z.double()).view(T, H, dv)
    assert rel_err(out[:, col:col + H * dv], want.reshape(T, -1)) < KTOL[dtype] * 0.5
    assert bool((out[:, :col] == 0).all()) and bool((out[:, col + H * dv:] == 0).all())


# ---------------------------------------------------------------- the state-space mixer
SSD_CASES = [  # heads, vdim, state, groups, parts, taps
    (4, 24, 20, 2, 3, 4), (1, 64, 64, 1, 1, 1), (3, 10, 136, 3, 2, 6), (8, 64, 128, 2, 4, 4), (6, 16, 128, 1, 6, 2), (4, 40, 8, 4, 1, 3)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", SSD_CASES)
@pytest.mark.parametrize("cuts", [[2, 2, 19, 1, 1, 1, 3, 40, 300, 60], [390]])
def test_state_space_mixer_between_its_products(dtype, case, cuts):
    """Convolution with bias, step sizes, the recurrence (short portions, portions of several segments, single tokens), skip,
    gate and norm in parts, from columns at an offset into a wider buffer; decays of nearly zero and nearly one; slots
    that held other sequences before; a token of one sequence that stands out hundreds of positions back."""
    from flashdecode_cuda_b200.parts.ssd import Mamba2
    H, dv, N, G, parts, taps = case
    torch.manual_seed(sum(case))
    dt, col0, acol, eps = TD[dtype], 4, 8, 1e-5
    mixer = Mamba2("m", 32, H, dv, N, G, parts, taps, eps)
    inner, C = H * dv, H * dv + 2 * G * N
    A_log, D, dt_bias = torch.randn(H) * 0.7, torch.randn(H), torch.randn(H) - 2
    A_log[0], dt_bias[-1] = -6.0, 3.0
    tensors = {"m.in": torch.zeros(inner + C + H, 32, dtype=dt), "m.conv": torch.randn(C, taps) * 0.5, "m.conv.b": torch.randn(C) * 0.3,
               "m.dt_bias": dt_bias, "m.A_log": A_log, "m.D": D, "m.norm": 1 + 0.1 * torch.randn(inner), "m.o": torch.zeros(32, inner, dtype=dt)}
    keep = dict(tensors)
    rt = _Rt()
    rt.dtype, rt.status, rt.sm_count = dt, new_status(), 148
    mixer.bind({k: v.to(DEV) for k, v in tensors.items()}, rt)
    lens, slots = [391 if sum(cuts) < 391 else 390, 150], [2, 0]
    lens[0] = min(lens[0], sum(cuts))
    u = [torch.randn(n, col0 + inner + C + H + 3).to(dt) for n in lens]
    u[0][5] *= 4
    from flashdecode_cuda_b200.engine.model import Workspace
    ws = Workspace(torch.device(DEV))

    class Ctx:
        pass

    class Lc:
        writes = True
        states = {"state": torch.zeros(4, H, N, dv, device=DEV), "ring": torch.full((4, taps, C), 7.0, device=DEV)}
    if taps == 1:
        del Lc.states["ring"]
    got = [torch.zeros(n, inner) for n in lens]
    for rows, ctx_lens, n in portions(lens, cuts):
        c = Ctx()
        c.T, c.ws, c.n_rows, c.max_q_len = sum(n), ws, len(rows), max(n)
        c.tok_row, c.tok_pos, c.row_slot, c.row_q_start, c.row_q_len, c.row_ctx_len = step_arrays(ctx_lens, n, [slots[r] for r in rows])
        proj = torch.cat([u[r][a:a + k] for r, a, k in zip(rows, ctx_lens, n)]).to(DEV).contiguous()
        act = torch.zeros(c.T, acol + inner + 4, dtype=dt, device=DEV)
        mixer.inner(c, proj, col0, Lc, act, acol, 0.6)
        at = 0
        for r, a, k in zip(rows, ctx_lens, n):
            got[r][a:a + k] = act[at:at + k, acol:acol + inner].float().cpu()
            at += k
        assert bool((act[:, :acol] == 0).all()) and bool((act[:, acol + inner:] == 0).all())
    assert int(rt.status) == 0
    for r, S in enumerate(lens):
        x = u[r][:, col0:].double()
        z, conv, raw = x[:, :inner], x[:, inner:inner + C], x[:, inner + C:inner + C + H]
        conv = F.silu(P.short_conv(conv, keep["m.conv"].double(), keep["m.conv.b"].double()))
        xs, B, Cc = torch.split(conv, [inner, G * N, G * N], dim=-1)

        def mixed(round_to):
            """The mixer's output; the convolved channels enter the recurrence rounded to ``round_to``."""
            parts_in = [t.to(round_to).double() for t in (xs, B, Cc)]
            y = P.ssd_recurrence(parts_in[0].reshape(S, H, dv), parts_in[1].reshape(S, G, N), parts_in[2].reshape(S, G, N),
                                 P.softplus(raw + dt_bias.double()), A_log.double(), torch.zeros(H).double()).reshape(S, inner)
            y = y + (D.double()[:, None] * xs.reshape(S, H, dv)).reshape(S, inner)
            return 0.6 * P.gated_part_norm(y, z, keep["m.norm"].double(), parts, eps)
        want = mixed(torch.float64)
        if dtype == "float32":
            assert rel_err(got[r], want) < 5e-5, f"sequence {r}"
        else:
            # long portions round the convolved channels: a part whose channels nearly cancel may move by what that moves it
            moved = (mixed(torch.bfloat16) - want).abs().view(S, parts, -1).amax(-1, keepdim=True)
            err = (got[r].double() - want).abs().view(S, parts, -1)
            assert bool((err < 1e-2 * want.abs().max() + 3 * moved).all()), f"sequence {r}"


# ---------------------------------------------------------------- capped attention with a keyless term
CAP_CASES = [  # d, dv, group, kv heads, window, softcap, sink, page
    (64, 64, 2, 2, 19, 5.0, True, 16), (128, 128, 4, 1, 33, 20.0, True, 64), (64, 64, 12, 1, None, 3.0, False, 8), (24, 40, 3, 2, 10, 8.0, True, 8),
    (128, 128, 1, 2, 1, 2.0, True, 16), (128, 128, 2, 2, None, 50.0, True, 16), (64, 64, 4, 2, 100, None, True, 16), (16, 8, 2, 1, 7, 1.0, False, 4),
    (128, 128, 16, 1, 70, 4.0, False, 64)]


def _cap_case(dtype, case, cuts, lens, tensor_cores=True):
    """Attention over a paged cache filled portion by portion, into columns of a wider buffer, scaled.  Every seventh key of
    a sequence is the query's own direction (it stands out just inside one query's window and just outside the next one's) and
    key 2 far back stands out for the last queries; the keyless terms are a good part of the denominators."""
    d, dv, G, n_kv, window, cap, sink, bs = case
    torch.manual_seed(d + dv + G + (window or 0))
    dt, n_q, scale, acol, oscale = TD[dtype], G * n_kv, 0.7 * d ** -0.5, 16, 1.3
    q = [torch.randn(n, n_q, d).to(dt) for n in lens]
    k = [torch.randn(n, n_kv, d).to(dt) for n in lens]
    v = [torch.randn(n, n_kv, dv).to(dt) for n in lens]
    for qq, kk in zip(q, k):
        one = torch.nn.functional.normalize(torch.randn(n_kv, d), dim=-1) * (d ** 0.5)
        kk[::7] = (one * 2.5).to(dt)
        kk[2] = (one * 3.5).to(dt)
        qq += (one.repeat_interleave(G, dim=0) * 1.0).to(dt)
    sk = torch.linspace(-1, 4, n_q) if sink else None
    slots = [1, 0]
    nb = [-(-n // bs) for n in lens]
    table = torch.full((2, max(nb) + 1), -1, dtype=torch.int32, device=DEV)
    perm = torch.randperm(sum(nb)).tolist()
    for r in range(len(lens)):
        table[slots[r], :nb[r]] = i32(perm[:nb[r]])
        perm = perm[nb[r]:]
    k_pool = torch.full((sum(nb), n_kv, bs, d), float("nan"), dtype=dt, device=DEV)
    v_pool = torch.full((sum(nb), n_kv, bs, dv), float("nan"), dtype=dt, device=DEV)
    status = new_status()
    got = [torch.zeros(n, n_q * dv) for n in lens]
    for rows, ctx, n in portions(lens, cuts):
        for r, c, m in zip(rows, ctx, n):
            for t in range(c, c + m):
                b = int(table[slots[r], t // bs])
                k_pool[b, :, t % bs], v_pool[b, :, t % bs] = k[r][t].to(DEV), v[r][t].to(DEV)
        tok_row, tok_pos, row_slot, q_start, q_len, ctx_len = step_arrays(ctx, n, [slots[r] for r in rows])
        T = sum(n)
        qs = torch.cat([q[r][c:c + m].reshape(m, -1) for r, c, m in zip(rows, ctx, n)]).to(DEV).contiguous()
        act = torch.zeros(T, acol + n_q * dv + 8, dtype=dt, device=DEV)
        splits, split_len, scratch = 1, 0, None
        if max(n) == 1:
            split_len = 32
            splits = max(1, -(-(max(ctx) + 1) // 32))
            scratch = f32(K.attention_scratch_floats(T, n_q, dv, splits)) if splits > 1 else None
        K.attention_ext(qs, k_pool, v_pool, act, table, tok_row, row_slot, q_start, q_len, ctx_len, len(rows), max(n), n_q, n_kv, d, scale,
                        window or 0, splits, split_len, scratch, status, softcap=cap or 0.0, sink=sk.to(DEV) if sink else None,
                        tensor_cores=tensor_cores, out_col=acol, out_scale=oscale)
        at = 0
        for r, c, m in zip(rows, ctx, n):
            got[r][c:c + m] = act[at:at + m, acol:acol + n_q * dv].float().cpu()
            at += m
        assert bool((act[:, :acol] == 0).all()) and bool((act[:, acol + n_q * dv:] == 0).all())
    assert int(status) == 0
    for r, S in enumerate(lens):
        want = oscale * P.attend(q[r].double(), k[r].double(), v[r].double(), scale, cap, window, sk.double() if sink else None)
        err = (got[r].double() - want.reshape(S, -1)).abs().amax(-1) / want.abs().max()
        assert float(err.max()) < (2e-5 if dtype == "float32" else 1.2e-2), f"{case}: sequence {r}, position {int(err.argmax())}"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", CAP_CASES)
@pytest.mark.parametrize("tensor_cores", [True, False])
def test_capped_attention_whole_prompts(dtype, case, tensor_cores):
    _cap_case(dtype, case, [150], [150, 77], tensor_cores)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", CAP_CASES)
def test_capped_attention_in_portions_and_token_by_token(dtype, case):
    _cap_case(dtype, case, [2, 61, 3] + [1] * 40 + [30] + [1] * 14, [150, 101])


@pytest.mark.parametrize("form", [1, 2, 4])
def test_capped_attention_in_every_form_of_the_decode_and_prompt_kernels(form):
    K.attn_decode_set_form(form)
    K.attn_prefill_set_form(min(form, 2))
    try:
        for case in (CAP_CASES[0], CAP_CASES[1], CAP_CASES[5]):
            _cap_case("bfloat16", case, [120] + [1] * 30, [150, 140])
    finally:
        K.attn_decode_set_form(0)
        K.attn_prefill_set_form(0)


# ---------------------------------------------------------------- feed-forward beside the mixers
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,C,xc,oc", [(3, 64, 8, 16), (70, 41, 3, 5), (1, 8, 0, 0)])
def test_relu_squared_between_columns(dtype, T, C, xc, oc):
    torch.manual_seed(T + C)
    x = torch.randn(T, xc + C + 5 - (xc + C + 5) % 8 + 8).to(TD[dtype])
    out = torch.zeros(T, oc + C + 16 - (oc + C) % 8, dtype=TD[dtype], device=DEV)
    K.relu2_cols(x.to(DEV), xc, out, oc, C)
    assert rel_err(out[:, oc:oc + C], P.relu_squared(x[:, xc:xc + C].double())) < KTOL[dtype] * 0.5
    assert bool((out[:, :oc] == 0).all()) and bool((out[:, oc + C:] == 0).all())


@pytest.mark.parametrize("M", [1, 3, 8, 16, 17, 40, 128])
@pytest.mark.parametrize("N,row,Kd", [(1168, 144, 256), (400, 16, 2048), (4096, 2048, 512)])
@pytest.mark.parametrize("biased", [False, True])
def test_products_whose_last_rows_are_a_feed_forwards(M, N, row, Kd, biased):
    """The streaming products' epilogue: rows from ``row`` on leave max(., 0)^2 in another buffer's columns, the others are as
    they are without it, and nothing else of either buffer changes."""
    from flashdecode_cuda_b200.parts.linear import matmul, takes_tail
    torch.manual_seed(M + N)
    x, w = torch.randn(M, Kd).bfloat16(), (torch.randn(N, Kd) / Kd ** 0.5).bfloat16()
    b = torch.randn(N).bfloat16() if biased else None
    col, ld = 8, 8 + N - row + 24
    assert takes_tail(M, N, Kd, torch.bfloat16, row, ld, col)
    out, out2 = torch.full((M, N), 7.0, dtype=torch.bfloat16, device=DEV), torch.full((M, ld), 7.0, dtype=torch.bfloat16, device=DEV)
    plain = torch.zeros_like(out)
    status = new_status()
    bd = b.to(DEV) if biased else None
    matmul(x.to(DEV), w.to(DEV), bd, plain, status=status)
    matmul(x.to(DEV), w.to(DEV), bd, out, status=status, tail=(row, out2, col))
    assert int(status) == 0
    assert torch.equal(out[:, :row], plain[:, :row]) and bool((out[:, row:] == 7).all())
    want = P.relu_squared((x.double() @ w.double().t() + (b.double() if biased else 0))[:, row:])
    assert rel_err(out2[:, col:col + N - row], want) < 1e-2
    assert bool((out2[:, :col] == 7).all()) and bool((out2[:, col + N - row:] == 7).all())


# ---------------------------------------------------------------- whole models
@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    tmp = tmp_path_factory.mktemp("bifatar")
    return {n: write_folder(tmp, n, seed=31) for n in NAMES}


@pytest.fixture(scope="module")
def engines(folders):
    return {(n, d): fd.load(folders[n], device="cuda", dtype=d) for n in NAMES for d in DTYPES}


def _vocab(name):
    return BIFATAR[name]["vocab"]


def _lengths(name):
    # around the windows (27 and 11 / none / 1 and 40), the taps and the pages
    return {"U": [1, 2, 5, 11, 12, 27, 28, 33, 75, 140], "V": [1, 16, 17, 64, 65, 129], "W": [1, 3, 9, 17, 40, 41, 100, 201]}[name]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
@pytest.mark.parametrize("block_size", [8, 64])
def test_whole_prompts(engines, folders, name, dtype, block_size):
    eng = engines[(name, dtype)]
    cache = eng.model.new_cache(max_tokens=320, block_size=block_size)
    for p in prompts_for(_vocab(name), _lengths(name), seed=1):
        slot = cache.admit()
        got = eng.model.step(cache, [slot], [p], "all")
        assert truth(folders[name], p).excess(got, range(len(p)), dtype) < 1, f"prompt of {len(p)} tokens"
        cache.release(slot)
    eng.model.check_status()
    cache.check_invariants()


def test_every_layer_in_float32(engines, folders):
    """The residual stream after every layer against the plain one."""
    for name in NAMES:
        eng = engines[(name, "float32")]
        (p,) = prompts_for(_vocab(name), [45], seed=2)
        trace = []
        P.forward(raw_config(folders[name]), weights_of(folders[name]), p, trace=trace)
        cache = eng.model.new_cache(max_tokens=64)
        slot = cache.admit()
        eng.model.trace = {}
        eng.model.step(cache, [slot], [p], None)
        got, eng.model.trace = eng.model.trace, None
        assert len(trace) == len(eng.model.schedule)
        for i, want in enumerate(trace):
            assert rel_err(got[f"layer.{i}"], want) < 1e-5, f"{name}: layer {i}"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_prefill_then_token_by_token_across_window_edges(engines, folders, name, dtype):
    """A prompt of one token or of thirty, then so many single tokens that every window of the model passes over
    decoded tokens and the kept positions are left behind while decoding."""
    eng = engines[(name, dtype)]
    cache = eng.model.new_cache(max_tokens=256, block_size=16)
    n_decode = {"U": 60, "V": 45, "W": 70}[name]
    for head in (1, 30):
        (p,) = prompts_for(_vocab(name), [head + n_decode], seed=3 + head)
        want = truth(folders[name], p)
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
    """Four hundred single tokens after a short prompt: the states keep what the plain recurrences keep, and the
    window's pages are given back and used again."""
    name = "U"
    eng = engines[(name, "float32")]
    (p,) = prompts_for(_vocab(name), [420], seed=9)
    want = oracle_logits(folders[name], p)
    cache = eng.model.new_cache(max_tokens=512, block_size=8)
    slot = cache.admit()
    eng.model.step(cache, [slot], [p[:20]], None)
    for i in range(20, len(p)):
        got = eng.model.step(cache, [slot], [[p[i]]], "last")
        if i % 50 == 0 or i > 410:
            assert rel_err(got[0], want[i]) < TOL["float32"], f"position {i}"
    cache.release(slot)
    eng.model.check_status()
    cache.check_invariants()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_portions_of_several_sizes(engines, folders, name, dtype):
    """A prompt cut into portions of 2, 3, 1, 7, 33, ... tokens gives the logits of the whole prompt."""
    eng = engines[(name, dtype)]
    (p,) = prompts_for(_vocab(name), [150], seed=5)
    want = truth(folders[name], p)
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
        bound = want.allowed(dtype) if dtype == "bfloat16" else want.allowed(dtype) * 0.05
        assert bool((apart < bound).all()), f"portions {sizes[:4]}..."
    eng.model.check_status()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_unequal_batch_equals_each_request_alone_and_slots_are_used_again(engines, folders, name, dtype):
    eng = engines[(name, dtype)]
    cache = eng.model.new_cache(max_tokens=64 * 8, block_size=8, max_slots=4)
    for batch_no, lengths in enumerate([[9, 80, 1, 44], [130, 3, 26], [5, 5, 62, 25]]):
        reqs = prompts_for(_vocab(name), lengths, seed=30 + batch_no)
        decode = [min(k, len(p) - 1) for k, p in zip([6, 40, 0, 9], reqs)]
        heads = [len(p) - k for p, k in zip(reqs, decode)]
        slots = [cache.admit() for _ in reqs]                 # the second and third batch get used slots, states and pages
        got = eng.model.step(cache, slots, [p[:h] for p, h in zip(reqs, heads)], "last")
        for i, (p, h) in enumerate(zip(reqs, heads)):
            assert truth(folders[name], p).excess(got[i], [h - 1], dtype) < 1
        live = [i for i in range(len(reqs)) if heads[i] < len(reqs[i])]
        for i in set(range(len(reqs))) - set(live):
            cache.release(slots[i])
        step = 0
        while live:
            got = eng.model.step(cache, [slots[i] for i in live], [[reqs[i][heads[i] + step]] for i in live], "last")
            for j, i in enumerate(live):
                want = truth(folders[name], reqs[i])
                assert want.excess(got[j], [heads[i] + step], dtype) < 1, f"batch {batch_no}, request {i}, decoded token {step}"
            step += 1
            for i in [i for i in live if heads[i] + step >= len(reqs[i])]:
                cache.release(slots[i])
                live.remove(i)
        cache.check_invariants()
        assert cache.blocks_in_use() == [0] * len(cache.groups)
    eng.model.check_status()


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


@pytest.mark.parametrize("seed", range(100, 124))
def test_configurations_drawn_at_random_in_float32(tmp_path, seed):
    """Sizes and layer orders nobody chose: a whole prompt, then a batch of unequal prompts decoded together, against
    the plain model."""
    cfg = random_config(seed)
    folder = fd.write_random_model(tmp_path / "m", cfg, seed)
    W = weights_of(folder)
    cfg = raw_config(folder)
    reqs = prompts_for(cfg["vocab"], [1, 37, 131], seed=seed)
    want = [Truth(cfg, W, r) for r in reqs]
    eng = fd.load(folder, device="cuda", dtype="float32")
    cache = eng.model.new_cache(max_tokens=256, max_slots=4, slack_blocks=4, block_size=16)
    s = cache.admit()
    assert want[2].excess(eng.model.step(cache, [s], [reqs[2]], "all"), range(len(reqs[2])), "float32") < 1, cfg
    cache.release(s)
    slots = [cache.admit() for _ in reqs]
    heads = [1, 30, 120]
    got = eng.model.step(cache, slots, [r[:h] for r, h in zip(reqs, heads)], "last")
    for i in range(3):
        assert want[i].excess(got[i], [heads[i] - 1], "float32") < 1, cfg
    cache.release(slots[0])
    for step in range(7):
        live = [i for i in (1, 2) if heads[i] + step < len(reqs[i])]
        got = eng.model.step(cache, [slots[i] for i in live], [[reqs[i][heads[i] + step]] for i in live], "last")
        for j, i in enumerate(live):
            assert want[i].excess(got[j], [heads[i] + step], "float32") < 1, (cfg, i, step)
    eng.model.check_status()
    cache.check_invariants()


@pytest.mark.parametrize("seed", range(200, 206))
def test_configurations_drawn_at_random_in_bfloat16(tmp_path, seed):
    cfg = random_config(seed)
    folder = fd.write_random_model(tmp_path / "m", cfg, seed)
    W = weights_of(folder)
    cfg = raw_config(folder)
    reqs = prompts_for(cfg["vocab"], [20, 150], seed=seed)
    want = [Truth(cfg, W, r) for r in reqs]
    eng = fd.load(folder, device="cuda", dtype="bfloat16")
    cache = eng.model.new_cache(max_tokens=256, max_slots=4, slack_blocks=4, block_size=16)
    slots = [cache.admit() for _ in reqs]
    heads = [10, 140]
    got = eng.model.step(cache, slots, [r[:h] for r, h in zip(reqs, heads)], "last")
    for i in range(2):
        assert want[i].excess(got[i], [heads[i] - 1], "bfloat16") < 1, cfg
    for step in range(10):
        got = eng.model.step(cache, slots, [[reqs[i][heads[i] + step]] for i in range(2)], "last")
        for i in range(2):
            assert want[i].excess(got[i], [heads[i] + step], "bfloat16") < 1, (cfg, i, step)
    eng.model.check_status()


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_prompts_at_sizes_of_the_tensor_core_kernels(tmp_path, dtype):
    """Heads of 64 and 128, prompts of several hundred tokens: the tensor-core attention kernels with cap, keyless term and
    window, many segments and chunks of the recurrences, narrow vectors expanded by products of their own; every position of
    each prompt alone, then the two together and decoded on."""
    import bifatar_helpers as H
    cfg = H.model(333, 128, 1e-5, [
        H.mamba2(4, 64, 128, 2, 2, 4, H.dense(96)),
        H.parallel(H.left(4, 2, 64, 64, 0.125, (64, 10000.0)), H.delta(2, 2, 64, 64, 4, 16), 0.7, 1.2, H.dense(96)),
        H.attention(4, 1, 128, 128, 0.9, (128, 10000.0), 15.0, 150, True, H.dense(64)),
        H.mamba2(2, 40, 72, 1, 4, 3, H.dense(64)),
        H.parallel(H.left(2, 1, 128, 128, 0.09, (32, 100.0)), H.delta(4, 2, 128, 32, 3, 24), None, None, H.dense(40)),
        H.attention(4, 1, 100, 128, 0.7, (64, 100.0), 5.0, 70, True, H.dense(64))])
    folder = fd.write_random_model(tmp_path / "m", cfg, 7)
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


@pytest.mark.parametrize("name", NAMES)
def test_greedy_generation_through_the_engine(folders, name):
    """``Engine.generate``: the scheduler admits five requests three at a time, decode steps replay captured graphs."""
    eng = fd.load(folders[name], device="cuda", dtype="float32")
    prompts = prompts_for(_vocab(name), [3, 30, 1, 70, 9], seed=50)
    got = eng.generate(prompts, 40, max_batch=3)
    for p, r in zip(prompts, got):
        assert r.tokens == plain_greedy(folders[name], p, 40)
    eng.model.check_status()


@pytest.mark.parametrize("name", ["U", "W"])
def test_greedy_generation_in_bfloat16_picks_a_best_token(folders, name):
    eng = fd.load(folders[name], device="cuda", dtype="bfloat16")
    prompts = prompts_for(_vocab(name), [5, 50, 2], seed=51)
    got = eng.generate(prompts, 30)
    for p, r in zip(prompts, got):
        full = p + r.tokens
        ref = oracle_logits(folders[name], full[:-1])
        scale = float(ref.abs().max())
        for i, tok in enumerate(r.tokens):
            row = ref[len(p) - 1 + i]
            assert float(row.max() - row[tok]) <= 2 * TOL["bfloat16"] * scale, f"token {i}"
    eng.model.check_status()


def test_command_line_generates(folders):
    p = prompts_for(_vocab("V"), [12], seed=52)[0]
    cmd = [sys.executable, "-m", "flashdecode_cuda_b200", "generate", "--model", str(folders["V"]), "--dtype", "float32",
           "--prompt-ids", ",".join(map(str, p)), "--max-new-tokens", "8"]
    r = subprocess.run(cmd, cwd=ROOT, capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert json.loads(r.stdout.strip().splitlines()[-1])["tokens"] == plain_greedy(folders["V"], p, 8)


@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_runner_replays_a_schedule(folders, tmp_path, dtype):
    """Prompts of unequal lengths in one step, then one token each, the shorter request ending earlier; the same
    request again afterwards in the freed slot."""
    name = "U"
    a, b = prompts_for(_vocab(name), [40, 9], seed=53)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:30], "want": [0, 23, 24, 29]},
                                     {"id": "b", "tokens": b[:7], "want": [6]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": [a[30]], "want": [0]}, {"id": "b", "tokens": [b[7]], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": [a[31]], "want": [0]}, {"id": "b", "tokens": [b[8]], "want": [0]}], "end": ["b"]}]
    steps += [{"step": 3 + i, "entries": [{"id": "a", "tokens": [a[32 + i]], "want": [0]}], "end": ["a"] if i == 7 else []}
              for i in range(8)]
    steps.append({"step": 11, "entries": [{"id": "c", "tokens": b, "want": [8]}], "end": ["c"]})
    out = tmp_path / "out"
    r = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(folders[name]), "--dtype", dtype, "--out", str(out),
                        "--max-tokens", "128"], input="\n".join(json.dumps(s) for s in steps) + "\n", cwd=ROOT,
                       capture_output=True, text=True, timeout=900)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(12)]
    V = _vocab(name)
    wa, wb = truth(folders[name], a), truth(folders[name], b)

    def read(i):
        return torch.frombuffer(bytearray((out / f"{i}.f32").read_bytes()), dtype=torch.float32).view(-1, V)
    assert wa.excess(read(0)[:4], [0, 23, 24, 29], dtype) < 1 and wb.excess(read(0)[4:], [6], dtype) < 1
    assert wa.excess(read(1), [30], dtype) < 1
    assert wa.excess(read(2)[:1], [31], dtype) < 1 and wb.excess(read(2)[1:], [8], dtype) < 1
    for i in range(8):
        assert wa.excess(read(3 + i), [32 + i], dtype) < 1
    assert wb.excess(read(11), [8], dtype) < 1
