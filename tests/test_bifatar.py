"""Bifatar without a GPU: the configuration reader, the blueprint, the cache's share (pages per kind of attention, states per
slot), stacked products, and the plain implementation's mechanisms against closed forms."""

import copy
import math

import pytest
import torch

import flashdecode_cuda_b200 as fd
from flashdecode_cuda_b200.cache.paged import PagedCache
from flashdecode_cuda_b200.config import ConfigError, load_config
from flashdecode_cuda_b200.engine.model import Model
from flashdecode_cuda_b200.parts.base import Runtime
from flashdecode_cuda_b200.parts.normed_attention import tensor_core_sizes
from flashdecode_cuda_b200.weights import loader as W
from bifatar_helpers import BIFATAR, random_config
from plain import bifatar_plain as P


# ---------------------------------------------------------------- configuration
@pytest.mark.parametrize("name", sorted(BIFATAR))
def test_config_round_trip(name):
    cfg = load_config(BIFATAR[name])
    assert cfg.architecture == "Bifatar" and cfg.unknown_keys == []
    assert load_config(cfg.to_dict()).to_dict() == cfg.to_dict()
    raw = BIFATAR[name]
    assert [L.type for L in cfg.layers] == [L["type"] for L in raw["layers"]]
    assert cfg.vocab == raw["vocab"] and cfg.width == raw["width"] and cfg.norm_eps == raw["norm"]["eps"]


def test_configurations_drawn_at_random_round_trip():
    for seed in range(40):
        cfg = load_config(random_config(seed))
        assert load_config(cfg.to_dict()).to_dict() == cfg.to_dict()
        m = Model.from_config(cfg, torch.float32, "cpu")
        names = [s.name for s in m.tensor_specs()]
        assert len(names) == len(set(names))


def test_what_a_file_leaves_out():
    cfg = load_config(BIFATAR["V"])
    par, att = cfg.layers[1].mixer, cfg.layers[2].mixer
    assert par.left_scale == par.right_scale == 1.0 and par.left.rot is None and cfg.layers[0].mlp is None
    assert att.softcap is None and att.window is None and att.rot is None and att.v_mix is False
    small = {"architecture": "Bifatar", "vocab": 8, "width": 8, "norm": {"eps": 1e-5}, "layers": [
        {"type": "mamba2", "mixer": {"heads": 2, "vdim": 4, "state": 4}},
        {"type": "parallel", "mixer": {"left": {"heads": 2, "kv_heads": 1, "dim": 4, "scale": 0.5}, "right": {"heads": 2, "dim": 4}}}]}
    cfg = load_config(small)
    m, r = cfg.layers[0].mixer, cfg.layers[1].mixer.right
    assert (m.groups, m.norm_groups, m.conv) == (1, 1, 1) and (r.kv_heads, r.vdim, r.conv, r.rank) == (2, 4, 1, None)
    assert cfg.layers[1].mixer.left.vdim == 4 and cfg.layers[0].mlp is None


def test_config_errors_name_the_place():
    def bad(change, match):
        raw = copy.deepcopy(BIFATAR["U"])
        change(raw)
        with pytest.raises(ConfigError, match=match):
            load_config(raw)
    bad(lambda c: c["layers"][3]["mixer"]["right"].pop("dim"), r"layers\[3\]\.mixer\.right misses 'dim'")
    bad(lambda c: c["layers"][1]["mixer"].update(groups=3), "multiple of groups")
    bad(lambda c: c["layers"][1]["mixer"].update(norm_groups=7), "norm_groups")
    bad(lambda c: c["layers"][0].update(type="retention"), "mixers are")
    bad(lambda c: c["layers"][3]["mixer"]["left"].update(kv_heads=4), "multiple of kv_heads")
    bad(lambda c: c["layers"][3]["mixer"]["right"].update(kv_heads=3), "multiple of kv_heads")
    bad(lambda c: c["layers"][0]["mixer"]["rot"].update(dims=34), "dims")
    bad(lambda c: c["layers"][0]["mixer"].update(softcap=-1.0), "soft cap")
    bad(lambda c: c["layers"][0]["mlp"].update(kind="moe"), "dense")
    bad(lambda c: c["layers"][4]["mixer"].update(vdim=24), "same kv_heads and vdim")
    bad(lambda c: c["norm"].pop("eps"), "norm misses 'eps'")
    odd = copy.deepcopy(BIFATAR["U"])
    odd["layers"][1]["mixer"]["clamp"] = 3
    with pytest.warns(UserWarning, match="does not define"):
        cfg = load_config(odd)
    assert cfg.unknown_keys == ["layers[1].mixer.clamp"] and cfg.to_dict() == load_config(BIFATAR["U"]).to_dict()


# ---------------------------------------------------------------- blueprint and cache layout
def test_blueprint_declares_the_tensors_and_what_every_layer_keeps():
    m = Model.from_config(load_config(BIFATAR["U"]), torch.float32, "cpu")
    spec = {s.name: s for s in m.tensor_specs()}
    assert {"embed", "head", "final.norm", "final.norm.b", "final.norm.alpha", "l0.norm1.alpha", "l0.mix.sink", "l1.mix.in",
            "l1.mix.conv.b", "l1.mix.D", "l3.mix.left.q.b", "l3.mix.left.k.norm", "l3.mix.right.a2", "l3.mix.right.v.conv", "l4.mix.vmix",
            "l4.mlp.down"} <= set(spec)
    assert not any(".norm2" in n for n in spec)                              # one norm per layer
    assert spec["l1.mix.in"].shape == (2 * 96 + 2 * 2 * 20 + 4, 96) and spec["l1.mix.conv"].shape == (96 + 2 * 2 * 20, 4)
    assert spec["l3.mix.right.q"].shape == (2 * 24, 96) and spec["l3.mix.right.v"].shape == (4 * 40, 96)
    assert spec["l3.mix.right.a2"].shape == (4 * 24, 12) and spec["l3.mix.right.g2"].shape == (4 * 40, 20)
    assert spec["l3.mix.left.q.norm"].shape == (6 * 40,) and spec["l4.mix.vmix"].shape == ()
    # the first layer that mixes values may or may not carry a constant; one that mixes nothing has none
    assert spec["l0.mix.vmix"].optional and not spec["l4.mix.vmix"].optional and "l2.mix.vmix" not in spec
    groups = [(g.n_layers, g.n_kv_heads, g.head_dim, g.value_dim, g.window) for g in m.cache_groups()]
    # (head sizes are filled up to one the tensor-core kernels take where that costs little)
    assert groups == [(2, 2, 32, 40, 27), (1, 1, 24, 16, 11), (1, 3, 40, 24, None)] or \
        groups == [(2, 2, *tensor_core_sizes(32, 40), 27), (1, 1, *tensor_core_sizes(24, 16), 11), (1, 3, *tensor_core_sizes(40, 24), None)]
    wide = Model.from_config(load_config(BIFATAR["W"]), torch.float32, "cpu")
    assert [b.mixer.names for b in wide.blocks] == [["left", "right", "mlp"], ["mix", "mlp"], ["mix"], ["mix", "mlp"], ["mix", "mlp"]]
    v = Model.from_config(load_config(BIFATAR["V"]), torch.float32, "cpu")
    assert [b.mixer.names for b in v.blocks] == [["mix"], ["left", "right"], ["mix", "mlp"], ["mix", "mlp"]]


def test_head_sizes_the_tensor_core_kernels_take():
    assert tensor_core_sizes(64, 64) == (64, 64) and tensor_core_sizes(128, 128) == (128, 128)
    assert tensor_core_sizes(64, 32) == (64, 64) and tensor_core_sizes(100, 128) == (128, 128)
    assert tensor_core_sizes(48, 80) == (48, 80) and tensor_core_sizes(20, 12) == (24, 16) and tensor_core_sizes(136, 128) == (136, 128)


def test_states_per_slot():
    m = Model.from_config(load_config(BIFATAR["U"]), torch.float32, "cpu")
    groups, states, runs = m._cache_layout()
    shapes = {s.name: tuple(s.shape) for s in states}
    assert shapes == {"run1.mix.state": (4, 20, 24), "run1.mix.ring": (4, 96 + 80), "run3.right.state": (4, 24, 40),
                      "run3.right.ring": (3, 2 * 2 * 24 + 4 * 40)}
    assert all(s.dtype == torch.float32 for s in states)
    one_tap = Model.from_config(load_config(BIFATAR["V"]), torch.float32, "cpu")
    assert not any("ring" in s.name for s in one_tap._cache_layout()[1])
    c = PagedCache(groups, states, num_blocks=8, max_slots=2, max_blocks_per_seq=4, block_size=4, dtype=torch.float32, device="cpu")
    a, b = c.admit(), c.admit()
    for st in c.states.values():
        st[a] += 3.0
        st[b] += 5.0
    c.release(a)
    assert c.admit() == a
    assert all(float(st[a].abs().max()) == 0.0 and float(st[b].min()) == 5.0 for st in c.states.values())


def test_branches_are_stacked_with_zeros_between():
    """The output matrix holds every branch's columns at a multiple of 8, zeros elsewhere, and a row of a multiple of 32; the
    stacked input matrix the branches' rows in order, biases where a branch has them."""
    raw = BIFATAR["W"]
    m = Model.from_config(load_config(raw), torch.float32, "cpu")
    tensors = W.random_tensors(m.tensor_specs(), 3, torch.float32)
    rt = Runtime(torch.device("cpu"), torch.float32, torch.zeros(1, dtype=torch.int32))
    par = m.blocks[0].mixer
    keep = {k: v.clone() for k, v in tensors.items()}
    par.bind(tensors, rt)
    assert par.fused and par.n_act % 32 == 0 and all(c % 8 == 0 for c in par.act_cols)
    used = torch.zeros(par.n_act, dtype=torch.bool)
    left, right, mlp = par.branches
    for b, c, n in zip(par.branches, par.act_cols, (3 * left.dvp, 3 * 9, 41)):
        used[c:c + n] = True
    assert bool((par.w_o[:, ~used] == 0).all()) and sorted(par.gaps) == sorted(
        (lo, hi) for lo, hi in par.gaps if not bool(used[lo:hi].any()))
    assert torch.equal(par.w_o[:, par.act_cols[1]:par.act_cols[1] + 27], keep["l0.mix.right.o"])
    assert torch.equal(par.w_o[:, par.act_cols[2]:par.act_cols[2] + 41], keep["l0.mlp.down"])
    assert torch.equal(par.w_in[par.in_cols[2]:], keep["l0.mlp.up"])
    assert float(par.b_in[par.in_cols[1]:].abs().max()) == 0.0 and float(par.b_in[:par.in_cols[1]].abs().max()) > 0


# ---------------------------------------------------------------- the plain mechanisms
def test_plain_norm_computes_no_mean_and_no_variance():
    w, b, alpha = torch.tensor([2.0, 1.0]).double(), torch.tensor([0.1, -1.0]).double(), torch.tensor(0.5).double()
    y = P.dyn_tanh(torch.tensor([[0.5, 100.0]]).double(), w, b, alpha)
    assert torch.allclose(y, torch.tensor([[2 * math.tanh(0.25) + 0.1, 0.0]]).double())


def test_plain_unit_vectors_and_norms():
    x = torch.tensor([[3.0, 4.0]]).double()
    assert torch.allclose(P.unit_vector(x), x / math.sqrt(25 + 1e-6), rtol=1e-14)
    assert torch.allclose(P.unit_rms(x, 0.5), x / math.sqrt(13.0), rtol=1e-14)
    y, z = torch.tensor([[1.0, 2.0, 3.0, 4.0]]).double(), torch.zeros(1, 4).double() + 50
    g = P.gated_part_norm(y, z, torch.ones(4).double(), 2, 1e-12)            # silu(50) = 50: every part by its own mean square
    assert torch.allclose(g, torch.tensor([[1, 2, 3, 4]]).double() / torch.tensor([[math.sqrt(2.5)] * 2 + [math.sqrt(12.5)] * 2]).double())


def test_plain_rotation_pairs_and_what_it_leaves():
    x = torch.zeros(2, 1, 8, dtype=torch.float64)
    x[1, 0, 0], x[1, 0, 5] = 1.0, 3.0
    y = P.rotate_half(x, 4, 10000.0)
    assert torch.allclose(y[1, 0], torch.tensor([math.cos(1), 0, math.sin(1), 0, 0, 3.0, 0, 0]).double())    # (0, 2) is a pair
    assert torch.equal(y[0], x[0])


def test_plain_short_conv_is_causal_and_ordered():
    u = torch.arange(1.0, 6.0, dtype=torch.float64)[:, None]
    w = torch.tensor([[100.0, 10.0, 1.0]], dtype=torch.float64)            # the last tap meets the newest value
    assert P.short_conv(u, w)[:, 0].tolist() == [1.0, 12.0, 123.0, 234.0, 345.0]
    assert P.short_conv(u, w, torch.tensor([0.5]).double())[:, 0].tolist() == [1.5, 12.5, 123.5, 234.5, 345.5]


def test_plain_state_space_recurrence_against_its_sum():
    torch.manual_seed(0)
    S, H, G, N, dv = 6, 4, 2, 3, 2
    x, B, C = torch.randn(S, H, dv).double(), torch.randn(S, G, N).double(), torch.randn(S, G, N).double()
    dt, A, D = torch.rand(S, H).double(), torch.randn(H).double(), torch.randn(H).double()
    y = P.ssd_recurrence(x, B, C, dt, A, D)
    for h in range(H):
        g = h // 2
        for t in range(S):
            want = D[h] * x[t, h]
            for j in range(t + 1):
                want = want + math.exp(-math.exp(A[h]) * float(dt[j + 1:t + 1, h].sum())) * dt[j, h] * (B[j, g] @ C[t, g]) * x[j, h]
            assert torch.allclose(y[t, h], want)


def test_plain_delta_rule_replaces_what_is_under_a_key():
    k = torch.zeros(4, 1, 3).double()
    k[0, 0, 0] = k[1, 0, 1] = k[2, 0, 0] = k[3, 0, 2] = 1.0
    v = torch.arange(1.0, 5.0).double()[:, None, None].expand(4, 1, 2).contiguous()
    q = torch.ones(4, 1, 3).double()
    one = torch.ones(4, 1).double()
    o = P.delta_recurrence(q, k, v, torch.ones(4, 1, 3).double(), one)
    assert o[:, 0, 0].tolist() == [1.0, 3.0, 5.0, 9.0]                       # 1; 1 + 2; 3 replaces 1; + 4
    half = P.delta_recurrence(q, k, v, torch.ones(4, 1, 3).double(), 0.5 * one)
    assert half[:, 0, 0].tolist() == [0.5, 1.5, 0.5 + 0.5 * (3 - 0.5) + 1.0, 0.5 + 0.5 * 2.5 + 1.0 + 2.0]
    g = torch.ones(4, 1, 3).double()
    g[2, 0, 1] = 0.0                                                         # token 2 forgets channel 1 before it writes
    assert P.delta_recurrence(q, k, v, g, one)[:, 0, 0].tolist() == [1.0, 3.0, 3.0, 7.0]


def test_plain_attention_window_cap_and_keyless_term():
    S = 6
    q, k = torch.zeros(S, 1, 2).double(), torch.zeros(S, 1, 2).double()
    v = torch.eye(S).double()[:, None, :]                                    # value j marks position j
    out = P.attend(q, k, v, 1.0, window=3)
    assert torch.allclose(out[5, 0], torch.tensor([0, 0, 0, 1, 1, 1.0]).double() / 3) and torch.allclose(out[1, 0, :2], torch.full((2,), 0.5).double())
    sunk = P.attend(q, k, v, 1.0, window=1, sink=torch.tensor([math.log(3.0)]).double())
    assert torch.allclose(torch.diagonal(sunk[:, 0]), torch.full((S,), 0.25).double())
    q2 = torch.tensor([[[1000.0, 0.0]]]).double().expand(2, 1, 2).contiguous()
    k2 = torch.tensor([[[1.0, 0.0]], [[-1.0, 0.0]]]).double()
    v2 = torch.tensor([[[1.0]], [[0.0]]]).double()
    out = P.attend(q2, k2, v2, 1.0, softcap=2.0)
    assert abs(float(out[1, 0, 0]) - math.exp(2) / (math.exp(2) + math.exp(-2))) < 1e-9


def test_plain_values_are_mixed_with_the_first_mixing_layers():
    """Three attention layers, the middle one not mixing: with one visible key per query the output of the last is its own
    and the first layer's values, and a change of the middle layer's v changes nothing of what is mixed."""
    torch.manual_seed(1)
    m = {"heads": 1, "kv_heads": 1, "dim": 2, "vdim": 2, "scale": 1.0, "mask": {"size": 1}, "v_mix": True}
    Wt = {f"l{i}.{n}": torch.randn(2, 2).double() for i in range(3) for n in "qkvo"}
    Wt.update({f"l{i}.vmix": torch.tensor(0.25).double() for i in range(3)}, **{f"l{i}.sink": torch.tensor([-1e9]).double() for i in range(3)})
    h, shared = torch.randn(3, 2).double(), {}
    P.attention_mixer(Wt, "l0", m, h, 1e-5, shared)
    P.attention_mixer(Wt, "l1", dict(m, v_mix=False), 2 * h, 1e-5, shared)
    out = P.attention_mixer(Wt, "l2", m, 3 * h, 1e-5, shared)
    want = (0.75 * (3 * h) @ Wt["l2.v"].t() + 0.25 * h @ Wt["l0.v"].t()) @ Wt["l2.o"].t()
    assert torch.allclose(out, want)


def test_random_model_folder_round_trip(tmp_path):
    folder = fd.write_random_model(tmp_path / "m", BIFATAR["W"], seed=3)
    assert load_config(folder).to_dict() == load_config(BIFATAR["W"]).to_dict()
    w = fd.weights.load_checkpoint(folder)
    assert w["l0.mix.right.a1"].shape == (7, 72) and w["l2.mix.in"].shape == (30 + 30 + 2 * 3 * 136 + 3, 72)
    logits = P.forward(BIFATAR["W"], w, [1, 2, 3, 4, 5])
    assert logits.shape == (5, 160) and bool(torch.isfinite(logits).all())
    nameless = copy.deepcopy(BIFATAR["W"])
    del nameless["layers"][0]["mixer"]["right"]["rank"]                      # a size only the checkpoint gives
    with pytest.raises(ValueError, match="only a checkpoint gives"):
        fd.write_random_model(tmp_path / "n", nameless, seed=3)
    m = Model.from_config(load_config(nameless), torch.float32, "cpu")
    W.check(m.tensor_specs(), w)
