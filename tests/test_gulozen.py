"""Gulozen without a GPU: configuration, blueprint, weights' checks, the rotation tables, and the plain
implementation's mechanisms against closed forms."""

import math
import warnings

import pytest
import torch

import flashdecode_cuda_b200 as fd
from flashdecode_cuda_b200.config import ConfigError, load_config
from flashdecode_cuda_b200.config.gulozen import GulozenConfig
from flashdecode_cuda_b200.engine.model import Model
from flashdecode_cuda_b200.parts.normed_attention import _pad_split_heads
from flashdecode_cuda_b200.parts.rope import RotaryScaled
from flashdecode_cuda_b200.weights import WeightError, check
import gulozen_helpers as GH
from gulozen_helpers import GULOZEN, random_config
from plain import gulozen_plain as P


@pytest.mark.parametrize("name", sorted(GULOZEN))
def test_configuration_round_trip(name):
    cfg = load_config(GULOZEN[name])
    assert isinstance(cfg, GulozenConfig) and cfg.architecture == "Gulozen"
    assert load_config(cfg.to_dict()).to_dict() == cfg.to_dict()
    assert not cfg.unknown_keys and "Gulozen" in cfg.summary()


def test_keys_left_out_take_their_neutral_values():
    raw = GH.model(50, 32, 1e-5, [GH.latent(2, 16, 4, 16, 8, 8, 0.25), GH.lightning(2, 8, 8)])
    del raw["layers"][0]["mixer"]["vdim"], raw["layers"][0]["mixer"]["rot"]["dims"], raw["layers"][1]["mixer"]["vdim"]
    cfg = load_config(raw)
    m = cfg.layers[0].mixer
    assert (m.vdim, m.rot_dim, m.rot_scaling, cfg.layers[1].mixer.vdim) == (16, 4, None, 8)
    assert (cfg.embedding_scale, cfg.norm_groups, cfg.taps) == (1.0, 1, 1)
    assert cfg.layers[0].mlp is None


@pytest.mark.parametrize("edit,text", [
    (lambda c: c.pop("width"), "misses 'width'"),
    (lambda c: c["norm"].pop("eps"), "misses 'eps'"),
    (lambda c: c["norm"].update(groups=5), "equal groups"),
    (lambda c: c.update(canon={"taps": 0}), "taps must be positive"),
    (lambda c: c["layers"][0].update(type="conv"), "mixers are"),
    (lambda c: c["layers"][0]["mixer"].update(rot_dim=6), "rot.dims the same"),
    (lambda c: c["layers"][0]["mixer"].update(rot_dim=3), "must be even"),
    (lambda c: c["layers"][0]["mixer"].pop("q_rank"), "misses 'q_rank'"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(scaling={"factor": 2.0}), "misses 'original'"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=9), "top <= experts"),
    (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "feed-forwards are"),
    (lambda c: c["layers"][1]["mixer"].update(decay=[0.5]), "1 numbers for 2 heads"),
])
def test_configuration_errors_name_their_place(edit, text):
    raw = GH.model(50, 32, 1e-5, [GH.latent(2, 16, 4, 16, 8, 8, 0.25, mlp=GH.moe(8, 2, 8)), GH.lightning(2, 8, 8)], 2, 3)
    edit(raw)
    with pytest.raises(ConfigError, match=text):
        load_config(raw)


def test_unknown_keys_warn_and_change_nothing():
    raw = GH.model(50, 32, 1e-5, [GH.lightning(2, 8, 8)])
    raw["layers"][0]["mixer"]["surprise"] = 1
    with warnings.catch_warnings(record=True) as w:
        warnings.simplefilter("always")
        cfg = load_config(raw)
    assert cfg.unknown_keys == ["layers[0].mixer.surprise"] and len(w) == 1


@pytest.mark.parametrize("name", sorted(GULOZEN))
def test_blueprint_tensors_pages_and_states(name):
    cfg = load_config(GULOZEN[name])
    mdl = Model.from_config(cfg, torch.float32, "cpu")
    shapes = {s.name: tuple(s.shape) for s in mdl.tensor_specs()}
    optional = {s.name for s in mdl.tensor_specs() if s.optional}
    assert {"embed", "final.norm", "head"} <= set(shapes)
    for i, L in enumerate(cfg.layers):
        p, m = f"l{i}", L.mixer
        assert shapes[f"{p}.canon1"] == (cfg.width, cfg.taps) and shapes[f"{p}.dwa"] == (i + 2,)
        assert (f"{p}.norm2" in optional) == (L.mlp is None)
        if L.type == "lightning":
            assert shapes[f"{p}.mix.norm"] == (m.heads * m.vdim,)
        else:
            assert shapes[f"{p}.mix.uq"] == (m.heads * (m.dim + m.rot_dim), m.q_rank)
            assert shapes[f"{p}.mix.dkv"] == (m.kv_rank + m.rot_dim, cfg.width) and shapes[f"{p}.mix.sink"] == (m.heads,)
    # one latent row per position and latent layer, nothing else; a matrix state per lightning layer; the convolution's
    # earlier inputs per layer
    groups, states, per_run = mdl._layout
    assert sum(g.n_layers for g in groups) == sum(L.type == "latent_attention" for L in cfg.layers)
    assert all(g.keys_only and g.n_kv_heads == 1 for g in groups)
    n_conv = len(cfg.layers) if cfg.taps > 1 else 0
    assert len(states) == n_conv + sum(L.type == "lightning" for L in cfg.layers)
    for s in states:
        assert s.dtype == torch.float32
        if s.name.endswith("input_conv"):
            assert s.shape == (cfg.taps - 1, cfg.width)


def test_a_wrong_checkpoint_is_reported_in_one_error():
    cfg = load_config(GULOZEN["A"])
    mdl = Model.from_config(cfg, torch.float32, "cpu")
    W = fd.random_weights(mdl, 1)
    check(mdl.tensor_specs(), W)
    del W["l1.mix.norm"]
    W["l2.dwa"] = torch.zeros(3)
    W["l0.extra"] = torch.zeros(1)
    with pytest.raises(WeightError) as e:
        check(mdl.tensor_specs(), W)
    assert all(t in str(e.value) for t in ("l1.mix.norm", "l2.dwa", "l0.extra"))


def test_head_parts_are_filled_up_apart():
    w = torch.arange(2 * 5 * 3, dtype=torch.float32).view(10, 3)
    out = _pad_split_heads(w, 2, (3, 4), (2, 4)).view(2, 8, 3)
    rows = w.view(2, 5, 3)
    assert torch.equal(out[:, :3], rows[:, :3]) and torch.equal(out[:, 4:6], rows[:, 3:])
    assert float(out[:, 3].abs().max()) == 0.0 and float(out[:, 6:].abs().max()) == 0.0


@pytest.mark.parametrize("dims,base,scaling", [(16, 10000.0, None), (48, 1e6, (8.0, 1024, 32.0, 1.0)), (8, 100.0, (4.0, 64, 8.0, 2.0)),
                                               (64, 30000.0, (6.0, 4096, 24.0, 1.5)), (2, 50.0, (2.0, 64, 1.0, 1.0))])
def test_rotation_tables_follow_the_stretched_frequencies(dims, base, scaling):
    sc = None if scaling is None else dict(zip(("factor", "original", "fast", "slow"), scaling))
    f, mag = P.rot_frequencies(dims, base, sc)
    for i, fi in enumerate(f.tolist()):
        f0 = base ** (-2.0 * i / dims)
        assert f0 / (sc["factor"] if sc else 1.0) - 1e-15 <= fi <= f0 + 1e-15
    if sc:
        assert mag == pytest.approx(0.1 * math.log(sc["factor"]) + 1.0)
    pos = RotaryScaled(dims, base, sc)
    got, gm = pos.frequencies()
    assert gm == pytest.approx(mag) and torch.allclose(got, f, rtol=1e-12, atol=0)


# ---------------------------------------------------------------- the plain implementation against closed forms
def test_plain_grouped_norm_norms_each_group_alone():
    torch.manual_seed(0)
    x, w = torch.randn(3, 12).double(), torch.randn(12).double()
    y = P.grouped_rms_norm(x, w, 0.0, 3) / w
    assert torch.allclose(y.view(3, 3, 4).pow(2).mean(-1), torch.ones(3, 3).double())
    one = P.grouped_rms_norm(x, w, 1e-5, 1)
    assert torch.allclose(one, P.rms_norm(x, w, 1e-5))
    x2 = x.clone()
    x2[:, 4:8] *= 100.0
    a, b = P.grouped_rms_norm(x, w, 1e-9, 3), P.grouped_rms_norm(x2, w, 1e-9, 3)
    assert torch.allclose(a, b, atol=1e-6)                   # a group's scale says nothing about the others


def test_plain_convolution_is_causal_and_starts_from_zeros():
    u = torch.arange(10, dtype=torch.float64).reshape(5, 2)
    w = torch.tensor([[1.0, 10.0, 100.0], [0.0, 0.0, 1.0]], dtype=torch.float64)
    y = P.causal_conv(u, w)
    assert y[:, 1].tolist() == u[:, 1].tolist()
    assert y[:, 0].tolist() == [0.0, 200.0, 420.0, 642.0, 864.0]


def test_plain_recurrence_against_its_unrolled_sum():
    torch.manual_seed(0)
    S, H, d, dv = 9, 2, 3, 4
    q, k, v = torch.randn(S, H, d).double(), torch.randn(S, H, d).double(), torch.randn(S, H, dv).double()
    g = torch.tensor([0.5, 0.9]).double()
    o, _ = P.decay_recurrence(q, k, v, g)
    t = S - 1
    want = sum((g ** (t - j))[:, None] * (q[t] * k[j]).sum(-1, keepdim=True) * v[j] for j in range(S))
    assert torch.allclose(o[t], want, atol=1e-12)
    _, state = P.decay_recurrence(q[:4], k[:4], v[:4], g)
    rest, _ = P.decay_recurrence(q[4:], k[4:], v[4:], g, state)
    assert torch.allclose(rest, o[4:], atol=1e-12)


def test_plain_attention_with_a_keyless_term():
    S, H, d = 6, 2, 4
    v = torch.randn(S, H, d).double()
    z = torch.zeros(S, H, d).double()
    sink = torch.tensor([0.0, math.log(3.0)]).double()
    o = P.sink_attention(z, z, v, 1.0, sink)
    for i in range(S):                                       # all scores zero: weights 1 / (keys + exp(sink))
        assert torch.allclose(o[i, 0], v[:i + 1, 0].sum(0) / (i + 2.0)) and torch.allclose(o[i, 1], v[:i + 1, 1].sum(0) / (i + 4.0))


def test_plain_routing_weights_are_the_scores_themselves():
    h = torch.eye(3, dtype=torch.float64)[:1]
    router = torch.tensor([[1.0, 0, 0], [3.0, 0, 0], [2.0, 0, 0]], dtype=torch.float64)
    ids, w = P.route(h, router, 2)
    s = torch.softmax(torch.tensor([1.0, 3.0, 2.0], dtype=torch.float64), 0)
    assert ids[0].tolist() == [1, 2] and torch.allclose(w[0], s[[1, 2]]) and float(w.sum()) < 1.0


def test_latent_basis_identity():
    """(q . U c) = (U^T q) . c and sum_j p_j (V c_j) = V sum_j p_j c_j: what lets attention run on the cached latents."""
    torch.manual_seed(2)
    U, V, q, c = torch.randn(5, 7).double(), torch.randn(4, 7).double(), torch.randn(5).double(), torch.randn(6, 7).double()
    p = torch.softmax(torch.randn(6).double(), 0)
    assert torch.allclose((c @ U.T) @ q, c @ (U.T @ q)) and torch.allclose(p @ (c @ V.T), V @ (p @ c))


@pytest.mark.parametrize("seed", range(8))
def test_drawn_configurations_are_valid_and_the_plain_model_runs(seed):
    raw = random_config(seed)
    cfg = load_config(raw)
    mdl = Model.from_config(cfg, torch.float32, "cpu")
    W = fd.random_weights(mdl, seed)
    check(mdl.tensor_specs(), W)
    logits, layers = P.forward(raw, W, [1, 2, 3, 4, 5], return_layers=True)
    assert logits.shape == (5, cfg.vocab) and layers.shape[0] == len(cfg.layers) and bool(torch.isfinite(logits).all())
    # prefix property: what a position's logits are does not depend on what follows
    assert torch.allclose(P.forward(raw, W, [1, 2, 3])[2], logits[2], atol=1e-9)
