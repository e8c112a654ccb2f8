"""Bifatar as a blueprint of parts.

A decoder of parallel layers: one Dynamic Tanh norm (tanh(alpha x) * w + b: no
mean, no variance) per layer, whose output the mixer and the feed-forward both
read, x += mixer(h) + ff(h).  A layer's mixer is a Mamba-2 state-space mixer;
or softmax attention (biased projections, q and k normed over the whole
projection, rotated) beside a gated delta rule with a decay per key channel,
their outputs added with fixed weights; or windowed softmax attention with
normed heads after the rotation, capped scores, a learned keyless term per head
and values mixed with those of the first layer that mixes values.  The
feed-forward is down(relu(up h)^2), or absent.  All of a layer's branches, the
feed-forward among them, share one input product and one output product.
Tensor names: ``embed``, ``l<i>.norm1`` (+ ``.b``, ``.alpha``), ``l<i>.mix.*``
(``.left.*`` and ``.right.*`` in a parallel layer), ``l<i>.mlp.*``,
``final.norm``, ``head``.
"""

from __future__ import annotations

from ..config.bifatar import BifatarConfig
from ..engine.blueprint import LayerSpec, ModelBlueprint, PartSpec, RunSpec
from ..registry import register_architecture

# The configuration gives no longest sequence: the rotation tables are built for what the first cache asks for.
NO_POSITION_LIMIT = 1 << 30


def bifatar_blueprint(cfg: BifatarConfig) -> ModelBlueprint:
    H, eps = cfg.width, cfg.norm_eps
    positions = {}

    def rotation(rot):
        if rot is None:
            return dict(position=None, rot_dims=0)
        positions.setdefault(rot.key(), PartSpec("position", "rotary_scaled",
                                                 dict(dims=rot.dims, base=rot.base, max_positions=NO_POSITION_LIMIT)))
        return dict(position=rot.key(), rot_dims=rot.dims)

    def attention(a, prefix, **options):
        return PartSpec("mixer", "qk_normed_attention",
                        dict(hidden_size=H, n_heads=a.heads, n_kv_heads=a.kv_heads, head_dim=a.dim, v_head_dim=a.vdim,
                             scale=a.scale, eps=eps, **rotation(a.rot), **options), prefix)

    layers = []
    values_shared = False                       # whether an earlier layer has left its values for the others
    for i, L in enumerate(cfg.layers):
        p, m = f"l{i}", L.mixer
        if L.type == "mamba2":
            branches = [PartSpec("mixer", "mamba2",
                                 dict(hidden_size=H, n_heads=m.heads, v_head_dim=m.vdim, state_size=m.state, n_groups=m.groups,
                                      norm_groups=m.norm_groups, taps=m.conv, eps=eps), f"{p}.mix")]
            names, scales = ["mix"], [1.0]
        elif L.type == "parallel":
            r = m.right
            branches = [attention(m.left, f"{p}.mix.left", bias=True),
                        PartSpec("mixer", "gated_delta_rule",
                                 dict(hidden_size=H, n_heads=r.heads, n_qk_heads=r.kv_heads, head_dim=r.dim, v_head_dim=r.vdim,
                                      taps=r.conv, eps=eps, decay_rank=r.rank, gate_rank=r.gate_rank), f"{p}.mix.right")]
            names, scales = ["left", "right"], [m.left_scale, m.right_scale]
        else:
            mix = None
            if m.v_mix:
                mix, values_shared = ("mix" if values_shared else "source"), True
            branches = [attention(m, f"{p}.mix", window=m.window, qk_norm=False, head_norm=True, softcap=m.softcap, sink=True,
                                  value_mix=mix)]
            names, scales = ["mix"], [1.0]
        if L.mlp is not None:
            branches.append(PartSpec("feed_forward", "dense_act",
                                     dict(hidden_size=H, intermediate_size=L.mlp.ff, activation="relu2"), f"{p}.mlp"))
            names, scales = names + ["mlp"], scales + [1.0]
        layers.append(LayerSpec("prenorm", dict(
            norm1=PartSpec("norm", "dyn_tanh", dict(size=H, tensor=f"{p}.norm1")),
            mixer=PartSpec("mixer", "parallel", dict(branches=branches, names=names, scales=scales, hidden_size=H), p))))
    return ModelBlueprint(
        hidden_size=H,
        vocab_size=cfg.vocab,
        embedding=PartSpec("embedding", "token_table", dict(vocab_size=cfg.vocab, hidden_size=H, tensor="embed")),
        positions=positions,
        layers=layers,
        schedule=[RunSpec(i) for i in range(len(layers))],
        final_norm=PartSpec("norm", "dyn_tanh", dict(size=H, tensor="final.norm")),
        head=PartSpec("head", "linear_head", dict(vocab_size=cfg.vocab, hidden_size=H, tensor="head")),
        max_positions=NO_POSITION_LIMIT,
    )


register_architecture("Bifatar", BifatarConfig, bifatar_blueprint)
