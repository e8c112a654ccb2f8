"""Gulozen as a blueprint of parts.

A decoder whose norms (RMS norms over groups of neighbouring channels) sit on
what a sub-layer puts out, x + norm(f(x)), not on what it reads.  Every mixer
reads its input plus a short causal convolution of it over time; after every
layer the stream becomes a learned average of the embedding output and all
layers' results so far.  A layer's mixer is either linear attention with one
constant decay per head, silu on q, k and v, a norm over the concatenated heads
and a sigmoid gate, or attention over one cached latent per position with a
query latent, a rotated key part shared by the heads, a learned keyless term
per head in the softmax denominator and a sigmoid gate.  The feed-forward is a
mixture of silu-gated experts weighted by their plain softmax scores, or absent.
Tensor names: ``embed``, ``l<i>.canon1`` / ``.dwa`` / ``.norm1`` / ``.norm2`` /
``.mix.*`` / ``.mlp.*``, ``final.norm``, ``head``.
"""

from __future__ import annotations

from ..config.gulozen import GulozenConfig
from ..engine.blueprint import LayerSpec, ModelBlueprint, PartSpec, RunSpec
from ..registry import register_architecture

# The configuration gives no longest sequence: the rotation tables are built for what the first cache asks for.
NO_POSITION_LIMIT = 1 << 30


def gulozen_blueprint(cfg: GulozenConfig) -> ModelBlueprint:
    H, eps = cfg.width, cfg.norm_eps
    positions = {}

    def norm(name, optional=False):
        return PartSpec("norm", "grouped_rmsnorm", dict(size=H, eps=eps, groups=cfg.norm_groups, tensor=name,
                                                        optional=optional))

    layers = []
    for i, L in enumerate(cfg.layers):
        p, mc = f"l{i}", L.mixer
        if L.type == "lightning":
            mixer = PartSpec("mixer", "lightning_attention",
                             dict(hidden_size=H, n_heads=mc.heads, head_dim=mc.dim, v_head_dim=mc.vdim, decay=mc.decay,
                                  eps=eps), f"{p}.mix")
        else:
            rope = mc.rotation_key()
            positions.setdefault(rope, PartSpec("position", "rotary_scaled",
                                                dict(dims=mc.rot_dim, base=mc.rot_base, scaling=mc.rot_scaling,
                                                     max_positions=NO_POSITION_LIMIT)))
            mixer = PartSpec("mixer", "latent_attention",
                             dict(hidden_size=H, n_heads=mc.heads, head_dim=mc.dim, v_head_dim=mc.vdim, kv_rank=mc.kv_rank,
                                  scale=mc.scale, eps=eps, q_rank=mc.q_rank, rot_dim=mc.rot_dim, position=rope, sink=True,
                                  gate=True), f"{p}.mix")
        parts = dict(norm1=norm(f"{p}.norm1"), mixer=mixer,
                     input_conv=PartSpec("input_conv", "causal_conv", dict(channels=H, taps=cfg.taps, tensor=f"{p}.canon1")),
                     depth=PartSpec("depth_average", "learned_average",
                                    dict(index=i, n_layers=len(cfg.layers), tensor=f"{p}.dwa")))
        if L.mlp is not None:
            parts["norm2"] = norm(f"{p}.norm2")
            parts["feed_forward"] = PartSpec("feed_forward", "routed_experts",
                                             dict(hidden_size=H, n_experts=L.mlp.experts, top=L.mlp.top,
                                                  expert_ff=L.mlp.expert_ff, expert_act="silu_gated", correction=False,
                                                  weight_scale=1.0), f"{p}.mlp")
        else:
            # a layer without a feed-forward may or may not carry its second norm's weight; it never runs
            parts["norm2"] = norm(f"{p}.norm2", optional=True)
        layers.append(LayerSpec("postnorm", parts))
    return ModelBlueprint(
        hidden_size=H,
        vocab_size=cfg.vocab,
        embedding=PartSpec("embedding", "token_table", dict(vocab_size=cfg.vocab, hidden_size=H, tensor="embed",
                                                            scale=cfg.embedding_scale)),
        positions=positions,
        layers=layers,
        schedule=[RunSpec(i) for i in range(len(cfg.layers))],
        final_norm=norm("final.norm"),
        head=PartSpec("head", "linear_head", dict(vocab_size=cfg.vocab, hidden_size=H, tensor="head")),
        max_positions=NO_POSITION_LIMIT,
    )


register_architecture("Gulozen", GulozenConfig, gulozen_blueprint)
