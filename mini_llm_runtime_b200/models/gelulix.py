"""Gelulix as a model plan: layers of three kinds in any order, whose norm stands behind the SUM of the scaled residual stream and a
sub-layer's result (`x = norm(a x + f(x))`, the `sum_norm` block; the sub-layers read the stream as it is, `identity` norms in front).
The mixers are gated linear attention with a decay per key channel (`gated_linear`), latent attention with a rotated key part under
YaRN frequencies and a learned sink (`latent_attention`), and the gated delta rule behind short convolutions with a decay per key
channel (`channel_delta`); a layer ends with a gated feed-forward with biases, or without one.  This module only turns a
`GelulixConfig` into data; the parts it names live in `parts/`.  Tensor names: `embed`, `l<i>.norm1|norm2`, `l<i>.mix.*`,
`l<i>.mlp.{gate,up,down}[.b]`, `final.norm`, `head`.
"""
from __future__ import annotations

from ..config.base import LayerSpec, ModelPlan, PartSpec, Run
from ..config.gelulix import ChannelDeltaConfig, GatedLinearConfig, GelulixConfig, LatentConfig
from ..config.registry import register_architecture


def gelulix_plan(cfg: GelulixConfig) -> ModelPlan:
    width = cfg.width
    norm = lambda name: PartSpec("group_rmsnorm", {"width": width, "groups": 1, "eps": cfg.norm_eps}, {"weight": name})
    plain = PartSpec("identity", {"width": width})
    block = PartSpec("sum_norm", {"alpha": cfg.alpha})
    positions, layers = {}, []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        m = layer.mixer
        named = lambda *roles: {role: f"{p}mix.{role}" for role in roles}
        common = {"hidden_size": width, "num_heads": m.heads, "head_dim": m.dim, "value_dim": m.vdim, "eps": cfg.norm_eps}
        if isinstance(m, GatedLinearConfig):
            mixer = PartSpec("gated_linear", {**common, "tau": m.tau, "decay_rank": m.decay_rank},
                             {**named("q", "k", "v", "g", "o", "a1", "a2", "norm"), "a2_bias": f"{p}mix.a2.b"})
        elif isinstance(m, LatentConfig):
            position = f"rot{i}"
            s = m.rot.scaling
            positions[position] = PartSpec("rotary_frequencies", {
                "base": m.rot.base, "dims": m.rot.dims, "interleaved": True,
                "yarn": {"factor": s.factor, "original": s.original, "fast": s.fast, "slow": s.slow} if s is not None else None})
            mixer = PartSpec("latent_attention", {**common, "rank": m.kv_rank, "scale": m.scale, "own_latent": True, "rot_dim": m.rot_dim,
                                                  "position": position, "sink": "learned"},
                             {**named("q", "dkv", "uk", "uv", "o", "sink"), "dkv_norm": f"{p}mix.dkv.norm"})
        elif isinstance(m, ChannelDeltaConfig):
            names = named("q", "k", "v", "b", "o", "A_log", "dt_bias", "norm", "a1", "a2", "g1", "g2")
            names.update({f"{role}_conv": f"{p}mix.{role}.conv" for role in ("q", "k", "v")})
            mixer = PartSpec("channel_delta", {**common, "num_qk_heads": m.qk_heads, "conv": m.conv, "decay_rank": m.decay_rank,
                                               "gate_rank": m.gate_rank}, names)
        else:
            raise TypeError(type(m).__name__)
        norms = {"pre_mixer": plain, "post_mixer": norm(p + "norm1")}
        ff = None
        if layer.ff is not None:
            names = {role: f"{p}mlp.{role}" for role in ("gate", "up", "down")}
            names.update({f"{role}_bias": f"{p}mlp.{role}.b" for role in ("gate", "up", "down")})
            ff = PartSpec("gated_bias", {"hidden_size": width, "intermediate_size": layer.ff, "activation": "silu"}, names)
            norms.update({"pre_feed_forward": plain, "post_feed_forward": norm(p + "norm2")})
        layers.append(LayerSpec(block=block, mixer=mixer, feed_forward=ff, norms=norms))
    return ModelPlan(
        architecture=cfg.architecture, hidden_size=width, vocab_size=cfg.vocab_size, max_positions=cfg.max_position_embeddings,
        embedding=PartSpec("token_embedding", {"vocab_size": cfg.vocab_size, "width": width}, {"weight": "embed"}),
        positions=positions, layers=tuple(layers), schedule=tuple(Run(i) for i in range(len(layers))), final_norm=norm("final.norm"),
        lm_head=PartSpec("linear_head", {"vocab_size": cfg.vocab_size, "width": width}, {"weight": "head"}),
        eos_token_ids=cfg.eos_token_ids)


register_architecture("Gelulix", GelulixConfig, gelulix_plan)
