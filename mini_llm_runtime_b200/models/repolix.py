"""Repolix as a model plan: an embedding times a constant, pre-norm layers of three kinds in any order whose sub-layers' results join the
stream times a vector (the `streams` block with one copy of the stream), a plain head.  The mixers are differential attention behind short
convolutions (`differential_attention`: two attention maps a head over the same values, their weighted difference normed; a sliding
window, YaRN frequencies), the state-space duality mixer (`state_space`) and the gated delta rule with a decay per key channel
(`channel_delta`); the feed-forward is routed experts with a softmax over all of them, groups, identity experts and a shared expert.
This module only turns a `RepolixConfig` into data; the parts it names live in `parts/`.  Tensor names: `embed`,
`l<i>.norm1|norm2|ls1|ls2`, `l<i>.mix.*`, `l<i>.mlp.{router, correction, e<j>.*, shared.*}`, `final.norm`, `head`.
"""
from __future__ import annotations

from ..config.base import LayerSpec, ModelPlan, PartSpec, Run
from ..config.gelulix import ChannelDeltaConfig
from ..config.registry import register_architecture
from ..config.repolix import DifferentialConfig, RepolixConfig, StateSpaceConfig

SWISH_ALPHA = 1.702          # an expert's y = g * sigmoid(1.702 g) * (u + 1)
UP_OFFSET = 1.0


def repolix_plan(cfg: RepolixConfig) -> ModelPlan:
    width = cfg.width
    norm = lambda name: PartSpec("rmsnorm", {"width": width, "eps": cfg.norm_eps}, {"weight": name})
    positions, layers = {}, []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        m = layer.mixer
        named = lambda *roles: {role: f"{p}mix.{role}" for role in roles}
        common = {"hidden_size": width, "num_heads": m.heads, "value_dim": m.vdim, "conv": m.conv, "eps": cfg.norm_eps}
        convolved = {f"{role}_conv": f"{p}mix.{role}.conv" for role in ("q", "k", "v")}
        if isinstance(m, DifferentialConfig):
            position = None
            if m.rot is not None:
                position, s = f"rot{i}", m.rot.scaling
                positions[position] = PartSpec("rotary_frequencies", {
                    "base": m.rot.base, "dims": m.rot.dims,
                    "yarn": {"factor": s.factor, "original": s.original, "fast": s.fast, "slow": s.slow} if s is not None else None})
            mixer = PartSpec("differential_attention", {**common, "num_kv_heads": m.kv_heads, "head_dim": m.dim, "scale": m.scale,
                                                        "diff": m.diff, "window": m.window, "position": position},
                             {**named("q", "k", "v", "o", "lq1", "lk1", "lq2", "lk2"), **convolved})
        elif isinstance(m, StateSpaceConfig):
            mixer = PartSpec("state_space", {**common, "num_groups": m.groups, "state_dim": m.state, "norm_groups": m.norm_groups},
                             {**named("in", "conv", "dt_bias", "A_log", "D", "norm", "o"), "conv_bias": f"{p}mix.conv.b"})
        elif isinstance(m, ChannelDeltaConfig):
            mixer = PartSpec("channel_delta", {**common, "num_qk_heads": m.qk_heads, "head_dim": m.dim, "decay_rank": m.decay_rank,
                                               "gate_rank": m.gate_rank},
                             {**named("q", "k", "v", "b", "o", "A_log", "dt_bias", "norm", "a1", "a2", "g1", "g2"), **convolved})
        else:
            raise TypeError(type(m).__name__)
        norms, scales, ff = {"pre_mixer": norm(p + "norm1")}, {"scale1": p + "ls1"}, None
        if layer.mlp is not None:
            e = layer.mlp
            names = {"router": p + "mlp.router", "correction": p + "mlp.correction"}
            for j in range(e.experts):
                names.update({f"e{j}.{role}": f"{p}mlp.e{j}.{role}" for role in ("gate", "up", "down")})
            if e.shared is not None:
                names.update({f"shared.{role}": f"{p}mlp.shared.{role}" for role in ("gate", "up", "down")})
            ff = PartSpec("routed_experts", {"hidden_size": width, "intermediate_size": e.expert.ff, "experts": e.experts, "top": e.top,
                                             "groups": e.groups, "keep": e.keep, "identity": e.identity, "router": "softmax_scores",
                                             "activation": "swish", "alpha": SWISH_ALPHA, "up_offset": UP_OFFSET, "limit": e.expert.limit,
                                             "shared_intermediate_size": e.shared.ff if e.shared is not None else None,
                                             "shared_limit": e.shared.limit if e.shared is not None else None, "shared_gate": False}, names)
            norms["pre_feed_forward"] = norm(p + "norm2")
            scales["scale2"] = p + "ls2"
        block = PartSpec("streams", {"width": width, "streams": 1, "connected": False}, scales)
        layers.append(LayerSpec(block=block, mixer=mixer, feed_forward=ff, norms=norms))
    return ModelPlan(
        architecture=cfg.architecture, hidden_size=width, vocab_size=cfg.vocab_size, max_positions=cfg.max_position_embeddings,
        embedding=PartSpec("hashed_embedding", {"vocab_size": cfg.vocab_size, "width": width, "scale": cfg.embedding_scale}, {"weight": "embed"}),
        positions=positions, layers=tuple(layers), schedule=tuple(Run(i) for i in range(len(layers))),
        final_norm=PartSpec("streams_rmsnorm", {"width": width, "eps": cfg.norm_eps}, {"weight": "final.norm"}),
        lm_head=PartSpec("linear_head", {"vocab_size": cfg.vocab_size, "width": width}, {"weight": "head"}),
        eos_token_ids=cfg.eos_token_ids)


register_architecture("Repolix", RepolixConfig, repolix_plan)
