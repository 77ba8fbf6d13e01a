"""Rorutar as a list of parts.

The embedding is a token's row times a constant.  A layer is pre-norm, ``x += mixer(norm1(x)); x += ff(norm2(x))``, with RMS
norms.  The mixer is two side by side, ``left_scale * left(h) + right_scale * right(h)``: on the left, attention over a window
and the sequence's first tokens (grouped heads, one norm over all of q and one over all of k, a rotation in halves with
linearly scaled positions, soft-capped scores, a sink of score 0); on the right, a state-space mixer with one decay per head
and token.  The feed-forward is a mixture of gated experts whose gate and up sides are clamped (sigmoid scores, the choice
from the groups with the best two scores, the chosen scores over their sum), or absent.  A run of layers may be passed
through several times with the same weights, each pass with a cache and a state of its own.  Tensor names: ``embed``,
``l<i>.norm1``, ``l<i>.norm2``, ``l<i>.mix.left.*``, ``l<i>.mix.right.*``, ``l<i>.mlp.*``, ``final.norm``, ``head``.
"""
from __future__ import annotations

from ..config.model_config import RorutarConfig
from ..config.registry import register_architecture
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry

GATE_ALPHA = 1.702          # the factor inside the experts' sigmoid


def _mixer(m, cfg: RorutarConfig) -> PartSpec:
    a, s = m.left, m.right
    left = {"num_heads": a.heads, "num_kv_heads": a.kv_heads, "head_dim": a.dim, "v_dim": a.vdim, "scale": a.scale,
            "eps": cfg.norm_eps, "qk_norm": True, "qk_norm_over": "all", "window": a.window, "keep_first": a.keep_first,
            "softcap": a.softcap, "sink": True, "q_proj": "mix.left.q", "k_proj": "mix.left.k", "v_proj": "mix.left.v",
            "o_proj": "mix.left.o", "q_norm": "mix.left.q.norm", "k_norm": "mix.left.k.norm",
            "position": PartSpec("rope", {"head_dim": a.dim, "rotary_dim": a.rot_dims, "theta": a.rot_base,
                                          "max_positions": cfg.max_positions, "style": "neox",
                                          "scaling_factor": a.rot_factor})}
    right = {"num_heads": s.heads, "value_dim": s.vdim, "state_dim": s.state, "groups": s.groups, "conv": s.conv,
             "norm_parts": s.norm_groups, "eps": cfg.norm_eps, "in_proj": "mix.right.in", "conv_weight": "mix.right.conv",
             "conv_bias": "mix.right.conv.b", "dt_bias": "mix.right.dt_bias", "A_log": "mix.right.A_log", "D": "mix.right.D",
             "norm": "mix.right.norm", "o_proj": "mix.right.o"}
    return PartSpec("parallel_mixers", {"left": PartSpec("gqa_attention", left), "right": PartSpec("state_space", right),
                                        "scales": (m.left_scale, m.right_scale)})


def _feed_forward(f) -> PartSpec:
    if f is None:
        return PartSpec("none")
    return PartSpec("moe", {
        "num_experts": f.experts, "top_k": f.top, "groups": (f.groups, f.keep), "group_rank": 2, "expert_size": f.ff,
        "activation": ("clamped_swish", f.limit, GATE_ALPHA), "gated": True, "scoring": "sigmoid", "renormalize": True,
        "router": "mlp.router", "expert_gate": "mlp.e{e}.gate", "expert_up": "mlp.e{e}.up", "expert_down": "mlp.e{e}.down"})


def rorutar_spec(cfg: RorutarConfig) -> ModelSpec:
    def norm(name: str, optional: bool = False) -> PartSpec:
        return PartSpec("rmsnorm", {"size": cfg.width, "eps": cfg.norm_eps, "weight": name, "optional": optional})

    layers = tuple(
        LayerSpec(prefix=f"l{i}.", block="prenorm_residual", mixer=_mixer(l.mixer, cfg), mixer_norm=norm("norm1"),
                  feed_forward=_feed_forward(l.mlp), feed_forward_norm=norm("norm2", optional=l.mlp is None))
        for i, l in enumerate(cfg.layers))
    return ModelSpec(
        architecture=cfg.architecture, hidden_size=cfg.width, vocab_size=cfg.vocab, max_positions=cfg.max_positions,
        embedding_tensor="embed", layers=layers, schedule=tuple(ScheduleEntry(i) for i in cfg.schedule()),
        final_norm=norm("final.norm"), lm_head_tensor="head", tie_word_embeddings=False, eos_token_ids=cfg.eos_token_ids,
        embedding_scale=cfg.embedding_scale)


register_architecture("Rorutar", RorutarConfig.from_dict, rorutar_spec)
