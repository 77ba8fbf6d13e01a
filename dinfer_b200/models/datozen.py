"""Datozen as a list of parts.

The embedding is a token's row plus its position's.  A layer is parallel behind one RMS norm, ``h = norm1(x); x += mixer(h) +
ff(h)``, and ends with the layer's token input: a part of the token's row of a second table, gated by the stream, projected
back and normed before it is added (``parts/token_side.py``).  The mixer is attention over chunks of positions: grouped heads
with a norm of q and k per head, a rotation in halves of a head's first elements (its frequencies stretched by a ramp),
values that are cached turned by their position and turned back at the query, a learned sink and one sigmoid gate per head.
The feed-forward is dense with an xIELU and no gate matrix, a mixture of gated silu experts (softmax scores; the choice by
score plus correction, from the best groups; identity experts at the end of the list; the scores as weights, not
renormalized; a shared expert), or absent.  A run of layers may be passed through several times with the same weights, each
pass with a cache of its own.  The head is the embedding table.  Tensor names: ``embed``, ``pos``, ``side.embed``,
``l<i>.norm1``, ``l<i>.mix.*``, ``l<i>.mlp.*``, ``l<i>.side.*``, ``final.norm``.
"""
from __future__ import annotations

from ..config.model_config import DatozenConfig
from ..config.registry import register_architecture
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry


def _mixer(l, cfg: DatozenConfig) -> PartSpec:
    m = l.mixer
    rope = {"head_dim": m.dim, "rotary_dim": m.rot_dims, "theta": m.rot_base, "max_positions": cfg.max_positions, "style": "neox"}
    if m.scaling:
        rope["ramp"] = m.scaling.to_dict()
    return PartSpec("gqa_attention", {
        "num_heads": m.heads, "num_kv_heads": m.kv_heads, "head_dim": m.dim, "v_dim": m.vdim, "scale": m.scale,
        "eps": cfg.norm_eps, "qk_norm": True, "position": PartSpec("rope", rope), "window": m.chunk, "chunked": True,
        "value_turn": m.rot_base, "sink": "mix.sink", "gate_proj": "mix.g", "gate_per": "head", "q_proj": "mix.q",
        "k_proj": "mix.k", "v_proj": "mix.v", "o_proj": "mix.o", "q_norm": "mix.q.norm", "k_norm": "mix.k.norm"})


def _feed_forward(f) -> PartSpec:
    if f is None:
        return PartSpec("none")
    if f.kind == "dense":
        return PartSpec("plain_mlp", {"intermediate_size": f.ff, "activation": "xielu", "up_proj": "mlp.up",
                                      "down_proj": "mlp.down", "act": "mlp.act"})
    return PartSpec("moe", {
        "num_experts": f.experts, "identity": f.identity, "top_k": f.top, "groups": (f.groups, f.keep), "expert_size": f.ff,
        "shared_size": f.shared_ff, "activation": "silu", "gated": True, "scoring": "softmax", "renormalize": False,
        "router": "mlp.router", "correction": "mlp.correction", "expert_gate": "mlp.e{e}.gate", "expert_up": "mlp.e{e}.up",
        "expert_down": "mlp.e{e}.down", "shared_gate_up": "mlp.shared.gate", "shared_up": "mlp.shared.up",
        "shared_down": "mlp.shared.down"})


def datozen_spec(cfg: DatozenConfig) -> ModelSpec:
    def norm(name: str) -> PartSpec:
        return PartSpec("rmsnorm", {"size": cfg.width, "eps": cfg.norm_eps, "weight": name})

    n = len(cfg.layers)
    layers = tuple(
        LayerSpec(prefix=f"l{i}.", block="shared_norm_residual", mixer=_mixer(l, cfg), mixer_norm=norm("norm1"),
                  feed_forward=_feed_forward(l.mlp), feed_forward_norm=PartSpec("none"),
                  extras={"token_side": {"dim": cfg.side_dim, "index": i, "layers": n, "vocab_size": cfg.vocab,
                                         "eps": cfg.norm_eps, "table": "side.embed", "gate_proj": "side.gate",
                                         "out_proj": "side.proj", "norm": "side.norm"}})
        for i, l in enumerate(cfg.layers))
    return ModelSpec(
        architecture=cfg.architecture, hidden_size=cfg.width, vocab_size=cfg.vocab, max_positions=cfg.max_positions,
        embedding_tensor="embed", layers=layers, schedule=tuple(ScheduleEntry(i) for i in cfg.schedule()),
        final_norm=norm("final.norm"), lm_head_tensor="head", tie_word_embeddings=True, eos_token_ids=cfg.eos_token_ids,
        embedding=PartSpec("positioned_table", {"tensor": "embed", "vocab_size": cfg.vocab, "positions": "pos",
                                                "max_positions": cfg.max_positions}))


register_architecture("Datozen", DatozenConfig.from_dict, datozen_spec)
