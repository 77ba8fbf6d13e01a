"""Rorutar without a device: the configuration reader and its refusals, the declared tensors, what a layer keeps, kept first
pages in the cache managers, and the plain implementation against itself (pieces against whole, each mechanism against a
second way of writing it)."""
import copy
import math
import random

import pytest
import torch

import helpers as H
import plain_rorutar as P
import rorutar_cases as C
from dinfer_b200.cache.manager import CacheManager, GroupSpec
from dinfer_b200.config.model_config import ConfigError, RorutarConfig
from dinfer_b200.config.registry import resolve_architecture

F64 = torch.float64


def test_config_round_trip_and_spec():
    for name, d in C.CONFIGS.items():
        arch = resolve_architecture(d)
        cfg = arch.parse_config(d)
        assert isinstance(cfg, RorutarConfig) and cfg == RorutarConfig.from_dict(cfg.to_dict())
        spec = arch.build_spec(cfg)
        spec.check()
        assert not spec.tie_word_embeddings and spec.embedding_scale == d["embedding"]["scale"]
        assert all(l.block == "prenorm_residual" and l.mixer.kind == "parallel_mixers" for l in spec.layers)
        assert [l.feed_forward.kind for l in spec.layers] == ["none" if l["mlp"] is None else "moe" for l in d["layers"]]
        assert [e.layer for e in spec.schedule] == P.schedule(d) and all(e.cache_from is None for e in spec.schedule)
        for l, raw in zip(spec.layers, d["layers"]):
            m = raw["mixer"]
            assert l.mixer.get("scales") == (m["left_scale"], m["right_scale"])
            assert l.mixer.get("left").get("keep_first") == m["left"].get("mask", {}).get("keep_first", 0)
            assert l.mixer.get("left").get("window") == m["left"].get("mask", {}).get("size")


def test_config_defaults():
    """Sections a layer or the model may leave out: scaled positions, the mask, the soft cap, groups, the loop, scales."""
    d = copy.deepcopy(C.RORUTAR_A)
    left, f = d["layers"][0]["mixer"]["left"], d["layers"][0]["mlp"]
    del d["loop"], d["embedding"], left["rot"]["scaling"], left["mask"], left["softcap"], f["router"]["groups"], d["layers"][0]["mixer"]["left_scale"]
    cfg = RorutarConfig.from_dict(d)
    l = cfg.layers[0]
    assert cfg.loop is None and cfg.embedding_scale == 1.0 and cfg.schedule() == (0, 1, 2, 3)
    assert (l.mixer.left.rot_factor, l.mixer.left.window, l.mixer.left.keep_first, l.mixer.left.softcap) == (1.0, None, 0, 0.0)
    assert (l.mlp.groups, l.mlp.keep, l.mixer.left_scale) == (1, 1, 1.0)


@pytest.mark.parametrize("path, value", [
    (("norm", "eps"), 0.0), (("layers", 0, "type"), "retention"), (("layers", 0, "mixer", "left"), None),
    (("layers", 0, "mixer", "right"), None), (("layers", 0, "mixer", "left", "kv_heads"), 3),
    (("layers", 0, "mixer", "left", "heads"), 0), (("layers", 0, "mixer", "left", "scale"), None),
    (("layers", 0, "mixer", "left", "scale"), 0.0), (("layers", 0, "mixer", "left", "mask", "size"), 0),
    (("layers", 0, "mixer", "left", "mask", "keep_first"), -1), (("layers", 0, "mixer", "left", "softcap"), -2.0),
    (("layers", 0, "mixer", "left", "rot", "dims"), 14), (("layers", 0, "mixer", "left", "rot", "dims"), 5),
    (("layers", 0, "mixer", "left", "rot", "scaling", "factor"), 0.0), (("layers", 0, "mixer", "right", "groups"), 4),
    (("layers", 0, "mixer", "right", "norm_groups"), 7), (("layers", 0, "mixer", "right", "conv"), 0),
    (("layers", 0, "mixer", "right", "state"), None), (("layers", 0, "mlp", "kind"), "dense"),
    (("layers", 0, "mlp", "expert", "limit"), None), (("layers", 0, "mlp", "expert", "limit"), 0.0),
    (("layers", 0, "mlp", "router", "groups", "count"), 4), (("layers", 0, "mlp", "router", "groups", "keep"), 4),
    (("layers", 0, "mlp", "router", "top"), 5), (("loop", "stop"), 5), (("loop", "times"), 0), (("loop", "start"), 3),
    (("vocab",), None), (("width",), 0), (("layers",), [])])
def test_config_refusals(path, value):
    d = copy.deepcopy(C.RORUTAR_A)
    at = d
    for k in path[:-1]:
        at = at[k]
    if value is None:
        del at[path[-1]]
    else:
        at[path[-1]] = value
    with pytest.raises(ConfigError):
        RorutarConfig.from_dict(d)


def test_declared_tensors():
    from dinfer_b200.weights.random_init import model_declarations
    decls = {x.name: tuple(x.shape) for x in model_declarations(C.RORUTAR_A)}
    w = 64
    assert decls["embed"] == (300, w) and decls["head"] == (300, w) and decls["final.norm"] == (w,)
    assert decls["l0.norm1"] == (w,) and decls["l0.norm2"] == (w,)
    assert decls["l0.mix.left.q"] == (48, w) and decls["l0.mix.left.k"] == (24, w) and decls["l0.mix.left.v"] == (40, w)
    assert decls["l0.mix.left.q.norm"] == (48,) and decls["l0.mix.left.k.norm"] == (24,) and decls["l0.mix.left.o"] == (w, 80)
    inner, channels = 60, 60 + 2 * 2 * 14
    assert decls["l0.mix.right.in"] == (inner + channels + 6, w) and decls["l0.mix.right.conv"] == (channels, 4)
    assert decls["l0.mix.right.conv.b"] == (channels,) and decls["l0.mix.right.norm"] == (inner,) and decls["l0.mix.right.o"] == (w, inner)
    assert all(decls["l0.mix.right." + n] == (6,) for n in ("dt_bias", "A_log", "D"))
    assert decls["l0.mlp.router"] == (6, w) and decls["l0.mlp.e5.gate"] == (24, w) and decls["l0.mlp.e5.down"] == (w, 24)
    assert "l2.mlp.router" not in decls and "l0.mlp.e6.up" not in decls


def test_what_a_layer_keeps():
    from dinfer_b200.parts.base import BuildEnv, split_needs
    from dinfer_b200.models.decoder import DecoderModel
    arch = resolve_architecture(C.RORUTAR_A)
    m = DecoderModel(arch.build_spec(arch.parse_config(C.RORUTAR_A)), BuildEnv(torch.device("cpu"), torch.float32, 64, 128))
    needs = [split_needs(n) for n in m.cache_needs()]
    assert len(needs) == 6 and m.graph_capturable()
    kv, st = needs[0]
    assert (kv.num_kv_heads, kv.head_dim, kv.window, kv.keep_first) == (2, 20, 7, 3)
    assert st.dtype == torch.float32 and st.shape == ((6 * 14 * 10 + 3 * (60 + 56) + 3) // 4 * 4,)
    assert needs[5][0].window is None and needs[5][0].keep_first == 0
    assert needs[1] == needs[3] and needs[2] == needs[4]     # the loop's passes each keep their own


def test_open_ends_of_other_mixers():
    """A weighted sum of two mixers needs both to have open ends; attention with gates or biases has none."""
    import dinfer_b200.models.decoder  # noqa: F401
    from dinfer_b200.parts.base import MIXERS, BuildEnv
    from dinfer_b200.parts.spec import PartSpec
    env = BuildEnv(torch.device("cpu"), torch.float32, 32, 64)
    att = {"num_heads": 2, "num_kv_heads": 1, "head_dim": 8}
    assert MIXERS.get("gqa_attention")(att, env, "").open_ends() == (32, 16)
    assert MIXERS.get("gqa_attention")(dict(att, gate_proj="g"), env, "").open_ends() is None
    assert MIXERS.get("gqa_attention")(dict(att, bias=True), env, "").open_ends() is None
    assert MIXERS.get("gqa_attention")(dict(att, qk_norm=True), env, "").open_ends() is None
    with pytest.raises(ValueError):
        MIXERS.get("parallel_mixers")({"left": PartSpec("gqa_attention", dict(att, bias=True)), "right": PartSpec("gqa_attention", att),
                                       "scales": (1.0, 1.0)}, env, "")
    with pytest.raises(ValueError):
        MIXERS.get("gqa_attention")(dict(att, qk_norm=True, qk_norm_over="all", gate_proj="g"), env, "")


def test_gate_constants():
    from dinfer_b200.kernels.lib import KernelError
    from dinfer_b200.kernels.ops import gate_constants
    assert gate_constants("silu") == ("silu", 0.0, 0.0) and gate_constants(("clamped_swish", 2, 1.5)) == ("clamped_swish", 2.0, 1.5)
    for bad in ("clamped_swish", ("silu", 1.0, 1.0), ("clamped_swish", 0.0, 1.0)):
        with pytest.raises(KernelError):
            gate_constants(bad)


@pytest.mark.parametrize("native", [False, True])
@pytest.mark.parametrize("keep, kept_pages", [(0, 0), (1, 1), (4, 1), (5, 2), (11, 3)])
def test_kept_pages_stay(native, keep, kept_pages):
    """The pages that hold a request's kept first tokens stay while the window passes, the others go back."""
    from dinfer_b200.cache.native import NativeCacheManager
    m = (NativeCacheManager if native else CacheManager)([GroupSpec(window=6, keep_first=keep)], 4, [20], 2)
    assert m.allocate("a", 40)
    m.advance("a", 40)                                       # the next query, 40, sees 35 .. 40 and the kept tokens
    assert [i for i, b in enumerate(m.block_table("a", 0)) if b >= 0] == list(range(kept_pages)) + [8, 9]
    m.check_invariants()
    m.free("a")
    assert m.num_free_blocks(0) == 20


def _weights(cfg, seed=3):
    from dinfer_b200.weights.random_init import model_declarations, random_tensor
    return {d.name: C.shape_weight(d.name, random_tensor(d, seed, 0.1, 0.3, torch.float32)).double() for d in model_declarations(cfg)}


@pytest.mark.parametrize("name", ["A", "C", "D"])
def test_plain_in_pieces_is_plain_whole(name):
    cfg = C.CONFIGS[name]
    W = _weights(cfg)
    ids = H.random_tokens(random.Random(1), 60, cfg["vocab"])
    whole = P.forward(cfg, W, ids, P.new_state(cfg))
    state, parts, at = P.new_state(cfg), [], 0
    for n in (1, 2, 30, 1, 26):
        parts.append(P.forward(cfg, W, ids[at:at + n], state))
        at += n
    assert torch.allclose(torch.cat(parts), whole, atol=1e-9, rtol=1e-9)


def test_plain_visible_keys():
    assert P.visible(9, {"size": 3, "keep_first": 2}) == [0, 1, 7, 8, 9]
    assert P.visible(3, {"size": 3, "keep_first": 2}) == [0, 1, 2, 3] and P.visible(1, {"size": 1, "keep_first": 0}) == [1]
    assert P.visible(2, {"size": 1, "keep_first": 9}) == [0, 1, 2] and P.visible(2, None) == [0, 1, 2]


def test_plain_state_space_is_the_sum_over_the_past():
    """The recurrence written out: y_t = sum_s prod(decays between) dt_s (C_t . B_s) x_s + D x_t."""
    m = C.states(4, 3, 5, 2, 3, 2)
    g = torch.Generator().manual_seed(0)
    width, T = 9, 12
    inner, ch = 12, 12 + 20
    W = {"mix.right.in": torch.randn(inner + ch + 4, width, generator=g), "mix.right.conv": torch.randn(ch, 3, generator=g),
         "mix.right.conv.b": torch.randn(ch, generator=g), "mix.right.dt_bias": torch.randn(4, generator=g),
         "mix.right.A_log": torch.randn(4, generator=g), "mix.right.D": torch.randn(4, generator=g),
         "mix.right.norm": torch.rand(inner, generator=g) + 0.5, "mix.right.o": torch.eye(inner)}
    h = torch.randn(T, width, generator=g, dtype=F64)
    st = P.new_mixer_state({"left": C.attention(1, 1, 2, 2, 1.0, 10.0, 2), "right": m})["right"]
    got = P.scalar_decay(h, W, m, st, 1e-5)
    proj = h @ W["mix.right.in"].double().T
    z, xbc, dt = proj[:, :inner], proj[:, inner:inner + ch], proj[:, inner + ch:]
    pad = torch.cat([torch.zeros(2, ch, dtype=F64), xbc])
    act = torch.nn.functional.silu(sum(pad[j:j + T] * W["mix.right.conv"][:, j].double() for j in range(3)) + W["mix.right.conv.b"].double())
    x, B, Cc = act[:, :inner].reshape(T, 4, 3), act[:, inner:inner + 10].reshape(T, 2, 5), act[:, inner + 10:].reshape(T, 2, 5)
    step = torch.nn.functional.softplus(dt + W["mix.right.dt_bias"].double())
    log_decay = -torch.exp(W["mix.right.A_log"].double()) * step
    y = torch.zeros(T, 4, 3, dtype=F64)
    for t in range(T):
        for hd in range(4):
            for s in range(t + 1):
                w = torch.exp(log_decay[s + 1:t + 1, hd].sum()) * step[s, hd] * (Cc[t, hd // 2] @ B[s, hd // 2])
                y[t, hd] += w * x[s, hd]
            y[t, hd] += W["mix.right.D"][hd].double() * x[t, hd]
    y = y.reshape(T, inner) * torch.nn.functional.silu(z)
    halves = y.reshape(T, 2, 6)
    want = (halves / (halves.pow(2).mean(-1, keepdim=True) + 1e-5).sqrt()).reshape(T, inner) * W["mix.right.norm"].double()
    assert torch.allclose(got, want, atol=1e-10)


def test_plain_choice():
    """The group with the single best expert is not the group with the best two; groups of one expert; every group kept."""
    z = torch.tensor([9.0, -9.0, 1.0, 1.0])
    assert [e for e, _ in P.choose(z, {"count": 2, "keep": 1}, 2)] == [2, 3]
    assert [e for e, _ in P.choose(z, {"count": 4, "keep": 2}, 2)] == [0, 2]
    got = P.choose(z, {"count": 1, "keep": 1}, 3)
    assert [e for e, _ in got] == [0, 2, 3] and math.isclose(sum(w for _, w in got), 1.0)


def test_plain_clamps():
    W = {"gate": torch.eye(3), "up": torch.eye(3), "down": torch.eye(3)}
    y = P.clamped_expert(torch.tensor([[5.0, -5.0, 0.5]], dtype=F64), W, "", 2.0)[0]
    swish = lambda g: g / (1.0 + math.exp(-1.702 * g))
    assert torch.allclose(y, torch.tensor([swish(2.0) * 3.0, swish(-5.0) * -1.0, swish(0.5) * 1.5], dtype=F64))


def test_plain_sink_and_soft_cap():
    """One key: its weight is e^s / (1 + e^s) with the capped score."""
    m = C.attention(1, 1, 2, 2, 3.0, 10.0, 2, softcap=1.5)
    W = {"mix.left." + n: torch.eye(2) for n in "qkvo"}
    W.update({"mix.left.q.norm": torch.ones(2), "mix.left.k.norm": torch.ones(2)})
    st = {"k": torch.zeros(0, 1, 2, dtype=F64), "v": torch.zeros(0, 1, 2, dtype=F64)}
    h = torch.tensor([[2.0, 1.0]], dtype=F64)
    s = 1.5 * math.tanh(2.0 * 3.0 / 1.5)                     # both normed rows are sqrt(2) long
    want = h * (math.exp(s) / (1.0 + math.exp(s)))
    assert torch.allclose(P.window_attention(h, W, m, st, 1e-12), want, atol=1e-6)
