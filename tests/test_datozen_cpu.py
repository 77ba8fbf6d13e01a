"""Datozen without a device: the configuration reader and its refusals, the declared tensors, the schedule of looped layers,
chunks in the cache managers, and the plain implementation against itself (pieces against whole, each mechanism against a
second way of writing it)."""
import copy
import math
import random

import pytest
import torch

import helpers as H
import plain_datozen as P
import datozen_cases as C
from dinfer_b200.cache.manager import CacheManager, GroupSpec
from dinfer_b200.config.model_config import ConfigError, DatozenConfig
from dinfer_b200.config.registry import resolve_architecture

F64 = torch.float64


def test_config_round_trip_and_spec():
    for name, d in C.CONFIGS.items():
        arch = resolve_architecture(d)
        cfg = arch.parse_config(d)
        assert isinstance(cfg, DatozenConfig) and cfg.to_dict() == DatozenConfig.from_dict(cfg.to_dict()).to_dict()
        spec = arch.build_spec(cfg)
        spec.check()
        assert spec.tie_word_embeddings and spec.embedding.kind == "positioned_table"
        assert all(l.block == "shared_norm_residual" and l.mixer.kind == "gqa_attention" for l in spec.layers)
        ff = {None: "none", "dense": "plain_mlp", "moe": "moe"}
        assert [l.feed_forward.kind for l in spec.layers] == [ff[(l["mlp"] or {}).get("kind")] for l in d["layers"]]
        assert [e.layer for e in spec.schedule] == P.schedule(d) and all(e.cache_from is None for e in spec.schedule)


def test_schedule_of_looped_layers():
    assert P.schedule(C.DATOZEN_A) == [0, 1, 2, 1, 2, 1, 2, 3]
    assert P.schedule(C.DATOZEN_B) == [0, 1, 0, 1, 2]
    assert P.schedule(C.DATOZEN_C) == [0, 1, 2] and P.schedule(C.DATOZEN_D) == [0, 1, 1, 1, 1]
    d = dict(C.DATOZEN_A, loop={"start": 0, "stop": 4, "times": 1})
    assert DatozenConfig.from_dict(d).schedule() == (0, 1, 2, 3)


def test_config_defaults():
    """Sections a layer or the model may leave out: identity experts, groups, a shared expert, stretching, the loop."""
    d = copy.deepcopy(C.DATOZEN_A)
    del d["loop"], d["layers"][0]["mixer"]["rot"]["scaling"]
    r = d["layers"][1]["mlp"]
    del r["router"]["identity"], r["router"]["groups"], r["shared"]
    cfg = DatozenConfig.from_dict(d)
    f = cfg.layers[1].mlp
    assert cfg.loop is None and cfg.layers[0].mixer.scaling is None
    assert (f.identity, f.groups, f.keep, f.shared_ff) == (0, 1, 1, 0)


@pytest.mark.parametrize("path, value", [
    (("norm", "eps"), 0.0), (("layers", 0, "type"), "retention"), (("layers", 0, "mixer", "kv_heads"), 3),
    (("layers", 0, "mixer", "heads"), 0), (("layers", 0, "mixer", "scale"), None), (("layers", 0, "mixer", "mask"), None),
    (("layers", 0, "mixer", "mask", "size"), 0), (("layers", 0, "mixer", "rot", "dims"), 14), (("layers", 0, "mixer", "rot", "dims"), 5),
    (("layers", 0, "mixer", "vdim"), 7), (("layers", 0, "mixer", "rot", "scaling", "factor"), 0.0),
    (("layers", 1, "mlp", "kind"), "sparse"), (("layers", 1, "mlp", "router", "groups", "count"), 4),
    (("layers", 1, "mlp", "router", "groups", "keep"), 4), (("layers", 1, "mlp", "router", "top"), 7),
    (("layers", 1, "mlp", "router", "identity"), -3), (("layers", 0, "mlp", "ff"), 0), (("max_positions",), None),
    (("token_side",), None), (("token_side", "dim"), 0), (("loop", "stop"), 5), (("loop", "times"), 0), (("loop", "start"), 3),
    (("vocab",), None), (("layers",), [])])
def test_config_refusals(path, value):
    d = copy.deepcopy(C.DATOZEN_A)
    at = d
    for k in path[:-1]:
        at = at[k]
    if value is None:
        del at[path[-1]]
    else:
        at[path[-1]] = value
    with pytest.raises(ConfigError):
        DatozenConfig.from_dict(d)


def test_declared_tensors():
    from dinfer_b200.weights.random_init import model_declarations
    decls = {x.name: tuple(x.shape) for x in model_declarations(C.DATOZEN_A)}
    w = 64
    assert decls["embed"] == (300, w) and decls["pos"] == (400, w) and decls["side.embed"] == (300, 48) and "head" not in decls
    assert decls["l0.norm1"] == (w,) and decls["final.norm"] == (w,) and "l0.norm2" not in decls
    assert decls["l0.mix.q"] == (48, w) and decls["l0.mix.k"] == (24, w) and decls["l0.mix.v"] == (40, w)
    assert decls["l0.mix.q.norm"] == (12,) and decls["l0.mix.k.norm"] == (12,) and decls["l0.mix.sink"] == (4,)
    assert decls["l0.mix.g"] == (4, w) and decls["l0.mix.o"] == (w, 80)
    assert decls["l0.mlp.up"] == (48, w) and decls["l0.mlp.act"] == (2,) and "l0.mlp.gate" not in decls
    assert decls["l1.mlp.router"] == (9, w) and decls["l1.mlp.correction"] == (9,) and "l1.mlp.e6.up" not in decls
    assert decls["l1.mlp.e5.gate"] == (24, w) and decls["l1.mlp.shared.gate"] == (40, w)
    assert "l2.mlp.up" not in decls and "l3.mlp.shared.up" not in decls and decls["l3.mlp.correction"] == (4,)
    assert decls["l3.side.gate"] == (12, w) and decls["l3.side.proj"] == (w, 12) and decls["l3.side.norm"] == (w,)


@pytest.mark.parametrize("native", [False, True])
def test_chunks_give_pages_back(native):
    """A chunk's pages stay until the next chunk's first token is due, whatever the page size; the pages of a chunk that
    begins inside a page keep that page."""
    from dinfer_b200.cache.native import NativeCacheManager
    make = NativeCacheManager if native else CacheManager
    m = make([GroupSpec(window=10, chunked=True), GroupSpec(window=10)], 4, [20, 20], 2)

    def held(req, g):
        return [i for i, b in enumerate(m.block_table(req, g)) if b >= 0]
    assert m.allocate("a", 9)
    m.advance("a", 9)                                       # the token to come, 9, is the chunk's last
    assert held("a", 0) == [0, 1, 2]
    assert m.allocate("a", 10)
    m.advance("a", 10)                                      # 10 begins the second chunk: pages 0, 1 (0..7) are passed
    assert held("a", 0) == [2] and held("a", 1) == [0, 1, 2]
    assert m.allocate("a", 23)
    m.advance("a", 19)                                      # still the second chunk
    assert held("a", 0) == [2, 3, 4, 5] and held("a", 1) == [2, 3, 4, 5]
    m.advance("a", 20)
    assert held("a", 0) == [5]
    m.advance("a", 23)
    assert held("a", 0) == [5] and m.num_free_blocks(0) == 19
    m.check_invariants()
    m.free("a")
    assert m.num_free_blocks(0) == 20 and m.num_free_blocks(1) == 20


def test_managers_agree_on_chunks():
    from dinfer_b200.cache.native import NativeCacheManager
    rng = random.Random(5)
    for groups in ([GroupSpec(window=7, chunked=True)], [GroupSpec(window=12, chunked=True), GroupSpec(window=3, block_size=2, chunked=True)]):
        a, b = CacheManager(groups, 4, [40] * len(groups), 3), NativeCacheManager(groups, 4, [40] * len(groups), 3)
        at = {"x": 0, "y": 0}
        for _ in range(200):
            r = rng.choice(["x", "y"])
            n = rng.randrange(1, 9)
            if at[r] + n > 60:
                a.free(r); b.free(r)
                at[r] = 0
                continue
            assert a.allocate(r, at[r] + n) and b.allocate(r, at[r] + n)
            at[r] += n
            a.advance(r, at[r]); b.advance(r, at[r])
            for g in range(len(groups)):
                assert a.block_table(r, g) == b.block_table(r, g)
        a.check_invariants(); b.check_invariants()


def test_prefix_cache_refuses_chunks():
    with pytest.raises(ValueError):
        CacheManager([GroupSpec(window=8, chunked=True)], 4, 8, 2, enable_prefix_caching=True)


@pytest.mark.parametrize("dims, base, scaling", [(8, 300.0, (4.0, 40.0, 6.0, 1.0)), (4, 50.0, (2.5, 64.0, 3.0, 3.0)),
                                                 (64, 10000.0, (16.0, 4096.0, 32.0, 1.0)), (6, 10000.0, (8.0, 30.0, 20.0, 0.5))])
def test_stretched_frequencies(dims, base, scaling):
    from dinfer_b200.parts.rope import ramp_frequencies, rope_table
    s = dict(zip(("factor", "original", "fast", "slow"), scaling))
    f, mult = P.stretched(dims, base, s)
    got, got_mult = ramp_frequencies(dims, base, *scaling)
    assert torch.allclose(got, torch.tensor(f, dtype=F64), rtol=1e-13) and math.isclose(mult, got_mult)
    table = rope_table(dims, base, 50, "cpu", ramp=scaling).double()
    x = torch.randn(50, 1, dims, dtype=F64)
    want = P.turn(x, torch.arange(50), f, mult)
    c, sn = table[:, :dims // 2], table[:, dims // 2:]
    u, v = x[:, 0, :dims // 2], x[:, 0, dims // 2:]
    assert torch.allclose(torch.cat([u * c - v * sn, v * c + u * sn], dim=1), want[:, 0], atol=1e-5)


def _weights(cfg, seed=3):
    from dinfer_b200.weights.random_init import model_declarations, random_tensor
    return {d.name: random_tensor(d, seed, 0.2, 0.3, torch.float32).double() for d in model_declarations(cfg)}


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


def test_plain_attention_with_turned_values_is_relative():
    """Values turned by j and back by i are the values turned by j - i: moving a whole chunk-aligned sequence by a number of
    positions that keeps the chunks changes nothing."""
    m = C.DATOZEN_A["layers"][0]["mixer"]
    W = {k[3:]: v for k, v in _weights(C.DATOZEN_A).items() if k.startswith("l0.")}
    h = torch.randn(7, 64, dtype=F64)
    empty = lambda n: {"k": torch.zeros(n, 2, 12, dtype=F64), "v": torch.zeros(n, 2, 20, dtype=F64)}
    at_zero = P.chunk_attention(h, W, m, empty(0), 1e-5)
    at_fourteen = P.chunk_attention(h, W, m, empty(14), 1e-5)
    assert torch.allclose(at_zero, at_fourteen, atol=1e-12)
    assert not torch.allclose(at_zero, P.chunk_attention(h, W, m, empty(3), 1e-5), atol=1e-3)      # a chunk begins inside


def test_plain_choice():
    """Groups, negative choice scores, identity experts: against a brute-force ranking of every expert."""
    g = torch.Generator().manual_seed(0)
    for n, count, keep, top in ((12, 4, 2, 3), (9, 3, 1, 3), (6, 6, 5, 4), (8, 1, 1, 8)):
        for _ in range(30):
            z, c = torch.randn(n, generator=g) * 3, torch.randn(n, generator=g) - 1.5
            got = P.choose(z, c, {"count": count, "keep": keep}, top)
            s = torch.softmax(z.double(), -1)
            choice = s + c.double()
            best = choice.reshape(count, -1).max(dim=1).values
            kept = torch.topk(best, keep).indices.tolist()
            masked = torch.full((n,), -float("inf"), dtype=F64)
            for k in kept:
                lo = k * (n // count)
                masked[lo:lo + n // count] = choice[lo:lo + n // count]
            want = torch.topk(masked, top).indices.tolist()
            assert [e for e, _ in got] == want and all(abs(w - float(s[e])) < 1e-12 for e, w in got)


def test_plain_activation():
    z = torch.tensor([-30.0, -2.0, -1e-3, 0.0, 1e-3, 2.0, 30.0], dtype=F64)
    p, q = torch.tensor(0.3, dtype=F64), torch.tensor(-0.8, dtype=F64)
    ap, an = math.log1p(math.exp(0.3)), 0.5 + math.log1p(math.exp(-0.8))
    want = [ap * v * v + 0.5 * v if v > 0 else an * (math.expm1(v) - v) + 0.5 * v for v in z.tolist()]
    assert torch.allclose(P.xielu(z, p, q), torch.tensor(want, dtype=F64), atol=1e-12)
