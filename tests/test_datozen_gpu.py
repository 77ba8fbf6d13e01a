"""Datozen on the device: every new mechanism alone against the plain implementation's function for it, then tiny models
that differ in every size replayed whole / with a decoded tail / in portions down to two tokens / mixed on a pool that only
holds the most demanding step, the trace runner as a process, and greedy generation through ``LLM``."""
import json
import os
import random

import numpy as np
import pytest
import torch

import helpers as H
import plain_datozen as P
import datozen_cases as C
from test_sobivik_gpu import DT, F64, PLAN, Bench, close, dev, env, i32, rms_err, rows_for, run_cut, weights_for

pytestmark = pytest.mark.gpu


# ---------------------------------------------------------------- chunked attention through its part

ATT = [  # heads, kv heads, dim, vdim, chunk, rot dims, stretching, page size
    (4, 2, 12, 20, 7, 8, (4.0, 40.0, 6.0, 1.0), 16), (6, 1, 24, 14, 16, 24, None, 4), (3, 3, 10, 6, 33, 2, None, 16),
    (4, 1, 64, 64, 24, 32, (6.0, 90.0, 8.0, 1.5), 16), (2, 2, 32, 32, 40, 16, None, 8), (4, 2, 128, 128, 50, 128, None, 16),
    (6, 2, 64, 64, 1000, 24, None, 64), (1, 1, 96, 40, 1, 96, None, 16), (2, 1, 256, 256, 20, 64, None, 16)]


def att_case(H_, G, D, V, chunk, rot, scaling):
    m = C.attention(H_, G, D, V, chunk, 300.0, rot, 0.7 * D ** -0.5, scaling)["mixer"]
    from dinfer_b200.parts.spec import PartSpec
    rope = {"head_dim": D, "rotary_dim": rot, "theta": 300.0, "max_positions": 1024, "style": "neox"}
    if scaling:
        rope["ramp"] = m["rot"]["scaling"]
    p = {"num_heads": H_, "num_kv_heads": G, "head_dim": D, "v_dim": V, "scale": m["scale"], "eps": 1e-5, "qk_norm": True,
         "position": PartSpec("rope", rope), "window": chunk, "chunked": True, "value_turn": 300.0, "sink": "mix.sink",
         "gate_proj": "mix.g", "gate_per": "head", "q_proj": "mix.q", "k_proj": "mix.k", "v_proj": "mix.v", "o_proj": "mix.o",
         "q_norm": "mix.q.norm", "k_norm": "mix.k.norm"}
    return m, p


def empty_state(m):
    return {"k": torch.zeros(0, m["kv_heads"], m["dim"], dtype=F64), "v": torch.zeros(0, m["kv_heads"], m["vdim"], dtype=F64)}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H_, G, D, V, chunk, rot, scaling, block_size", ATT)
def test_chunk_attention(dtype, H_, G, D, V, chunk, rot, scaling, block_size):
    """Prompts beside portions behind a history beside decoded tokens: keys and values of different widths (plain-arithmetic
    kernel) and of one width (tensor-core kernels in bfloat16), chunks smaller and larger than a page, than a tile and than
    the request, chunks of one token (only the sink beside the token itself)."""
    import dinfer_b200.models.decoder  # noqa: F401
    from dinfer_b200.parts.base import MIXERS
    width = 64
    m, p = att_case(H_, G, D, V, chunk, rot, scaling)
    W = weights_for(MIXERS.get("gqa_attention")(p, env(width, torch.float32), "").declare(), dtype, D + V, std=0.15,
                    scale={"mix.sink": 12.0, "mix.q.norm": 12.0, "mix.k.norm": 12.0, "mix.g": 4.0})
    bench = Bench("gqa_attention", p, W, dtype, width, block_size=block_size, num_blocks=4096 // block_size)
    bench.binding.kv.zero_()         # as the engine makes it: the TMA kernels fetch whole pages, and 0 * NaN is no 0
    inputs = rows_for(width, dtype, 5)
    got = run_cut(bench, inputs, PLAN)
    for r, x in inputs.items():
        close(got[r], P.chunk_attention(x.double(), W, m, empty_state(m), 1e-5), dtype, r)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("D, chunk", [(24, 40), (64, 40), (64, 128), (128, 200), (32, 16)])
def test_chunk_edges(dtype, D, chunk):
    """One key stands out from every other by far.  A query of the same chunk finds it, wherever in the chunk it lies (the
    chunk's first position too); the first query of the next chunk does not, although the key is its neighbour.  As a
    prompt's row, as the first row of a portion and decoded alone."""
    m = {"heads": 1, "kv_heads": 1, "dim": D, "vdim": D, "scale": 1.0, "rot": {"base": 1e6, "dims": 2}, "mask": {"size": chunk}}
    _, p = att_case(1, 1, D, D, chunk, 2, None)
    from dinfer_b200.parts.spec import PartSpec
    p.update(scale=1.0, value_turn=1e6, position=PartSpec("rope", {"head_dim": D, "rotary_dim": 2, "theta": 1e6, "max_positions": 1024}))
    width = D
    eye = torch.eye(D)
    W = {"mix.q": eye, "mix.k": eye, "mix.v": eye, "mix.o": eye, "mix.q.norm": torch.full((D,), 1.0),
         "mix.k.norm": torch.full((D,), 1.0), "mix.sink": torch.tensor([1.0]), "mix.g": torch.zeros(1, D)}
    g = torch.Generator().manual_seed(D + chunk)
    for key_at, ask in ((chunk, 2 * chunk - 1), (chunk, chunk + 1), (2 * chunk - 1, 2 * chunk), (chunk - 1, chunk), (0, chunk - 1),
                        (2 * chunk - 2, 2 * chunk - 1), (chunk, 2 * chunk)):
        T = 2 * chunk + 3
        x = torch.randn(T, width, generator=g)
        x[:, 4] = 0.0
        x[key_at, :] = torch.randn(width, generator=g) * 0.05
        x[key_at, 4] = 3.0                                      # after the norm this key is sqrt(D) along element 4
        x[ask, :] = torch.randn(width, generator=g) * 0.05
        x[ask, 4] = 3.0
        x = x.to(DT[dtype]).float()
        want = P.chunk_attention(x.double(), W, m, empty_state(m), 1e-5)
        seen = ask // chunk == key_at // chunk
        for cut_ in ("prompt", "portion", "decoded"):
            bench = Bench("gqa_attention", p, W, dtype, width, block_size=16, num_blocks=64)
            bench.binding.kv.zero_()
            sizes = {"prompt": [T], "portion": [ask, T - ask], "decoded": [ask, 1, T - ask - 1]}[cut_]
            out, at = [], 0
            for n in sizes:
                if n:
                    out.append(bench.run([("a", x[at:at + n])]))
                at += n
            close(torch.cat(out), want, dtype, (key_at, ask, cut_))
        # what the key adds shows: without it the row differs
        y = x.clone()
        y[key_at] = 0.01
        moved = float((P.chunk_attention(y.double(), W, m, empty_state(m), 1e-5)[ask] - want[ask]).abs().max())
        assert (moved > 1e-3) == seen, (key_at, ask, moved)


@pytest.mark.parametrize("D, H_, G, block_size, chunk", [
    (64, 4, 2, 16, 150), (128, 8, 2, 16, 64), (64, 2, 2, 64, 200), (128, 4, 1, 8, 97), (32, 4, 4, 4, 70), (128, 4, 4, 16, 512),
    (64, 6, 2, 16, 130), (64, 8, 8, 16, 9)])
def test_tensor_core_attention_in_chunks(D, H_, G, block_size, chunk):
    """The tensor-core kernels (tcgen05 prompt kernels with 64- and 128-key tiles, the TMA decode kernel with its key
    splits, the mma.sync kernel) with chunks and learned sinks, against the plain-arithmetic kernel on the same cache, where
    pages that no query needs are missing from the tables: a prompt over several chunks, portions behind a history that
    begin, end and lie inside a chunk, decoded tokens at a chunk's first and last position."""
    from dinfer_b200.kernels import attention_ops, ops
    g = torch.Generator().manual_seed(D + H_)
    scale = 0.6 * D ** -0.5
    seqs = [(0, 300), (7 * chunk, 1), (chunk - 5, 140), (0, 1), (chunk - 1, 1), (2 * chunk, 60), (3 * chunk - 1, 2), (chunk + 3, 1)]
    total = [a + b for a, b in seqs]
    pages = [(n + block_size - 1) // block_size for n in total]
    perm = torch.randperm(sum(pages), generator=g)
    tab = torch.full((len(seqs), max(pages)), -1, dtype=torch.int32)
    at = 0
    for b, n in enumerate(pages):
        tab[b, :n] = perm[at:at + n]
        tab[b, :seqs[b][0] // chunk * chunk // block_size] = -1       # passed: given back
        at += n
    cache = torch.randn(sum(pages), 2, G, block_size, D, generator=g).to(torch.bfloat16).cuda()
    T = sum(b for _, b in seqs)
    q = torch.randn(T, H_ * D, generator=g).to(torch.bfloat16).cuda()
    sinks = dev(torch.randn(H_, generator=g) * 1.5 + 1.0)
    pos = torch.cat([torch.arange(a, a + b) for a, b in seqs]).to(torch.int32).cuda()
    cu = i32(np.concatenate([[0], np.cumsum([b for _, b in seqs])]))
    seq_lens, table = i32(total), dev(tab)
    want = torch.empty(T, H_ * D, dtype=torch.bfloat16, device="cuda")
    kw = dict(chunked=True, sinks=sinks)
    ops.attention_generic(q, want, cache, table, cu, pos, H_, G, D, scale, chunk, **kw)
    other = torch.empty_like(want)
    ops.attention_generic(q, other, cache, table, cu, pos, H_, G, D, scale, chunk, chunked=True, sinks=sinks + 1.0)
    assert float((want.float() - other.float()).abs().max()) > 0.02          # the sinks matter at these scores
    prompt_rows = torch.cat([torch.arange(int(cu[i]), int(cu[i + 1])) for i, (_, b) in enumerate(seqs) if b > 1]).cuda()
    decode_rows = torch.cat([torch.arange(int(cu[i]), int(cu[i + 1])) for i, (_, b) in enumerate(seqs) if b == 1]).cuda()
    group = H_ // G

    def near(got, rows, what):
        d = float((got[rows].float() - want[rows].float()).abs().max())
        assert d <= 2e-2, (what, d)

    for splits in (1, 4):
        got = torch.full_like(want, float("nan"))
        attention_ops.attention_tc(q, got, cache, table, cu, seq_lens, H_, G, D, scale, chunk, 300, True, True, splits, **kw)
        near(got, torch.arange(T).cuda(), f"mma.sync kernel, {splits} splits")
    if attention_ops.decode_supported(torch.bfloat16, D, group, block_size) and block_size >= 8:
        for splits in (1, 2, 8):
            got = torch.full_like(want, float("nan"))
            attention_ops.attention_decode(q, got, cache, table, cu, seq_lens, H_, G, D, scale, chunk, splits, **kw)
            near(got, decode_rows, f"decode kernel, {splits} splits")
    if attention_ops.umma_supported(torch.bfloat16, D, group, block_size):
        lens = [b for _, b in seqs]
        bound = attention_ops.umma_pair_bound(lens, group)
        for ks in (1, 2):
            got = torch.full_like(want, float("nan"))
            attention_ops.attention_umma(q, got, cache, table, cu, seq_lens, H_, G, D, scale, chunk, 300, ks, bound, **kw)
            near(got, prompt_rows, f"tcgen05 kernel, keys shared {ks} ways")
        if attention_ops.umma64_supported(torch.bfloat16, D, group, block_size):
            got = torch.full_like(want, float("nan"))
            attention_ops.attention_umma64(q, got, cache, table, cu, seq_lens, H_, G, D, scale, chunk, 300, bound, **kw)
            near(got, prompt_rows, "tcgen05 kernel with 64-key tiles")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("chunked", [False, True])
@pytest.mark.parametrize("window", [1, 5, 16, 100])
def test_plain_kernel_windows_and_sinks(dtype, chunked, window):
    """The plain-arithmetic kernel's windows, chunks and sinks against the softmax written out; sinks far above and far
    below every score."""
    from dinfer_b200.kernels import ops
    g = torch.Generator().manual_seed(window)
    T, H_, G, D, bs = 60, 4, 2, 12, 8
    q, k, v = (torch.randn(T, n, D, generator=g).to(DT[dtype]) for n in (H_, G, G))
    sinks = torch.tensor([40.0, -40.0, 1.0, 0.0])
    cache = torch.zeros(8, 2, G, bs, D, dtype=DT[dtype])
    for j in range(T):
        cache[j // bs, 0, :, j % bs], cache[j // bs, 1, :, j % bs] = k[j], v[j]
    got = torch.empty(T, H_ * D, dtype=DT[dtype], device="cuda")
    ops.attention_generic(dev(q.reshape(T, -1)), got, dev(cache), i32([list(range(8))]), i32([0, T]), i32(list(range(T))), H_, G, D, 0.5,
                          window, chunked=chunked, sinks=dev(sinks))
    want = torch.zeros(T, H_, D, dtype=F64)
    for t in range(T):
        first = t // window * window if chunked else max(0, t - window + 1)
        for h in range(H_):
            s = k[first:t + 1, h // 2].double() @ q[t, h].double() * 0.5
            a = torch.softmax(torch.cat([s, sinks[h:h + 1].double()]), 0)[:-1]
            want[t, h] = a @ v[first:t + 1, h // 2].double()
    assert float((got.double().cpu() - want.reshape(T, -1)).abs().max()) <= (1e-5 if dtype == "float32" else 2e-2)


# ---------------------------------------------------------------- turned values, the heads' outputs

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H_, G, D, V, rot, T", [(4, 2, 64, 64, 32, 9), (32, 8, 128, 128, 64, 600), (3, 3, 128, 128, 128, 3), (6, 2, 256, 256, 16, 5),
                                                 (4, 2, 64, 64, 20, 7), (4, 2, 12, 20, 8, 11), (2, 1, 80, 80, 40, 4), (5, 1, 64, 32, 64, 6)])
def test_keys_and_values_turned(dtype, H_, G, D, V, rot, T):
    """Head norm, rotation and the turned values in the cache: sizes of the kernel without shared memory (a token's heads
    walked over, or a thread group each) and of the general one; slots all over the cache, tokens that are not stored."""
    from dinfer_b200.kernels import ops
    from dinfer_b200.parts.rope import rope_table
    g = torch.Generator().manual_seed(D + V + T)
    bs, eps, base = 8, 1e-5, 500.0
    x = torch.randn(T, ((H_ + G) * D + G * V + 15) // 8 * 8, generator=g).to(DT[dtype])
    wq, wk = (1.0 + torch.randn(D, generator=g) * 0.3).to(DT[dtype]), (1.0 + torch.randn(D, generator=g) * 0.3).to(DT[dtype])
    pos = torch.randint(0, 400, (T,), generator=g)
    blocks = (T + bs - 1) // bs + 1
    slots = torch.randperm(blocks * bs, generator=g)[:T].to(torch.int32)
    slots[1] = -1
    ramp = (4.0, 100.0, 8.0, 1.0)
    table, v_table = rope_table(rot, base, 400, "cuda", ramp=ramp), rope_table(V, base, 400, "cuda")
    cache = torch.full((blocks, 2, G, bs, max(D, V)), 7.0, dtype=DT[dtype], device="cuda")
    rows = dev(x)
    ops.qkv_post_general(rows, i32(pos.tolist()), H_, G, D, V, eps, dev(wq), dev(wk), True, True, table, cache, dev(slots), bs,
                         v_cos_sin=v_table)
    f, mult = P.stretched(rot, base, dict(zip(("factor", "original", "fast", "slow"), ramp)))
    q = P.turn(P.rms_norm(x[:, :H_ * D].double().reshape(T, H_, D), wq, eps), pos, f, mult)
    k = P.turn(P.rms_norm(x[:, H_ * D:(H_ + G) * D].double().reshape(T, G, D), wk, eps), pos, f, mult)
    v = P.turn(x[:, (H_ + G) * D:(H_ + G) * D + G * V].double().reshape(T, G, V), pos, P.plain_frequencies(V, base))
    tol = 2e-5 if dtype == "float32" else 3e-2
    assert torch.allclose(rows[:, :H_ * D].double().cpu().reshape(T, H_, D), q, atol=tol, rtol=tol)
    assert torch.equal(rows[:, (H_ + G) * D:].cpu(), x[:, (H_ + G) * D:])
    c = cache.double().cpu()
    stored = torch.zeros(blocks * bs, dtype=torch.bool)
    for t in range(T):
        s = int(slots[t])
        if s < 0:
            continue
        stored[s] = True
        assert torch.allclose(c[s // bs, 0, :, s % bs, :D], k[t], atol=tol, rtol=tol)
        assert torch.allclose(c[s // bs, 1, :, s % bs, :V], v[t], atol=tol, rtol=tol)
    free = ~stored.reshape(blocks, bs)
    assert bool((c.permute(0, 3, 1, 2, 4)[free] == 7.0).all())


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H_, V, T", [(4, 64, 5), (32, 128, 600), (6, 112, 3), (3, 20, 7), (2, 6, 4), (1, 256, 2), (5, 7, 3)])
@pytest.mark.parametrize("turned, gated", [(True, True), (True, False), (False, True)])
def test_heads_out(dtype, H_, V, T, turned, gated):
    from dinfer_b200.kernels import ops
    from dinfer_b200.parts.rope import rope_table
    if turned and V % 2:
        return
    g = torch.Generator().manual_seed(V)
    x, gate = torch.randn(T, H_ * V, generator=g).to(DT[dtype]), torch.randn(T, H_ + 5, generator=g).to(DT[dtype])
    pos = torch.randint(0, 300, (T,), generator=g)
    got = ops.heads_out(dev(x), i32(pos.tolist()), H_, V, rope_table(V, 90.0, 300, "cuda") if turned else None,
                        dev(gate)[:, 2:2 + H_] if gated else None).double().cpu()
    want = x.double().reshape(T, H_, V)
    if turned:
        want = P.turn(want, pos, P.plain_frequencies(V, 90.0), sign=-1.0)
    if gated:
        want = want * P.sigmoid(gate[:, 2:2 + H_].double())[:, :, None]
    tol = 1e-5 if dtype == "float32" else 2e-2
    assert torch.allclose(got, want.reshape(T, -1), atol=tol, rtol=tol)


# ---------------------------------------------------------------- the router and the experts

@pytest.mark.parametrize("n, count, keep, top, T", [(12, 4, 2, 3, 50), (9, 3, 1, 3, 7), (6, 6, 5, 4, 1), (8, 1, 1, 8, 33), (160, 8, 3, 6, 200),
                                                    (40, 1, 1, 1, 5), (66, 33, 4, 2, 64)])
@pytest.mark.parametrize("corrected", [True, False])
def test_route_choice(n, count, keep, top, T, corrected):
    """The chosen experts in their order and the scores as weights; corrections that make every choice score negative; rows
    where the best group is the one with the single best expert, not the best sum."""
    from dinfer_b200.kernels import moe_ops
    g = torch.Generator().manual_seed(n + T)
    z = torch.randn(T, n, generator=g) * 3
    c = torch.randn(n, generator=g) * 0.4 - 1.5 if corrected else torch.zeros(n)
    wide = torch.cat([z, torch.full((T, 3), 50.0)], dim=1)                    # columns behind the experts are not experts
    ids, w = moe_ops.route_choice(dev(wide), n, top, dev(c) if corrected else None, "softmax", False, count, keep)
    for t in range(T):
        want = P.choose(z[t], c, {"count": count, "keep": keep}, top)
        assert ids[t].tolist() == [e for e, _ in want], t
        assert torch.allclose(w[t].double().cpu(), torch.tensor([s for _, s in want], dtype=F64), rtol=1e-5, atol=1e-7)
    ids2, w2 = moe_ops.route_choice(dev(wide), n, top, dev(c) if corrected else None, "softmax", True, count, keep)
    assert torch.equal(ids, ids2) and torch.allclose(w2.sum(dim=1), torch.ones(T, device="cuda"), atol=1e-5)
    if not corrected and count == 1:
        ids3, w3, _ = moe_ops.route(dev(wide), n, top, "softmax", False)
        assert torch.equal(ids, ids3) and torch.allclose(w, w3, rtol=1e-5)


def test_route_choice_refuses():
    from dinfer_b200.kernels import moe_ops
    from dinfer_b200.kernels.lib import KernelError
    z = torch.zeros(2, 12, device="cuda")
    for kw in (dict(groups=5, keep=1), dict(groups=4, keep=5), dict(groups=4, keep=0), dict(groups=4, keep=1)):
        with pytest.raises(KernelError):
            moe_ops.route_choice(z, 12, 4, None, "softmax", False, **kw)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("E, ident, top, count, keep, ff, shared, width, T", [
    (6, 3, 2, 3, 2, 24, 40, 64, 37), (4, 0, 1, 2, 1, 20, 0, 72, 5), (2, 2, 2, 4, 3, 20, 12, 40, 64), (7, 2, 4, 3, 2, 12, 20, 128, 1),
    (8, 2, 3, 5, 3, 64, 96, 128, 700), (1, 5, 3, 2, 2, 16, 8, 64, 90), (3, 1, 4, 1, 1, 8, 0, 66, 20)])
def test_experts_with_groups_and_identity(dtype, E, ident, top, count, keep, ff, shared, width, T):
    """The part against the plain form: identity experts among the chosen ones, tokens that choose nothing else, all
    experts chosen, few rows and enough for the tcgen05 grouped product (700 tokens)."""
    import dinfer_b200.models.decoder  # noqa: F401
    from dinfer_b200.parts.base import FEED_FORWARDS
    p = {"num_experts": E, "identity": ident, "top_k": top, "groups": (count, keep), "expert_size": ff, "shared_size": shared,
         "activation": "silu", "gated": True, "scoring": "softmax", "renormalize": False, "router": "mlp.router",
         "correction": "mlp.correction", "expert_gate": "mlp.e{e}.gate", "expert_up": "mlp.e{e}.up", "expert_down": "mlp.e{e}.down",
         "shared_gate_up": "mlp.shared.gate", "shared_up": "mlp.shared.up", "shared_down": "mlp.shared.down"}
    part = FEED_FORWARDS.get("moe")(p, env(width, DT[dtype]), "")
    W = weights_for(part.declare(), dtype, E + top, std=0.2, scale={"mlp.router": 2.0, "mlp.correction": 3.0})
    part.bind({k: dev(v, DT[dtype]) for k, v in W.items()})
    x = (torch.randn(T, width, generator=torch.Generator().manual_seed(T)) * 1.5).to(DT[dtype]).float()
    got = part.forward(dev(x, DT[dtype])).double().cpu()
    f = C.moe(E, ident, top, count, keep, ff, shared)
    want = P.expert_ff(x.double(), W, f)
    # a choice that hangs on less than a rounding of the products is not what this test is about
    z = P.lin(x.double(), W["mlp.router"])
    sure = torch.ones(T, dtype=torch.bool)
    for t in range(T):
        a = P.choose(z[t], W["mlp.correction"], f["router"]["groups"], top)
        for d in (1e-4, -1e-4):
            jitter = torch.where(torch.arange(E + ident) % 2 == 0, d, -d)
            sure[t] &= {e for e, _ in a} == {e for e, _ in P.choose(z[t] + jitter, W["mlp.correction"], f["router"]["groups"], top)}
    assert int(sure.sum()) >= 0.9 * T
    close(got[sure], want[sure], dtype)
    if ident:
        assert any(e >= E for t in range(T) for e, _ in P.choose(z[t], W["mlp.correction"], f["router"]["groups"], top)) or T == 1


# ---------------------------------------------------------------- the feed-forward without a gate

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("ff, width, T", [(48, 64, 1), (40, 64, 30), (36, 72, 45), (96, 128, 600), (2048, 256, 8), (1024, 512, 700), (28, 50, 9)])
def test_xielu_feed_forward(dtype, ff, width, T):
    """The activation in the epilogue of the decode product (with and without split K), of the two-SM prompt product, and as
    a kernel of its own between; inputs of both signs, large and near zero."""
    import dinfer_b200.models.decoder  # noqa: F401
    from dinfer_b200.parts.base import FEED_FORWARDS
    part = FEED_FORWARDS.get("plain_mlp")({"intermediate_size": ff, "activation": "xielu", "up_proj": "mlp.up", "down_proj": "mlp.down",
                                           "act": "mlp.act"}, env(width, DT[dtype]), "")
    W = weights_for(part.declare(), dtype, ff, std=1.0 / width ** 0.5, scale={"mlp.act": 12.0})
    part.bind({k: dev(v, DT[dtype]) for k, v in W.items()})
    x = torch.randn(T, width, generator=torch.Generator().manual_seed(T)).to(DT[dtype]).float()
    x[0] *= 3.0
    close(part.forward(dev(x, DT[dtype])).double().cpu(), P.dense_ff(x.double(), W), dtype)


@pytest.mark.parametrize("act", ["relu", "relu2", "silu", "gelu_tanh"])
@pytest.mark.parametrize("T, width, ff", [(5, 128, 96), (9, 1024, 256), (600, 64, 136)])
def test_other_activations_without_a_gate(act, T, width, ff):
    """The same epilogues with the other activations (few rows with and without split K, prompt rows)."""
    import dinfer_b200.models.decoder  # noqa: F401
    from dinfer_b200.parts.base import FEED_FORWARDS
    part = FEED_FORWARDS.get("plain_mlp")({"intermediate_size": ff, "activation": act}, env(width, torch.bfloat16), "")
    W = weights_for(part.declare(), "bfloat16", ff, std=1.0 / width ** 0.5)
    part.bind({k: dev(v, torch.bfloat16) for k, v in W.items()})
    x = torch.randn(T, width, generator=torch.Generator().manual_seed(T)).to(torch.bfloat16).float()
    f = {"relu": lambda z: z.clamp(min=0), "relu2": lambda z: z.clamp(min=0) ** 2, "silu": P.silu, "gelu_tanh": P.gelu_tanh}[act]
    close(part.forward(dev(x, torch.bfloat16)).double().cpu(), P.lin(f(P.lin(x.double(), W["up_proj.weight"])), W["down_proj.weight"]), "bfloat16")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_xielu_values(dtype):
    from dinfer_b200.kernels import moe_ops
    z = torch.cat([torch.linspace(-20, 20, 797), torch.tensor([-100.0, -1e-3, -1e-5, 0.0, 1e-5, 1e-3, 50.0])]).to(DT[dtype])
    for n in (z.numel(), z.numel() - 3):                     # a length of whole vectors and not
        x = dev(z[:n])
        got = moe_ops.xielu(x, torch.empty_like(x), 0.7, 1.2).double().cpu()
        zz = z[:n].double()
        want = torch.where(zz > 0, 0.7 * zz * zz + 0.5 * zz, 1.2 * (torch.expm1(zz) - zz) + 0.5 * zz)
        assert torch.allclose(got, want, rtol=2e-6 if dtype == "float32" else 5e-3, atol=1e-7 if dtype == "float32" else 1e-3)


# ---------------------------------------------------------------- the token side

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("dim, width, T", [(12, 64, 9), (5, 72, 40), (32, 128, 600), (9, 50, 3)])
def test_token_side(dtype, dim, width, T):
    """The part's own rows and the join around them, in a block whose sublayers put out zeros; token ids that name the last
    step's samples; the layer's part of a row that holds three layers'."""
    import dinfer_b200.models.decoder  # noqa: F401
    from dinfer_b200.kernels import stream_ops
    from dinfer_b200.parts.token_side import TokenSide
    eps = 3e-6
    p = {"dim": dim, "index": 1, "layers": 3, "vocab_size": 50, "eps": eps, "table": "side.embed", "gate_proj": "side.gate",
         "out_proj": "side.proj", "norm": "side.norm"}
    side = TokenSide(p, env(width, DT[dtype]), "")
    W = weights_for(side.declare(), dtype, dim, std=0.3)
    side.bind({k: dev(v, DT[dtype]) for k, v in W.items()})
    g = torch.Generator().manual_seed(T)
    x, a, f = torch.randn(T, width, generator=g), torch.randn(T, width, generator=g).to(DT[dtype]), torch.randn(T, width, generator=g).to(DT[dtype])
    real = [int(v) for v in torch.randint(0, 50, (T,), generator=g)]
    sampled = [31, 7]
    given = [(-1 - r if t % 5 == 2 else real[t]) for t, r in ((t, t % 2) for t in range(T))]
    real = [sampled[-v - 1] if v < 0 else v for v in given]

    class Ctx:
        token_ids, prev_tokens = i32(given), i32(sampled)
    for second in (None, f):
        stream, cast = dev(x), torch.empty(T, width, dtype=DT[dtype], device="cuda")
        stream_ops.branch_join(stream, dev(a), dev(second) if second is not None else None, cast)
        want = x.double() + a.double() + (second.double() if second is not None else 0.0)
        assert torch.allclose(stream.double().cpu(), want, atol=1e-5)
        assert torch.equal(cast.cpu(), stream.cpu().to(DT[dtype]))
        y = side.forward(cast, Ctx)
        stream_ops.gain_norm_join(y, side.norm.weight.float(), eps, stream, stream)
        want = P.token_side(want, real, W, 1, dim, eps, W["side.embed"])
        close(stream.double().cpu(), want, dtype)


# ---------------------------------------------------------------- whole models

LENGTHS = {"A": {"a": 1, "b": 2, "c": 45, "d": 131, "e": 77},
           "B": {"a": 150, "b": 3, "c": 66, "d": 1, "e": 19},
           "C": {"a": 97, "b": 40, "c": 2, "d": 71},
           "D": {"a": 120, "b": 1, "c": 33, "d": 64},
           "E": {"a": 190, "b": 17, "c": 65, "d": 270}}
BF16_WORST, BF16_RMS, BF16_OVER = 0.25, 0.06, 0.1


class Oracle:
    def __init__(self, model_dir):
        self.cfg = json.load(open(os.path.join(model_dir, "config.json")))
        self.W = C.load_weights(model_dir)
        self._cache = {}

    def logits(self, ids):
        key = tuple(ids)
        if key not in self._cache:
            self._cache[key] = P.forward(self.cfg, self.W, list(ids), P.new_state(self.cfg)).numpy()
        return self._cache[key]


@pytest.fixture(scope="module")
def model_dirs(tmp_path_factory):
    out = {}
    for name, cfg in C.CONFIGS.items():
        for dt in DT:
            out[(name, dt)] = C.write_model(str(tmp_path_factory.mktemp(f"datozen{name}_{dt}")), cfg, 11 + ord(name), DT[dt])
    return out


_REQUESTS = {}


def requests(name, model_dirs):
    if name not in _REQUESTS:
        cfg, rng = C.CONFIGS[name], random.Random(7 + ord(name))
        oracle = Oracle(model_dirs[(name, "bfloat16")])
        tokens = {r: H.random_tokens(rng, n, cfg["vocab"]) for r, n in LENGTHS[name].items()}
        _REQUESTS[name] = (tokens, {r: oracle.logits(t) for r, t in tokens.items()})
    return _REQUESTS[name]


@pytest.mark.parametrize("block_size", [4, 16, 64])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(C.CONFIGS))
def test_replay_all_ways(model_dirs, name, dtype, block_size):
    """Every position of every request: whole / with a decoded tail long enough to pass pages and chunks / in portions down
    to two tokens / mixed with up to four live requests (some sitting steps out) on a pool that only holds the most
    demanding step, so that pages and state slots are freed and used again."""
    model_dir = model_dirs[(name, dtype)]
    rng = random.Random(99 + ord(name))
    lengths = LENGTHS[name]
    tokens, want = requests(name, model_dirs)
    schedules = {
        "whole": H.schedule_whole(lengths),
        "tail": H.schedule_tail(lengths, 70),
        "chunks": H.schedule_chunks(lengths, rng),
        "mixed": H.schedule_mixed(lengths, rng),
        "mixed2": H.schedule_mixed(dict(reversed(list(lengths.items()))), rng, max_live=3, decode_tail=40),
    }
    max_tokens = max(H.max_live_tokens(s, round_to=max(64, block_size)) for s in schedules.values())
    rp = H.LocalReplay(model_dir, dtype, max_tokens, block_size=block_size)
    worst, spread, over = {}, {}, {}
    for sname, steps in schedules.items():
        got = H.run_schedule(rp, steps, tokens, tag=sname + "/")
        worst[sname] = max(H.rel_err(got[r], want[r]) for r in tokens)
        rows = np.concatenate([np.abs(got[r].astype(np.float64) - want[r]).max(axis=1) / np.abs(want[r]).max() for r in tokens])
        keep = rows <= BF16_WORST
        over[sname] = float(1.0 - keep.mean()) if np.isfinite(rows).all() else 1.0
        g, w = np.concatenate([got[r] for r in tokens])[keep], np.concatenate([want[r] for r in tokens])[keep]
        spread[sname] = rms_err(g, w) if keep.any() else float("inf")
    assert rp.close() == 0
    # 32-bit is the sharp test.  In bfloat16 a router whose choice hangs on less than a rounding picks another expert for
    # that token than the 64-bit implementation does, so a few positions may be far off there; the others are held to a root
    # mean square.
    if dtype == "float32":
        bad = {k: v for k, v in worst.items() if not v <= H.TOLERANCE[dtype]}
    else:
        bad = {k: (over[k], spread[k]) for k in worst if not (over[k] <= BF16_OVER and spread[k] <= BF16_RMS)}
    assert not bad, f"{name} {dtype} pages of {block_size}: {bad} (largest: {worst}; over: {over}; rms: {spread})"


def test_residual_stream_layer_by_layer(model_dirs):
    """The 32-bit engine's residual stream after every run of a layer (looped layers each time) against the plain
    implementation's, a prompt in two portions and a decoded token."""
    from dinfer_b200.config.engine_config import EngineConfig
    from dinfer_b200.engine.batch import StepEntry
    from dinfer_b200.engine.runner import ModelRunner
    from dinfer_b200.parts.block import SharedNormResidual
    model_dir = model_dirs[("A", "float32")]
    cfg = C.CONFIGS["A"]
    ids = H.random_tokens(random.Random(3), 40, cfg["vocab"])
    want = []
    P.forward(cfg, C.load_weights(model_dir), ids, P.new_state(cfg), residuals=want)
    runner = ModelRunner.from_dir(model_dir, EngineConfig(max_model_len=64, max_num_seqs=2, max_num_batched_tokens=64, num_blocks=8,
                                                          block_size=16, dtype="float32", enable_cuda_graph=False))
    seen = []
    plain_forward = SharedNormResidual.forward

    def spy(self, stream, ctx, cache, next_block=None):
        plain_forward(self, stream, ctx, cache, next_block)
        seen.append(stream.x.double().cpu().clone())
    SharedNormResidual.forward = spy
    try:
        for lo, hi in ((0, 25), (25, 39), (39, 40)):
            runner.step([StepEntry("r", ids[lo:hi], [])])
    finally:
        SharedNormResidual.forward = plain_forward
    L = len(P.schedule(cfg))
    assert len(seen) == 3 * L and len(want) == L
    for i in range(L):
        got = torch.cat([seen[s * L + i] for s in range(3)])
        assert torch.allclose(got, want[i], atol=2e-4, rtol=2e-4), i


def test_block_without_a_token_side():
    """The arrangement alone: both branches stay pending and the next norm adds them; also in front of another
    arrangement's norm."""
    import dinfer_b200.models.decoder  # noqa: F401
    from dinfer_b200.parts.base import BLOCKS, NORMS, FeedForward, Mixer, ResidualStream
    width = 40

    class Twice(Mixer):
        def forward(self, x, ctx, cache):
            return 2.0 * x

    class Thrice(FeedForward):
        def forward(self, x, ctx=None, sink=None):
            return 3.0 * x
    e = env(width, torch.float32)
    norm = NORMS.get("rmsnorm")({"size": width, "eps": 1e-6, "weight": "w"}, e, "")
    norm.bind({"w": torch.ones(width, device="cuda")})
    b = BLOCKS.get("shared_norm_residual")(Twice({}, e), norm, Thrice({}, e), NORMS.get("none")({}, e, ""))
    b.configure({}, e, "")
    x = torch.randn(6, width)
    s = ResidualStream(dev(x))
    b.forward(s, None, None)
    b.forward(s, None, None)
    h = P.rms_norm(x.double(), torch.ones(width), 1e-6)
    x1 = x.double() + 5.0 * h
    want = P.rms_norm(x1 + 5.0 * P.rms_norm(x1, torch.ones(width), 1e-6), torch.ones(width), 1e-6)
    assert torch.allclose(norm.forward(s.x, delta=s.pending).double().cpu(), want, atol=1e-5)


def test_trace_runner_and_first_tokens(model_dirs, tmp_path):
    """Through ``bin/trace_run`` as a process: the first tokens of sequences (a request of one token, the first two
    positions of others), and a request that sits steps out while others come and go."""
    model_dir = model_dirs[("A", "float32")]
    cfg = C.CONFIGS["A"]
    rng = random.Random(5)
    tokens = {r: H.random_tokens(rng, n, cfg["vocab"]) for r, n in {"p": 1, "q": 2, "r": 70, "s": 45}.items()}
    oracle = Oracle(model_dir)
    rp = H.Replay(model_dir, "float32", str(tmp_path / "out"), 256)
    try:
        a = rp.step([{"id": "p", "tokens": tokens["p"], "want": [0]}, {"id": "r", "tokens": tokens["r"][:2], "want": [0, 1]}], ["p"])
        b = rp.step([{"id": "q", "tokens": tokens["q"], "want": [0, 1]}, {"id": "s", "tokens": tokens["s"][:40], "want": [39]}], ["q"])
        c = rp.step([{"id": "r", "tokens": tokens["r"][2:], "want": [67]}, {"id": "s", "tokens": tokens["s"][40:41], "want": [0]}], ["r"])
        d = rp.step([{"id": "s", "tokens": tokens["s"][41:], "want": [3]}], ["s"])
    finally:
        assert rp.close() == 0
    for got, want in ((a[0], oracle.logits(tokens["p"])[0]), (a[1:], oracle.logits(tokens["r"])[:2]),
                      (b[:2], oracle.logits(tokens["q"])), (b[2], oracle.logits(tokens["s"])[39]),
                      (c[0], oracle.logits(tokens["r"])[69]), (c[1], oracle.logits(tokens["s"])[40]),
                      (d[0], oracle.logits(tokens["s"])[44])):
        assert H.rel_err(np.asarray(got), np.asarray(want)) <= H.TOLERANCE["float32"]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "E"])
def test_greedy_generation_through_the_entry_point(model_dirs, name, dtype):
    """``LLM.generate``: scheduler, chunked prompts (a token budget below the prompts' lengths), decode steps replayed as CUDA
    graphs (token ids that are still on the device reach the token side), greedy sampling; more requests than run at once;
    long decoding over several chunks; on a pool that forces pages back into use."""
    from dinfer_b200 import LLM, SamplingParams
    model_dir = model_dirs[(name, dtype)]
    cfg = C.CONFIGS[name]
    rng = random.Random(21)
    prompts = [H.random_tokens(rng, n, cfg["vocab"]) for n in (1, 5, 23, 40, 9, 31)]
    llm = LLM(model_dir, dtype=dtype, max_model_len=160, max_num_seqs=4, max_num_batched_tokens=16, block_size=16,
              num_blocks=48)
    outs = llm.generate(prompts, SamplingParams(temperature=0.0, max_tokens=80, ignore_eos=True))
    oracle = Oracle(model_dir)
    exact = total = 0
    for p, o in zip(prompts, outs):
        assert len(o.output_ids) == 80
        lg = oracle.logits(list(p) + list(o.output_ids))
        exact += sum(int(lg[len(p) - 1 + i].argmax()) == t for i, t in enumerate(o.output_ids))
        total += 80
    assert exact >= (0.8 if dtype == "bfloat16" else 0.99) * total, (exact, total)
    assert any(isinstance(k, int) for k in llm.runner._graphs)
