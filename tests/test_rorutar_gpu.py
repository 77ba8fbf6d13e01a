"""Rorutar on the device: every new mechanism alone against the plain implementation's function for it, then tiny models
that differ in every size replayed whole / with a decoded tail / in portions down to two tokens / mixed on a pool that only
holds the most demanding step, the trace runner as a process, and greedy generation through ``LLM``."""
import json
import os
import random

import numpy as np
import pytest
import torch

import helpers as H
import plain_rorutar as P
import rorutar_cases as C
from test_sobivik_gpu import DT, F64, PLAN, Bench, close, dev, env, i32, rms_err, rows_for, run_cut, weights_for

pytestmark = pytest.mark.gpu


# ---------------------------------------------------------------- one norm over all of q and one over all of k

@pytest.mark.parametrize("act", ["float32", "bfloat16"])
@pytest.mark.parametrize("given", ["float32", "act"])
@pytest.mark.parametrize("H_, G, D, V, rot, inter, normed, T", [
    (4, 2, 64, 64, 64, False, True, 9), (32, 8, 128, 128, 128, False, True, 3), (3, 3, 10, 6, 4, False, True, 5),
    (6, 2, 40, 48, 16, False, True, 4), (5, 1, 16, 20, 16, False, False, 7), (4, 2, 12, 20, 6, True, True, 6),
    (2, 1, 32, 32, 0, False, True, 3), (1, 1, 256, 8, 8, False, True, 2)])
def test_qkv_post_whole(act, given, H_, G, D, V, rot, inter, normed, T):
    """Norms as wide as the projections, rotation in halves and in neighbours, scaled values; rows wider than q, k, v; slots
    all over the cache, tokens that are not stored; the projected rows stay as they were."""
    from dinfer_b200.kernels import ops
    from dinfer_b200.parts.rope import rope_table
    g = torch.Generator().manual_seed(D + V + T)
    bs, eps, base, v_scale = 8, 1e-5, 500.0, -0.6
    dt, gt = DT[act], torch.float32 if given == "float32" else DT[act]
    x = (torch.randn(T, ((H_ + G) * D + G * V + 15) // 8 * 8, generator=g) * 2.0).to(gt)
    wq, wk = 1.0 + torch.randn(H_ * D, generator=g) * 0.3, 1.0 + torch.randn(G * D, generator=g) * 0.3
    pos = torch.randint(0, 400, (T,), generator=g)
    blocks = (T + bs - 1) // bs + 1
    slots = torch.randperm(blocks * bs, generator=g)[:T].to(torch.int32)
    slots[1] = -1
    table = rope_table(rot, base, 400, "cuda", 3.0) if rot else None
    cache = torch.full((blocks, 2, G, bs, max(D, V)), 7.0, dtype=dt, device="cuda")
    rows, q_out = dev(x), torch.empty(T, H_ * D, dtype=dt, device="cuda")
    ops.qkv_post_whole(rows, i32(pos.tolist()), H_, G, D, V, eps, dev(wq) if normed else None, dev(wk) if normed else None, table,
                       q_out, cache, dev(slots), bs, interleaved=inter, v_scale=v_scale)
    assert torch.equal(rows.cpu(), x)
    q, k = x[:, :H_ * D].double(), x[:, H_ * D:(H_ + G) * D].double()
    if normed:
        q, k = P.rms_norm(q, wq, eps), P.rms_norm(k, wk, eps)
    q, k = q.reshape(T, H_, D), k.reshape(T, G, D)
    if rot:
        order = torch.arange(D)
        if inter:                                            # neighbours: the same turn on elements put into halves
            order[:rot] = torch.cat([torch.arange(0, rot, 2), torch.arange(1, rot, 2)])
        back = torch.argsort(order)
        f = P.frequencies({"dims": rot, "base": base, "scaling": {"factor": 3.0}})
        q, k = P.turn(q[..., order], pos, f)[..., back], P.turn(k[..., order], pos, f)[..., back]
    v = x[:, (H_ + G) * D:(H_ + G) * D + G * V].double().reshape(T, G, V) * v_scale
    tol = dict(rtol=2e-5, atol=2e-5) if act == "float32" else dict(rtol=1e-2, atol=1e-2)
    assert torch.allclose(q_out.double().cpu().reshape(T, H_, D), q, **tol)
    c = cache.double().cpu()
    stored = torch.zeros(blocks * bs, dtype=torch.bool)
    for t in range(T):
        s = int(slots[t])
        if s < 0:
            continue
        stored[s] = True
        assert torch.allclose(c[s // bs, 0, :, s % bs, :D], k[t], **tol)
        assert torch.allclose(c[s // bs, 1, :, s % bs, :V], v[t], **tol)
    assert bool((c.permute(0, 3, 1, 2, 4)[~stored.reshape(blocks, bs)] == 7.0).all())


# ---------------------------------------------------------------- attention through its part

ATT = [  # heads, kv heads, dim, vdim, rot dims, factor, soft cap, window, kept tokens, page size
    (4, 2, 12, 20, 8, 4.0, 3.0, 7, 3, 16), (6, 1, 24, 14, 24, None, 6.0, 16, 16, 4), (3, 3, 10, 6, 2, 2.0, None, 33, 40, 16),
    (4, 1, 64, 64, 32, 8.0, 5.0, 24, 5, 16), (2, 2, 32, 32, 16, None, 4.0, 40, 17, 8), (4, 2, 128, 128, 128, 3.0, 9.0, 50, 64, 16),
    (6, 2, 64, 64, 24, None, 2.0, 1000, 3, 64), (1, 1, 96, 40, 96, 2.0, 4.0, 1, 1, 16), (2, 1, 256, 256, 64, None, 8.0, 20, 0, 16),
    (6, 2, 64, 64, 64, 2.0, 7.0, 30, 9, 16), (4, 4, 64, 64, 64, 1.5, None, None, 0, 16), (8, 2, 64, 64, 16, 1.0, 6.0, 1, 0, 8)]


def att_params(m, eps=1e-5):
    from dinfer_b200.parts.spec import PartSpec
    rope = {"head_dim": m["dim"], "rotary_dim": m["rot"]["dims"], "theta": m["rot"]["base"], "max_positions": 1024, "style": "neox",
            "scaling_factor": (m["rot"].get("scaling") or {}).get("factor", 1.0)}
    mask = m.get("mask") or {}
    return {"num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "head_dim": m["dim"], "v_dim": m["vdim"], "scale": m["scale"],
            "eps": eps, "qk_norm": True, "qk_norm_over": "all", "position": PartSpec("rope", rope), "window": mask.get("size"),
            "keep_first": mask.get("keep_first", 0), "softcap": m.get("softcap"), "sink": True, "q_proj": "mix.left.q",
            "k_proj": "mix.left.k", "v_proj": "mix.left.v", "o_proj": "mix.left.o", "q_norm": "mix.left.q.norm",
            "k_norm": "mix.left.k.norm"}


def att_state(m):
    return {"k": torch.zeros(0, m["kv_heads"], m["dim"], dtype=F64), "v": torch.zeros(0, m["kv_heads"], m["vdim"], dtype=F64)}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H_, G, D, V, rot, factor, cap, window, keep, block_size", ATT)
def test_window_attention(dtype, H_, G, D, V, rot, factor, cap, window, keep, block_size):
    """Prompts beside portions behind a history beside decoded tokens: keys and values of different widths (plain-arithmetic
    kernel) and of one width (tensor-core kernels in bfloat16), windows and kept tokens smaller and larger than a page, than
    a tile and than the request."""
    import dinfer_b200.models.decoder  # noqa: F401
    from dinfer_b200.parts.base import MIXERS
    width = 64
    m = C.attention(H_, G, D, V, 0.7 * D ** -0.5, 300.0, rot, factor, cap, window, keep)
    p = att_params(m)
    W = weights_for(MIXERS.get("gqa_attention")(p, env(width, torch.float32), "").declare(), dtype, D + V, std=0.15,
                    scale={"q.norm": 14.0, "k.norm": 8.0})
    bench = Bench("gqa_attention", p, W, dtype, width, block_size=block_size, num_blocks=4096 // block_size)
    bench.binding.kv.zero_()         # as the engine makes it: the TMA kernels fetch whole pages, and 0 * NaN is no 0
    inputs = rows_for(width, dtype, 5)
    got = run_cut(bench, inputs, PLAN)
    for r, x in inputs.items():
        close(got[r], P.window_attention(x.double(), W, m, att_state(m), 1e-5), dtype, r)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("D, window, keep", [(24, 40, 6), (64, 40, 6), (64, 130, 20), (128, 70, 1), (32, 16, 33), (64, 25, 16)])
def test_window_and_kept_edges(dtype, D, window, keep):
    """One key stands out from every other by far.  A query finds it while it is among the last ``window`` or the first
    ``keep`` keys, and not one position further; as a prompt's row, as the first row of a portion and decoded alone."""
    m = C.attention(1, 1, D, D, 1.0, 1e6, 2, None, 40.0, window, keep)
    p = att_params(m)
    p.update(scale=1.0)
    eye = torch.eye(D)
    W = {"mix.left." + n: eye for n in "qkvo"}
    W.update({"mix.left.q.norm": torch.ones(D), "mix.left.k.norm": torch.ones(D)})
    g = torch.Generator().manual_seed(D + window)
    far = window + keep + 30
    for key_at, ask in ((0, far), (keep - 1, far), (keep, far), (keep + 1, far), (far - window + 1, far), (far - window, far),
                        (far - window - 1, far), (far, far), (keep, keep + window - 1), (keep, keep + window)):
        T = far + 3
        x = torch.randn(T, D, generator=g)
        x[:, 4] = 0.0
        x[key_at] = torch.randn(D, generator=g) * 0.05
        x[key_at, 4] = 3.0                                      # after the norm this key is sqrt(D) along element 4
        x[ask] = torch.randn(D, generator=g) * 0.05
        x[ask, 4] = 3.0
        x[ask, 5] = 3.0
        x = x.to(DT[dtype]).float()
        want = P.window_attention(x.double(), W, m, att_state(m), 1e-5)
        seen = ask - key_at < window or key_at < keep
        for sizes in ([T], [ask, T - ask], [ask, 1, T - ask - 1]):
            bench = Bench("gqa_attention", p, W, dtype, D, block_size=16, num_blocks=64)
            bench.binding.kv.zero_()
            out, at = [], 0
            for n in sizes:
                out.append(bench.run([("a", x[at:at + n])]))
                at += n
            close(torch.cat(out), want, dtype, (key_at, ask, sizes))
        y = x.clone()                                           # what the key adds shows: without it the row differs
        y[key_at] = 0.01
        moved = float((P.window_attention(y.double(), W, m, att_state(m), 1e-5)[ask] - want[ask]).abs().max())
        assert (moved > 1e-3) == seen, (key_at, ask, moved)


@pytest.mark.parametrize("D, H_, G, block_size, window, keep", [
    (64, 4, 2, 16, 150, 6), (128, 8, 2, 16, 64, 70), (64, 2, 2, 64, 200, 64), (128, 4, 1, 8, 97, 1), (32, 4, 4, 4, 70, 10),
    (128, 4, 4, 16, 512, 16), (64, 6, 2, 16, 130, 200), (64, 8, 8, 16, 9, 3), (64, 4, 4, 16, 300, 0)])
@pytest.mark.parametrize("cap", [0.0, 1.2, 25.0])
def test_tensor_core_attention_with_kept_tokens(D, H_, G, block_size, window, keep, cap):
    """The tensor-core kernels (tcgen05 prompt kernels with 64- and 128-key tiles, the TMA decode kernel with its key
    splits, the mma.sync kernel) with kept first tokens, soft caps and the sink, against the plain-arithmetic kernel on the
    same cache, where the pages that no query needs are missing from the tables."""
    from dinfer_b200.kernels import attention_ops, ops
    g = torch.Generator().manual_seed(D + H_)
    scale = 0.9 * D ** -0.5
    seqs = [(0, 300), (3 * window, 1), (window - 5, 140), (0, 1), (window - 1, 1), (2 * window + keep, 60), (keep + window, 2),
            (window + 3, 1), (700, 1), (650, 90)]
    total = [a + b for a, b in seqs]
    pages = [(n + block_size - 1) // block_size for n in total]
    perm = torch.randperm(sum(pages), generator=g)
    tab = torch.full((len(seqs), max(pages)), -1, dtype=torch.int32)
    at = 0
    for b, n in enumerate(pages):
        tab[b, :n] = perm[at:at + n]
        at += n
        tab[b, (keep + block_size - 1) // block_size:max(0, seqs[b][0] - window + 1) // block_size] = -1      # given back
    cache = torch.randn(sum(pages), 2, G, block_size, D, generator=g).to(torch.bfloat16).cuda()
    T = sum(b for _, b in seqs)
    q = torch.randn(T, H_ * D, generator=g).to(torch.bfloat16).cuda()
    pos = torch.cat([torch.arange(a, a + b) for a, b in seqs]).to(torch.int32).cuda()
    cu = i32(np.concatenate([[0], np.cumsum([b for _, b in seqs])]))
    seq_lens, table = i32(total), dev(tab)
    want = torch.empty(T, H_ * D, dtype=torch.bfloat16, device="cuda")
    kw = dict(sink=True, keep_first=keep, softcap=cap)
    ops.attention_generic(q, want, cache, table, cu, pos, H_, G, D, scale, window, **kw)
    if cap == 1.2:
        other = torch.empty_like(want)
        ops.attention_generic(q, other, cache, table, cu, pos, H_, G, D, scale, window, sink=True, keep_first=keep)
        assert float((want.float() - other.float()).abs().max()) > 0.02      # the cap matters at these scores
    prompt_rows = torch.cat([torch.arange(int(cu[i]), int(cu[i + 1])) for i, (_, b) in enumerate(seqs) if b > 1]).cuda()
    decode_rows = torch.cat([torch.arange(int(cu[i]), int(cu[i + 1])) for i, (_, b) in enumerate(seqs) if b == 1]).cuda()
    group = H_ // G

    def near(got, rows, what):
        d = float((got[rows].float() - want[rows].float()).abs().max())
        assert d <= 2e-2, (what, d)

    for splits in (1, 4):
        got = torch.full_like(want, float("nan"))
        attention_ops.attention_tc(q, got, cache, table, cu, seq_lens, H_, G, D, scale, window, 300, True, True, splits, **kw)
        near(got, torch.arange(T).cuda(), f"mma.sync kernel, {splits} splits")
    if attention_ops.decode_supported(torch.bfloat16, D, group, block_size) and block_size >= 8:
        for splits in (1, 2, 8):
            got = torch.full_like(want, float("nan"))
            attention_ops.attention_decode(q, got, cache, table, cu, seq_lens, H_, G, D, scale, window, splits, **kw)
            near(got, decode_rows, f"decode kernel, {splits} splits")
    if attention_ops.umma_supported(torch.bfloat16, D, group, block_size):
        lens = [b for _, b in seqs]
        bound = attention_ops.umma_pair_bound(lens, group)
        for ks in (1, 2):
            got = torch.full_like(want, float("nan"))
            attention_ops.attention_umma(q, got, cache, table, cu, seq_lens, H_, G, D, scale, window, 300, ks, bound, **kw)
            near(got, prompt_rows, f"tcgen05 kernel, keys shared {ks} ways")
        if attention_ops.umma64_supported(torch.bfloat16, D, group, block_size):
            got = torch.full_like(want, float("nan"))
            attention_ops.attention_umma64(q, got, cache, table, cu, seq_lens, H_, G, D, scale, window, 300, bound, **kw)
            near(got, prompt_rows, "tcgen05 kernel with 64-key tiles")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("window, keep", [(0, 0), (1, 0), (5, 2), (16, 16), (9, 40), (100, 3)])
@pytest.mark.parametrize("cap", [0.0, 0.5, 30.0])
def test_plain_kernel_kept_tokens_and_caps(dtype, window, keep, cap):
    """The plain-arithmetic kernel against the softmax written out; scores far beyond the cap on both sides."""
    from dinfer_b200.kernels import ops
    g = torch.Generator().manual_seed(window)
    T, H_, G, D, bs = 60, 4, 2, 12, 8
    q, k, v = ((torch.randn(T, n, D, generator=g) * 1.7).to(DT[dtype]) for n in (H_, G, G))
    cache = torch.zeros(8, 2, G, bs, D, dtype=DT[dtype])
    for j in range(T):
        cache[j // bs, 0, :, j % bs], cache[j // bs, 1, :, j % bs] = k[j], v[j]
    got = torch.empty(T, H_ * D, dtype=DT[dtype], device="cuda")
    ops.attention_generic(dev(q.reshape(T, -1)), got, dev(cache), i32([list(range(8))]), i32([0, T]), i32(list(range(T))), H_, G, D, 0.5,
                          window, sink=True, keep_first=keep, softcap=cap)
    want = torch.zeros(T, H_, D, dtype=F64)
    for t in range(T):
        see = P.visible(t, {"size": window, "keep_first": keep} if window else None)
        for h in range(H_):
            s = k[see, h // 2].double() @ q[t, h].double() * 0.5
            if cap:
                s = cap * torch.tanh(s / cap)
            a = torch.softmax(torch.cat([s, torch.zeros(1, dtype=F64)]), 0)[:-1]
            want[t, h] = a @ v[see, h // 2].double()
    assert float((got.double().cpu() - want.reshape(T, -1)).abs().max()) <= (1e-5 if dtype == "float32" else 3e-2)


# ---------------------------------------------------------------- the state-space mixer

SSM = [  # heads, vdim, state, groups, taps, norm parts
    (6, 10, 14, 2, 4, 3), (3, 7, 5, 1, 5, 3), (4, 32, 16, 4, 3, 1), (2, 64, 128, 1, 4, 2), (8, 16, 64, 2, 2, 8), (1, 100, 9, 1, 1, 5),
    (5, 4, 200, 5, 4, 1), (4, 68, 72, 2, 6, 4), (2, 20, 300, 1, 3, 2), (12, 8, 130, 3, 4, 2)]


def ssm_params(m, eps=1e-5):
    return {"num_heads": m["heads"], "value_dim": m["vdim"], "state_dim": m["state"], "groups": m["groups"], "conv": m["conv"],
            "norm_parts": m["norm_groups"], "eps": eps, **{k: "mix.right." + v for k, v in (
                ("in_proj", "in"), ("conv_weight", "conv"), ("conv_bias", "conv.b"), ("dt_bias", "dt_bias"), ("A_log", "A_log"),
                ("D", "D"), ("norm", "norm"), ("o_proj", "o"))}}


def ssm_weights(p, dtype, width, seed):
    import dinfer_b200.models.decoder  # noqa: F401
    from dinfer_b200.parts.base import MIXERS
    W = weights_for(MIXERS.get("state_space")(p, env(width, torch.float32), "").declare(), dtype, seed, std=0.15,
                    scale={"right.conv": 3.0, "conv.b": 2.0, "dt_bias": 8.0, "right.D": 6.0, "right.norm": 7.0})
    n = W["mix.right.A_log"].numel()
    W["mix.right.A_log"] = (torch.linspace(-6.0, 2.0, n) if n > 1 else torch.tensor([-4.0])).to(torch.bfloat16).float()
    return W


def ssm_state(m):
    return P.new_mixer_state({"left": C.attention(1, 1, 2, 2, 1.0, 10.0, 2), "right": m})["right"]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads, vdim, state, groups, taps, parts", SSM)
def test_state_space(dtype, heads, vdim, state, groups, taps, parts):
    """Decoded tokens, portions shorter than the convolution and longer than a chunk, requests that sit steps out, slots that
    other requests held (which hold NaN before the first); sizes of the vector kernels and of the others."""
    width = 48
    m = C.states(heads, vdim, state, groups, taps, parts)
    p = ssm_params(m)
    W = ssm_weights(p, dtype, width, heads + state)
    bench = Bench("state_space", p, W, dtype, width)
    inputs = rows_for(width, dtype, 7)
    got = run_cut(bench, inputs, PLAN)
    for r, x in inputs.items():
        close(got[r], P.scalar_decay(x.double(), W, m, ssm_state(m), 1e-5), dtype, r)


@pytest.mark.parametrize("sizes", [[1100], [64, 64, 128, 1, 63, 780], [700] + [1] * 20 + [380], [2, 3, 65, 1030]])
def test_state_space_over_many_chunks(sizes):
    """More chunks than the walk holds in flight, portions that end at a chunk's edge, decoding behind them; heads that
    remember everything beside heads that forget at once."""
    width = 24
    m = C.states(4, 8, 12, 2, 4, 2)
    p = ssm_params(m)
    W = ssm_weights(p, "float32", width, 3)
    x = torch.randn(1100, width, generator=torch.Generator().manual_seed(1))
    bench = Bench("state_space", p, W, "float32", width, block_size=32, num_blocks=40)
    out, at = [], 0
    for n in sizes:
        out.append(bench.run([("a", x[at:at + n])]))
        at += n
    close(torch.cat(out), P.scalar_decay(x.double(), W, m, ssm_state(m), 1e-5), "float32", sizes)


def test_state_space_decays_that_change():
    """Strong decays followed by weak ones inside a chunk: the running sum of their logarithms is large where the
    differences that count are small."""
    from dinfer_b200.kernels import state_ops
    H_, G, N, V, taps, T = 2, 1, 8, 8, 1, 128
    inner, ch = H_ * V, H_ * V + 2 * G * N
    g = torch.Generator().manual_seed(2)
    proj = torch.randn(T, inner + ch + H_, generator=g)
    proj[:, -H_:] = -4.0
    proj[:20, -H_:] = 40.0                                   # a step of 40: the state is forgotten, the sum falls by hundreds
    proj[64:90:5, -H_:] = 25.0
    W = {"mix.right.in": torch.eye(inner + ch + H_), "mix.right.conv": torch.ones(ch, 1), "mix.right.conv.b": torch.zeros(ch),
         "mix.right.dt_bias": torch.zeros(H_), "mix.right.A_log": torch.tensor([2.0, 1.0]), "mix.right.D": torch.zeros(H_),
         "mix.right.norm": torch.ones(inner), "mix.right.o": torch.eye(inner)}
    state = torch.zeros(2, (H_ * N * V + 3) // 4 * 4, device="cuda")
    y = state_ops.state_space(dev(proj), dev(W["mix.right.conv"]), dev(W["mix.right.conv.b"]), dev(W["mix.right.dt_bias"]),
                              dev(W["mix.right.A_log"]), dev(W["mix.right.D"]), state, i32([0, T]), i32([0]), i32([1]), H_, G, N, V,
                              taps, any_single=False, any_portion=True, max_q_len=T)
    x, B, Cc = (P.silu(t.double()) for t in (proj[:, inner:2 * inner], proj[:, 2 * inner:2 * inner + N], proj[:, 2 * inner + N:2 * inner + 2 * N]))
    dt = P.softplus(proj[:, -H_:].double())
    S, want = torch.zeros(H_, N, V, dtype=F64), torch.zeros(T, H_, V, dtype=F64)
    for t in range(T):
        for h in range(H_):
            S[h] = torch.exp(-torch.exp(W["mix.right.A_log"][h].double()) * dt[t, h]) * S[h] + dt[t, h] * torch.outer(B[t], x[t, h * V:(h + 1) * V])
            want[t, h] = Cc[t] @ S[h]
    err = (y.double().cpu().reshape(T, H_, V) - want).abs().amax(dim=2) / want.abs().amax(dim=2).clamp(min=1e-6)
    assert float(err.max()) < 2e-5, float(err.max())
    assert torch.allclose(state[0, :H_ * N * V].double().cpu().reshape(H_, N, V), S, rtol=2e-5, atol=1e-6)


@pytest.mark.parametrize("T, parts, inner_vdim", [(1, 1, 40), (700, 8, 64), (3, 2, 1300), (650, 1, 9)])
def test_state_space_post_pads(T, parts, inner_vdim):
    """Parts a warp holds, parts a CTA holds and longer ones; columns behind the result get zeros; bfloat16 and 32-bit."""
    from dinfer_b200.kernels import state_ops
    H_, G, N, taps = 4, 2, 6, 3
    inner, ch = H_ * inner_vdim, H_ * inner_vdim + 2 * G * N
    g = torch.Generator().manual_seed(T)
    y, proj, w = torch.randn(T, inner, generator=g), torch.randn(T, inner + ch + H_, generator=g), torch.randn(inner, generator=g)
    want = P.group_norm(y.double() * P.silu(proj[:, :inner].double()), w, parts, 1e-5)
    for dt, tol in ((torch.float32, 2e-5), (torch.bfloat16, 1e-2)):
        state = torch.zeros(3, (H_ * N * inner_vdim + 2 * ch + 3) // 4 * 4, device="cuda")
        wide = torch.full((T, (inner + 7) // 8 * 8 + 16), 5.0, dtype=dt, device="cuda")
        state_ops.state_space_post(dev(y), dev(proj), dev(w), 1e-5, parts, wide[:, 8:8 + (inner + 7) // 8 * 8], state, i32([0, T]), i32([1]),
                                   i32([1]), H_, G, N, inner_vdim, taps)
        got = wide.double().cpu()
        assert torch.allclose(got[:, 8:8 + inner], want, rtol=tol, atol=tol)
        assert bool((got[:, 8 + inner:8 + (inner + 7) // 8 * 8] == 0).all()) and bool((got[:, :8] == 5.0).all()) and bool((got[:, -8:] == 5.0).all())
        hist = state[1, H_ * N * inner_vdim:][:2 * ch].cpu().reshape(2, ch)
        padded = torch.cat([torch.zeros(2, ch), proj[:, inner:inner + ch]])
        assert torch.equal(hist, padded[-2:]) and bool((state[0] == 0).all()) and bool((state[2] == 0).all())


# ---------------------------------------------------------------- the two side by side

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name, layer", [("A", 0), ("A", 1), ("B", 0), ("B", 2), ("C", 0), ("C", 1), ("D", 1), ("E", 2)])
def test_weighted_sum_of_two_mixers(dtype, name, layer):
    import dinfer_b200.models.decoder  # noqa: F401
    from dinfer_b200.config.registry import resolve_architecture
    from dinfer_b200.parts.base import MIXERS
    cfg = C.CONFIGS[name]
    m, width = cfg["layers"][layer]["mixer"], 56
    arch = resolve_architecture(cfg)
    spec = arch.build_spec(arch.parse_config(cfg)).layers[layer].mixer
    W = weights_for(MIXERS.get(spec.kind)(spec.params, env(width, torch.float32), "").declare(), dtype, layer + 5, std=0.15,
                    scale={"q.norm": 14.0, "k.norm": 8.0, "right.conv": 3.0, "dt_bias": 8.0, "right.D": 6.0, "right.norm": 7.0, "A_log": 8.0})
    bench = Bench(spec.kind, dict(spec.params), W, dtype, width)
    bench.binding.kv.zero_()
    inputs = rows_for(width, dtype, 9)
    got = run_cut(bench, inputs, PLAN)
    for r, x in inputs.items():
        close(got[r], P.two_mixers(x.double(), W, m, P.new_mixer_state(m), cfg["norm"]["eps"]), dtype, r)


def test_two_attentions_cannot_share_a_cache():
    import dinfer_b200.models.decoder  # noqa: F401
    from dinfer_b200.parts.base import MIXERS
    from dinfer_b200.parts.spec import PartSpec
    att = PartSpec("gqa_attention", {"num_heads": 2, "num_kv_heads": 1, "head_dim": 8})
    with pytest.raises(ValueError):
        MIXERS.get("parallel_mixers")({"left": att, "right": att, "scales": (1.0, 1.0)}, env(32, torch.float32), "")


# ---------------------------------------------------------------- the router and the experts

@pytest.mark.parametrize("n, count, keep, top, T", [(12, 4, 2, 3, 50), (9, 3, 1, 3, 7), (6, 6, 5, 4, 1), (8, 1, 1, 8, 33), (160, 8, 3, 6, 200),
                                                    (40, 1, 1, 1, 5), (66, 33, 4, 2, 64), (10, 5, 2, 4, 90)])
def test_route_by_the_groups_best_two(n, count, keep, top, T):
    """The chosen experts in their order, the scores over their sum; rows where the group with the best expert is not the one
    with the best two; scores so small that they round to nothing beside 1, logits so large that every score rounds to 1."""
    from dinfer_b200.kernels import moe_ops
    g = torch.Generator().manual_seed(n + T)
    z = torch.randn(T, n, generator=g) * 3
    if T > 4:
        z[1] -= 60.0
        z[2] = torch.randperm(n, generator=g).float() * (10.0 / n) + 17.0
    wide = torch.cat([z, torch.full((T, 3), 50.0)], dim=1)                    # columns behind the experts are not experts
    ids, w = moe_ops.route_choice(dev(wide), n, top, None, "sigmoid", True, count, keep, group_rank=2)
    differs = 0
    for t in range(T):
        want = P.choose(z[t], {"count": count, "keep": keep}, top)
        assert ids[t].tolist() == [e for e, _ in want], t
        assert torch.allclose(w[t].double().cpu(), torch.tensor([s for _, s in want], dtype=F64), rtol=1e-5, atol=1e-7)
        best = z[t].reshape(count, -1).amax(dim=1).topk(keep).indices
        differs += not {e // (n // count) for e, _ in want} <= set(best.tolist())
    if 1 < count < n and keep < count and T > 20:
        assert differs > 0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("E, top, count, keep, ff, limit, width, T", [
    (6, 2, 3, 2, 24, 0.7, 64, 37), (4, 1, 2, 1, 20, 1.5, 72, 5), (9, 4, 3, 2, 12, 0.4, 128, 1), (8, 3, 4, 3, 64, 1.0, 128, 700),
    (3, 3, 1, 1, 8, 2.0, 66, 20), (16, 4, 4, 2, 128, 0.9, 256, 8), (5, 2, 5, 3, 40, 0.3, 64, 300)])
def test_clamped_experts(dtype, E, top, count, keep, ff, limit, width, T):
    """The part against the plain form: gates and up sides beyond both clamps, few rows and enough for the gate in the
    epilogue of the tcgen05 grouped product (700 tokens)."""
    import dinfer_b200.models.decoder  # noqa: F401
    from dinfer_b200.parts.base import FEED_FORWARDS
    p = {"num_experts": E, "top_k": top, "groups": (count, keep), "group_rank": 2, "expert_size": ff,
         "activation": ("clamped_swish", limit, 1.702), "gated": True, "scoring": "sigmoid", "renormalize": True,
         "router": "mlp.router", "expert_gate": "mlp.e{e}.gate", "expert_up": "mlp.e{e}.up", "expert_down": "mlp.e{e}.down"}
    part = FEED_FORWARDS.get("moe")(p, env(width, DT[dtype]), "")
    W = weights_for(part.declare(), dtype, E + top, std=0.2, scale={"mlp.router": 2.0})
    part.bind({k: dev(v, DT[dtype]) for k, v in W.items()})
    x = (torch.randn(T, width, generator=torch.Generator().manual_seed(T)) * 1.5).to(DT[dtype]).float()
    got = part.forward(dev(x, DT[dtype])).double().cpu()
    f = C.moe(E, top, count, keep, ff, limit)
    want = P.expert_ff(x.double(), W, f)
    g0 = P.lin(x.double(), W["mlp.e0.gate"])
    assert bool((g0 > limit).any()) and bool((g0 < -limit).any())
    # a choice that hangs on less than a rounding of the products is not what this test is about
    z = P.lin(x.double(), W["mlp.router"])
    sure = torch.ones(T, dtype=torch.bool)
    for t in range(T):
        a = P.choose(z[t], f["router"]["groups"], top)
        for d in (1e-4, -1e-4):
            jitter = torch.where(torch.arange(E) % 2 == 0, d, -d)
            sure[t] &= {e for e, _ in a} == {e for e, _ in P.choose(z[t] + jitter, f["router"]["groups"], top)}
    assert int(sure.sum()) >= 0.9 * T
    close(got[sure], want[sure], dtype)


@pytest.mark.parametrize("T, N, K", [(5, 96, 128), (30, 512, 1024), (600, 136, 64), (100, 64, 96)])
def test_clamped_gate_in_the_products(T, N, K):
    """The clamped gate in the epilogue of the decode product (with and without split K) and of the prompt product, and as a
    kernel of its own between; values beyond both clamps."""
    from dinfer_b200.parts.linear import Linear
    g = torch.Generator().manual_seed(T)
    w = (torch.randn(2 * N, K, generator=g) * 2.0 / K ** 0.5).to(torch.bfloat16)
    x = torch.randn(T, K, generator=g).to(torch.bfloat16)
    got = Linear(dev(w)).gated_pairs(dev(x), ("clamped_swish", 1.1, 1.3)).double().cpu()
    z = x.double() @ w.double().T
    gate, up = z[:, 0::2].clamp(max=1.1), z[:, 1::2].clamp(-1.1, 1.1)
    close(got, gate * P.sigmoid(1.3 * gate) * (up + 1.0), "bfloat16")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("pairs", [True, False])
def test_clamped_gate_values(dtype, pairs):
    from dinfer_b200.kernels import ops
    vals = torch.tensor([-1e4, -60.0, -2.0, -0.5, -1e-4, 0.0, 1e-4, 0.5, 2.0, 60.0, 1e4])
    gate, up = (t.reshape(-1) for t in torch.meshgrid(vals, vals, indexing="ij"))
    for n in (gate.numel(), 112):
        a, b = gate[:n].to(DT[dtype]), up[:n].to(DT[dtype])
        x = torch.stack([a, b], dim=1).reshape(1, -1) if pairs else torch.cat([a, b]).reshape(1, -1)
        x = x.expand(3, -1).contiguous()
        got = ops.gated_act(dev(x), torch.empty(3, n, dtype=DT[dtype], device="cuda"), ("clamped_swish", 7.0, 1.702), pairs=pairs).double().cpu()
        g, u = a.double().clamp(max=7.0), b.double().clamp(-7.0, 7.0)
        tol = 2e-6 if dtype == "float32" else 5e-3
        assert torch.allclose(got, (g * P.sigmoid(1.702 * g) * (u + 1.0)).expand(3, -1), rtol=tol, atol=tol)


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
            out[(name, dt)] = C.write_model(str(tmp_path_factory.mktemp(f"rorutar{name}_{dt}")), cfg, 11 + ord(name), DT[dt])
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
    """Every position of every request: whole / with a decoded tail long enough to pass pages and windows / in portions down
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
    from dinfer_b200.parts.block import PreNormResidual
    model_dir = model_dirs[("A", "float32")]
    cfg = C.CONFIGS["A"]
    ids = H.random_tokens(random.Random(3), 40, cfg["vocab"])
    want = []
    P.forward(cfg, C.load_weights(model_dir), ids, P.new_state(cfg), residuals=want)
    runner = ModelRunner.from_dir(model_dir, EngineConfig(max_model_len=64, max_num_seqs=2, max_num_batched_tokens=64, num_blocks=8,
                                                          block_size=16, dtype="float32", enable_cuda_graph=False))
    seen = []
    plain_forward = PreNormResidual.forward

    def spy(self, stream, ctx, cache, next_block=None):
        plain_forward(self, stream, ctx, cache, next_block)
        seen.append((stream.x + stream.pending).double().cpu().clone())      # (the layer's last sum waits for the next norm)
    PreNormResidual.forward = spy
    try:
        for lo, hi in ((0, 25), (25, 39), (39, 40)):
            runner.step([StepEntry("r", ids[lo:hi], [])])
    finally:
        PreNormResidual.forward = plain_forward
    L = len(P.schedule(cfg))
    assert len(seen) == 3 * L and len(want) == L
    for i in range(L):
        got = torch.cat([seen[s * L + i] for s in range(3)])
        assert torch.allclose(got, want[i], atol=2e-4, rtol=2e-4), i


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_split_norms(model_dirs, dtype):
    """Decode steps with the norms taken apart between the mixers' output product and the next product give what the whole
    form gives (where sizes allow it: bfloat16 rows of whole 16-byte pieces)."""
    from dinfer_b200.config.engine_config import EngineConfig
    from dinfer_b200.engine.batch import StepEntry
    from dinfer_b200.engine.runner import ModelRunner
    model_dir = model_dirs[("E", dtype)]
    ids = H.random_tokens(random.Random(8), 50, C.CONFIGS["E"]["vocab"])
    outs = []
    for split in (False, True):
        runner = ModelRunner.from_dir(model_dir, EngineConfig(max_model_len=64, max_num_seqs=2, max_num_batched_tokens=64, num_blocks=8,
                                                              block_size=16, dtype=dtype, enable_cuda_graph=False, split_norms=split))
        runner.step([StepEntry("r", ids[:40], [])])
        outs.append(torch.cat([runner.step([StepEntry("r", ids[i:i + 1], [0])]).float().cpu() for i in range(40, 50)]))
    assert rms_err(outs[0].numpy(), outs[1].numpy()) <= (1e-6 if dtype == "float32" else 0.05)


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
    graphs, greedy sampling; more requests than run at once; long decoding over several windows; on a pool that forces
    pages back into use."""
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
