"""Rorutar written out plainly and slowly in 64-bit, one function per mechanism.  It shares no code with the package.
Every function takes the rows of one request (whole, or a piece with the state an earlier piece left) and the tensors
by their names in the weight file.

    embed               token row times a constant
    rms_norm            x / sqrt(mean(x^2) + eps) * w
    turn                pairs (i, i + n/2) of a head's first n elements turned by position times frequency
    visible             which keys a query sees: a window and the sequence's first tokens
    window_attention    grouped heads; one norm over all of q and one over all of k; soft-capped scores; a sink of score 0
    short_conv          causal convolution per channel with a bias and silu
    group_norm          RMS norm of equal parts of a row
    scalar_decay        the state-space mixer: one decay per head and token, written in steps of dt
    two_mixers          a weighted sum of the two
    choose, expert_ff   the router (sigmoid scores, groups by their two best, chosen scores over their sum) and the experts
    schedule            the order in which the layers run
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

F64 = torch.float64


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.log1p(torch.exp(-torch.abs(z))) + torch.clamp(z, min=0.0)


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * w.double()


def lin(x, w):
    return x @ w.double().T


def embed(tokens: List[int], table, scale: float) -> torch.Tensor:
    return torch.stack([table[t].double() for t in tokens]) * scale


def frequencies(rot: Dict) -> List[float]:
    n = rot["dims"]
    factor = (rot.get("scaling") or {}).get("factor", 1.0)
    return [rot["base"] ** (-2.0 * i / n) / factor for i in range(n // 2)]


def turn(x, pos, freqs):
    """x [T, heads, D]: the first 2 * len(freqs) elements of a head in pairs (i, i + len(freqs)), turned by pos * f."""
    n = len(freqs)
    a = pos[:, None].double() * torch.tensor(freqs, dtype=F64)[None, :]
    c, s = a.cos()[:, None, :], a.sin()[:, None, :]
    u, v = x[..., :n], x[..., n:2 * n]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * n:]], dim=-1)


def visible(i: int, mask: Optional[Dict]) -> List[int]:
    """The keys that position i sees."""
    if not mask:
        return list(range(i + 1))
    return [j for j in range(i + 1) if i - j < mask["size"] or j < mask.get("keep_first", 0)]


def window_attention(h, W, m, state, eps, at="mix.left."):
    """state: {"k": [tokens so far, kv_heads, dim], "v": [.., kv_heads, vdim]} (rotated keys)."""
    T = h.shape[0]
    H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    start = state["k"].shape[0]
    pos = torch.arange(start, start + T)
    q = rms_norm(lin(h, W[at + "q"]), W[at + "q.norm"], eps).reshape(T, H, dk)
    k = rms_norm(lin(h, W[at + "k"]), W[at + "k.norm"], eps).reshape(T, G, dk)
    v = lin(h, W[at + "v"]).reshape(T, G, dv)
    f = frequencies(m["rot"])
    q, k = turn(q, pos, f), turn(k, pos, f)
    K = state["k"] = torch.cat([state["k"], k])
    V = state["v"] = torch.cat([state["v"], v])
    cap = m.get("softcap")
    out = torch.zeros(T, H, dv, dtype=F64)
    for t in range(T):
        see = visible(start + t, m.get("mask"))
        for hd in range(H):
            g = hd // (H // G)
            s = K[see, g] @ q[t, hd] * m["scale"]
            if cap:
                s = cap * torch.tanh(s / cap)
            top = max(float(s.max()), 0.0)
            e = torch.exp(s - top)
            out[t, hd] = (e / (e.sum() + math.exp(-top))) @ V[see, g]
    return lin(out.reshape(T, H * dv), W[at + "o"])


def short_conv(x, w, bias, history):
    """x [T, C], w [C, taps] (the last column weighs the current token), history [taps - 1, C]: what came before x.
    Returns (silu(convolution + bias), the new history)."""
    T, taps = x.shape[0], w.shape[1]
    full = torch.cat([history, x])
    y = torch.zeros_like(x)
    for t in range(T):
        for j in range(taps):
            y[t] += full[t + j] * w[:, j].double()
    return silu(y + bias.double()), full[full.shape[0] - (taps - 1):]


def group_norm(y, w, parts, eps):
    T, n = y.shape
    p = y.reshape(T, parts, n // parts)
    return (p / torch.sqrt((p * p).mean(dim=-1, keepdim=True) + eps)).reshape(T, n) * w.double()


def scalar_decay(h, W, m, state, eps, at="mix.right."):
    """state: {"S": [heads, state, vdim], "conv": [taps - 1, channels]}."""
    T = h.shape[0]
    H, G, N, P = m["heads"], m["groups"], m["state"], m["vdim"]
    inner = H * P
    z, xbc, dt = torch.split(lin(h, W[at + "in"]), [inner, inner + 2 * G * N, H], dim=1)
    xbc, state["conv"] = short_conv(xbc, W[at + "conv"], W[at + "conv.b"], state["conv"])
    x, B, C = torch.split(xbc, [inner, G * N, G * N], dim=1)
    dt = softplus(dt + W[at + "dt_bias"].double())
    decay = torch.exp(-torch.exp(W[at + "A_log"].double()) * dt)
    D = W[at + "D"].double()
    y = torch.zeros(T, H, P, dtype=F64)
    S = state["S"].clone()
    for t in range(T):
        for hd in range(H):
            g = hd // (H // G)
            xt, bt, ct = x[t, hd * P:(hd + 1) * P], B[t, g * N:(g + 1) * N], C[t, g * N:(g + 1) * N]
            S[hd] = decay[t, hd] * S[hd] + dt[t, hd] * torch.outer(bt, xt)
            y[t, hd] = ct @ S[hd] + D[hd] * xt
    state["S"] = S
    y = y.reshape(T, inner) * silu(z)
    return lin(group_norm(y, W[at + "norm"], m["norm_groups"], eps), W[at + "o"])


def two_mixers(h, W, m, state, eps):
    return (m["left_scale"] * window_attention(h, W, m["left"], state["left"], eps)
            + m["right_scale"] * scalar_decay(h, W, m["right"], state["right"], eps))


def choose(z, groups, top):
    """One token's router logits -> [(expert, weight)] in the order of the choice."""
    s = sigmoid(z.double())
    v = s.tolist()
    n, count = len(v), groups["count"]
    size = n // count
    best = [sum(sorted(v[g * size:(g + 1) * size])[-2:]) for g in range(count)]
    kept = sorted(range(count), key=lambda g: (-best[g], g))[:groups["keep"]]
    open_ = [e for e in range(n) if e // size in kept]
    picked = sorted(open_, key=lambda e: (-v[e], e))[:top]
    total = sum(v[e] for e in picked) + 1e-20
    return [(e, v[e] / total) for e in picked]


def clamped_expert(h, W, at, limit):
    g = torch.clamp(lin(h, W[at + "gate"]), max=limit)
    u = torch.clamp(lin(h, W[at + "up"]), min=-limit, max=limit)
    return lin(g * sigmoid(1.702 * g) * (u + 1.0), W[at + "down"])


def expert_ff(h, W, f, at="mlp."):
    r = f["router"]
    z = lin(h, W[at + "router"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, w in choose(z[t], r.get("groups") or {"count": 1, "keep": 1}, r["top"]):
            out[t] += w * clamped_expert(h[t:t + 1], W, f"{at}e{e}.", f["expert"]["limit"])[0]
    return out


def schedule(cfg) -> List[int]:
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if not lp:
        return list(range(n))
    return list(range(lp["start"])) + list(range(lp["start"], lp["stop"])) * lp["times"] + list(range(lp["stop"], n))


def new_mixer_state(m) -> Dict:
    a, b = m["left"], m["right"]
    channels = b["heads"] * b["vdim"] + 2 * b["groups"] * b["state"]
    return {"left": {"k": torch.zeros(0, a["kv_heads"], a["dim"], dtype=F64), "v": torch.zeros(0, a["kv_heads"], a["vdim"], dtype=F64)},
            "right": {"S": torch.zeros(b["heads"], b["state"], b["vdim"], dtype=F64),
                      "conv": torch.zeros(b["conv"] - 1, channels, dtype=F64)}}


def new_state(cfg) -> Dict:
    return {"runs": [new_mixer_state(cfg["layers"][i]["mixer"]) for i in schedule(cfg)]}


def forward(cfg, W, tokens: List[int], state, residuals: Optional[list] = None) -> torch.Tensor:
    """Logits [len(tokens), vocab] of the next piece of one request; ``state`` carries everything between pieces."""
    eps = cfg["norm"]["eps"]
    x = embed(tokens, W["embed"], (cfg.get("embedding") or {}).get("scale", 1.0))
    for i, st in zip(schedule(cfg), state["runs"]):
        l, p = cfg["layers"][i], f"l{i}."
        Wl = {k[len(p):]: v for k, v in W.items() if k.startswith(p)}
        x = x + two_mixers(rms_norm(x, Wl["norm1"], eps), Wl, l["mixer"], st, eps)
        if l.get("mlp"):
            x = x + expert_ff(rms_norm(x, Wl["norm2"], eps), Wl, l["mlp"])
        if residuals is not None:
            residuals.append(x.clone())
    return lin(rms_norm(x, W["final.norm"], eps), W["head"])
