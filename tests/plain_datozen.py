"""Datozen written out plainly and slowly in 64-bit, one function per mechanism.  It shares no code with the package.
Every function takes the rows of one request (whole, or a piece with the state an earlier piece left) and the tensors
by their names in the weight file.

    embed               token row + position row
    rms_norm            x / sqrt(mean(x^2) + eps) * w
    stretched           frequencies of a rotation stretched by a ramp, and the factor on its cosines and sines
    turn                pairs (i, i + n/2) of a row's first n elements turned by given angles
    chunk_attention     grouped heads that see the keys of their own chunk; head norms, rotated keys, values that are
                        turned by their position and turned back at the query, a learned sink, one gate per head
    dense_ff            down(act(up h)), the activation quadratic above zero and exponential below
    choose, expert_ff   the router (groups, a correction on the choice, identity experts) and the experts
    token_side          the per-layer token input behind the feed-forward
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


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def xielu(z, p, q):
    up = softplus(p) * z * z + 0.5 * z
    low = (0.5 + softplus(q)) * (torch.exp(torch.clamp(z, max=0.0)) - 1.0 - z) + 0.5 * z
    return torch.where(z > 0, up, low)


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * w.double()


def lin(x, w):
    return x @ w.double().T


def embed(tokens: List[int], W, start: int) -> torch.Tensor:
    return torch.stack([W["embed"][t].double() + W["pos"][start + n].double() for n, t in enumerate(tokens)])


def plain_frequencies(dims: int, base: float) -> List[float]:
    return [base ** (-2.0 * i / dims) for i in range(dims // 2)]


def stretched(dims: int, base: float, s: Optional[Dict]):
    """(frequencies, the factor on cos and sin); ``s`` None: no stretching."""
    f = plain_frequencies(dims, base)
    if not s:
        return f, 1.0

    def index(turns):
        return dims * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(index(s["fast"])), 0), min(math.ceil(index(s["slow"])), dims - 1)
    out = []
    for i, v in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(v / s["factor"] * r + v * (1.0 - r))
    return out, 0.1 * math.log(s["factor"]) + 1.0


def turn(x, pos, freqs, mult=1.0, sign=1.0):
    """x [T, heads, D]: the first 2 * len(freqs) elements of a head in pairs (i, i + len(freqs)), turned by sign * pos * f."""
    n = len(freqs)
    a = pos[:, None].double() * torch.tensor(freqs, dtype=F64)[None, :] * sign
    c, s = (a.cos() * mult)[:, None, :], (a.sin() * mult)[:, None, :]
    u, v = x[..., :n], x[..., n:2 * n]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * n:]], dim=-1)


def chunk_attention(h, W, m, state, eps, at="mix."):
    """state: {"k": [tokens so far, kv_heads, dim], "v": [.., kv_heads, vdim]} (rotated keys, turned values)."""
    T = h.shape[0]
    H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    start = state["k"].shape[0]
    pos = torch.arange(start, start + T)
    q = rms_norm(lin(h, W[at + "q"]).reshape(T, H, dk), W[at + "q.norm"], eps)
    k = rms_norm(lin(h, W[at + "k"]).reshape(T, G, dk), W[at + "k.norm"], eps)
    v = lin(h, W[at + "v"]).reshape(T, G, dv)
    rot = m["rot"]
    f, mult = stretched(rot["dims"], rot["base"], rot.get("scaling"))
    q, k = turn(q, pos, f, mult), turn(k, pos, f, mult)
    fv = plain_frequencies(dv, rot["base"])
    K = state["k"] = torch.cat([state["k"], k])
    V = state["v"] = torch.cat([state["v"], turn(v, pos, fv)])
    sink = W[at + "sink"].double()
    size = m["mask"]["size"]
    out = torch.zeros(T, H, dv, dtype=F64)
    for t in range(T):
        i = start + t
        first = i // size * size                                 # the chunk's first key
        for hd in range(H):
            g = hd // (H // G)
            s = K[first:i + 1, g] @ q[t, hd] * m["scale"]
            top = max(float(s.max()), float(sink[hd]))
            e = torch.exp(s - top)
            out[t, hd] = (e / (e.sum() + torch.exp(sink[hd] - top))) @ V[first:i + 1, g]
    out = turn(out, pos, fv, sign=-1.0)
    out = out * sigmoid(lin(h, W[at + "g"]))[:, :, None]
    return lin(out.reshape(T, H * dv), W[at + "o"])


def dense_ff(h, W, at="mlp."):
    act = W[at + "act"].double()
    return lin(xielu(lin(h, W[at + "up"]), act[0], act[1]), W[at + "down"])


def gated_ff(h, W, at):
    return lin(silu(lin(h, W[at + "gate"])) * lin(h, W[at + "up"]), W[at + "down"])


def choose(z, correction, groups, top):
    """One token's router logits -> [(expert, weight)] in the order of the choice."""
    s = torch.softmax(z.double(), dim=-1)
    c = (s + correction.double()).tolist()
    n, count = len(c), groups["count"]
    size = n // count
    best = [max(c[g * size:(g + 1) * size]) for g in range(count)]
    kept = sorted(range(count), key=lambda g: (-best[g], g))[:groups["keep"]]
    open_ = [e for e in range(n) if e // size in kept]
    return [(e, float(s[e])) for e in sorted(open_, key=lambda e: (-c[e], e))[:top]]


def expert_ff(h, W, f, at="mlp."):
    r = f["router"]
    E, n = r["experts"], r["experts"] + r.get("identity", 0)
    z = lin(h, W[at + "router"])
    out = gated_ff(h, W, at + "shared.") if f.get("shared") else torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, w in choose(z[t], W[at + "correction"], r.get("groups") or {"count": 1, "keep": 1}, r["top"]):
            assert e < n
            out[t] += w * (gated_ff(h[t:t + 1], W, f"{at}e{e}.")[0] if e < E else h[t])
    return out


def token_side(x, tokens, W, layer, dim, eps, table):
    e = torch.stack([table[t, layer * dim:(layer + 1) * dim].double() for t in tokens])
    y = lin(gelu_tanh(lin(x, W["side.gate"])) * e, W["side.proj"])
    return x + rms_norm(y, W["side.norm"], eps)


def schedule(cfg) -> List[int]:
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if not lp:
        return list(range(n))
    return list(range(lp["start"])) + list(range(lp["start"], lp["stop"])) * lp["times"] + list(range(lp["stop"], n))


def new_state(cfg) -> Dict:
    runs = []
    for i in schedule(cfg):
        m = cfg["layers"][i]["mixer"]
        runs.append({"k": torch.zeros(0, m["kv_heads"], m["dim"], dtype=F64), "v": torch.zeros(0, m["kv_heads"], m["vdim"], dtype=F64)})
    return {"pos": 0, "runs": runs}


def forward(cfg, W, tokens: List[int], state, residuals: Optional[list] = None) -> torch.Tensor:
    """Logits [len(tokens), vocab] of the next piece of one request; ``state`` carries everything between pieces."""
    eps = cfg["norm"]["eps"]
    x = embed(tokens, W, state["pos"])
    state["pos"] += len(tokens)
    for i, st in zip(schedule(cfg), state["runs"]):
        l, p = cfg["layers"][i], f"l{i}."
        Wl = {k[len(p):]: v for k, v in W.items() if k.startswith(p)}
        h = rms_norm(x, Wl["norm1"], eps)
        y = chunk_attention(h, Wl, l["mixer"], st, eps)
        f = l.get("mlp")
        if f:
            y = y + (dense_ff(h, Wl) if f["kind"] == "dense" else expert_ff(h, Wl, f))
        x = token_side(x + y, tokens, Wl, i, cfg["token_side"]["dim"], eps, W["side.embed"])
        if residuals is not None:
            residuals.append(x.clone())
    return lin(rms_norm(x, W["final.norm"], eps), W["embed"])
