"""Tiny Datozen configurations for the tests.  They differ from one another in every size and option, layer by layer too,
and use values that are easy to confuse when they happen to be equal or 1: values wider and narrower than keys, one key
head, as many key heads as heads, a rotation of the whole head and of a part, stretched (also by a ramp without width) and
not, chunks smaller than a page, of a page's size and longer than every request, loops of one and of several layers at the
start, in the middle, at the end and none, layers without feed-forward, experts without identity experts, groups that all
stay and a single one that stays, sizes no vector load or tensor-core tile divides, and sizes the tensor-core kernels take."""
from __future__ import annotations

import json
import os
from typing import Dict

import torch


def attention(heads, kv_heads, dim, vdim, chunk, base, rot, scale, scaling=None):
    r = {"base": base, "dims": rot}
    if scaling:
        r["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
                                           "rot": r, "mask": {"size": chunk}}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, identity, top, groups, keep, ff, shared=0):
    d = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "identity": identity, "top": top,
                                                         "groups": {"count": groups, "keep": keep}}}
    if shared:
        d["shared"] = {"ff": shared}
    return d


def layer(mixer, mlp):
    return dict(mixer, mlp=mlp)


def model(vocab, width, eps, max_positions, side, layers, loop=None):
    d = {"architecture": "Datozen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "max_positions": max_positions,
         "token_side": {"dim": side}, "layers": layers}
    if loop:
        d["loop"] = dict(zip(("start", "stop", "times"), loop))
    return d


# values wider than keys, chunks that cross pages, a loop in the middle, groups that split the identity experts
DATOZEN_A = model(300, 64, 1e-5, 400, 12, [
    layer(attention(4, 2, 12, 20, 7, 300.0, 8, 0.5, (4.0, 40.0, 6.0, 1.0)), dense(48)),
    layer(attention(6, 3, 16, 10, 24, 1000.0, 16, 0.3), moe(6, 3, 2, 3, 2, 24, 40)),
    layer(attention(2, 1, 20, 6, 40, 50.0, 4, 0.7, (2.5, 64.0, 3.0, 3.0)), None),
    layer(attention(5, 5, 8, 8, 33, 10000.0, 6, 0.4, (8.0, 30.0, 20.0, 0.5)), moe(4, 0, 1, 2, 1, 20))], loop=(1, 3, 3))
# heads the tensor-core attention takes, one key head, a loop from the first layer on, all groups kept
DATOZEN_B = model(515, 128, 3e-6, 512, 16, [
    layer(attention(4, 1, 64, 64, 48, 2000.0, 64, 0.2, (6.0, 90.0, 8.0, 1.5)), moe(5, 1, 3, 2, 2, 32)),
    layer(attention(2, 2, 32, 32, 21, 500.0, 16, 0.3), dense(96)),
    layer(attention(4, 2, 128, 128, 64, 3000.0, 32, 0.12), dense(56))], loop=(0, 2, 2))
# sizes nothing divides; no loop; chunks of a page's size and of one token more; a loop of the last layer in D
DATOZEN_C = model(331, 72, 1e-6, 300, 5, [
    layer(attention(3, 3, 10, 6, 16, 77.0, 10, 1.1), dense(28)),
    layer(attention(6, 2, 22, 14, 17, 400.0, 2, 0.6, (3.0, 25.0, 2.0, 0.7)), moe(7, 2, 4, 3, 2, 12, 20)),
    layer(attention(1, 1, 6, 18, 1000, 90.0, 4, 0.9), None)])
DATOZEN_D = model(257, 100, 2e-6, 260, 9, [
    layer(attention(5, 1, 14, 14, 5, 60.0, 6, 0.8), moe(2, 2, 2, 4, 3, 20, 12)),
    layer(attention(2, 2, 34, 30, 50, 5000.0, 20, 0.25, (5.0, 128.0, 10.0, 2.0)), dense(36))], loop=(1, 2, 4))
# sizes of real layers in small: heads of 128 and 64, eight experts and two identity experts
DATOZEN_E = model(400, 384, 5e-6, 640, 24, [
    layer(attention(8, 2, 64, 64, 100, 8000.0, 32, 0.15, (8.0, 200.0, 16.0, 1.0)), dense(448)),
    layer(attention(4, 2, 128, 128, 80, 20000.0, 128, 0.1), moe(8, 2, 3, 5, 3, 64, 96)),
    layer(attention(6, 3, 64, 128, 130, 700.0, 48, 0.12), moe(14, 2, 4, 4, 2, 48))], loop=(0, 3, 2))
CONFIGS = {"A": DATOZEN_A, "B": DATOZEN_B, "C": DATOZEN_C, "D": DATOZEN_D, "E": DATOZEN_E}


def write_model(path: str, cfg: dict, seed: int, dtype: torch.dtype, sharp: float = 2.0, std: float = 0.08) -> str:
    """Random weights shaped so that faults show: the query norms scaled by ``sharp`` (a token's attention then rests on few
    keys: a key lost or one too many moves the logits), sinks of different sizes that take a good part of the softmax,
    corrections that change the choice, routers sharp enough that the chosen scores differ, position rows and token
    inputs large enough to matter."""
    from dinfer_b200.weights.random_init import model_declarations, random_tensor
    from dinfer_b200.weights.safetensors_io import write_safetensors
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    tensors = []
    for d in model_declarations(cfg):
        t = random_tensor(d, seed, std, 0.3, torch.float32)
        n = d.name
        if n.endswith("mix.q.norm"):
            t = t * sharp
        elif n.endswith("mix.sink"):
            t = t * 20.0 + 1.0
        elif n.endswith("mlp.correction"):
            t = t * 4.0 - 0.6
        elif n.endswith("mlp.act"):
            t = t * 10.0
        elif n.endswith("mlp.router"):
            t = t * 6.0
        elif n in ("pos", "side.embed", "embed"):
            t = t * 8.0
        elif n.endswith(("side.gate", "side.proj")):
            t = t * 2.0
        tensors.append((n, t.to(torch.bfloat16).to(dtype)))     # the same values in every dtype
    write_safetensors(os.path.join(path, "model.safetensors"), tensors, metadata={"format": "pt"})
    return path


def load_weights(model_dir: str) -> Dict[str, torch.Tensor]:
    from safetensors.torch import load_file
    return load_file(os.path.join(model_dir, "model.safetensors"))
