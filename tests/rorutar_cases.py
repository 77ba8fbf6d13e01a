"""Tiny Rorutar configurations for the tests.  They differ from one another in every size and option, layer by layer too,
and use values that are easy to confuse when they happen to be equal or 1: values wider and narrower than keys, one key
head, as many key heads as heads, a rotation of the whole head and of a part, scaled positions and not, windows of one token,
smaller than a page, across pages and none at all, no kept tokens, kept tokens that fill pages and more of them than the
window, no soft cap, convolutions of one to five taps, one group for all heads and a group per head, norms over the whole row
and in many parts, states that no vector load divides, scales of 1 and below 0, groups of experts that all stay, a single one
that stays, groups of one expert, layers without feed-forward, loops at the start, in the middle, at the end and none."""
from __future__ import annotations

import json
import os
from typing import Dict

import torch


def attention(heads, kv_heads, dim, vdim, scale, base, rot, factor=None, softcap=None, window=None, keep=0):
    r = {"base": base, "dims": rot}
    if factor is not None:
        r["scaling"] = {"factor": factor}
    d = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": r}
    if softcap is not None:
        d["softcap"] = softcap
    if window is not None:
        d["mask"] = {"size": window, "keep_first": keep}
    return d


def states(heads, vdim, state, groups, conv, norm_groups):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}


def moe(experts, top, count, keep, ff, limit):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit},
            "router": {"experts": experts, "top": top, "groups": {"count": count, "keep": keep}}}


def layer(left, right, left_scale, right_scale, mlp):
    return {"type": "parallel", "mixer": {"left": left, "right": right, "left_scale": left_scale, "right_scale": right_scale},
            "mlp": mlp}


def model(vocab, width, eps, embedding_scale, layers, loop=None):
    d = {"architecture": "Rorutar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": embedding_scale},
         "layers": layers}
    if loop:
        d["loop"] = dict(zip(("start", "stop", "times"), loop))
    return d


# values wider than keys, windows that cross pages, kept tokens, a loop in the middle, a layer without feed-forward
RORUTAR_A = model(300, 64, 1e-5, 3.0, [
    layer(attention(4, 2, 12, 20, 0.5, 300.0, 8, 4.0, 3.0, 7, 3), states(6, 10, 14, 2, 4, 3), 0.7, 1.2, moe(6, 2, 3, 2, 24, 0.6)),
    layer(attention(6, 3, 16, 10, 0.3, 1000.0, 16, None, 8.0, 24, 18), states(3, 8, 20, 3, 2, 1), 1.0, 0.5, moe(8, 3, 2, 1, 20, 1.5)),
    layer(attention(2, 1, 20, 6, 0.7, 50.0, 4, 2.5, None, 40, 0), states(4, 16, 6, 1, 3, 4), 1.5, -0.4, None),
    layer(attention(5, 5, 8, 8, 0.4, 10000.0, 6, 8.0, 5.0), states(2, 12, 33, 2, 1, 6), 0.3, 1.0, moe(4, 4, 4, 4, 12, 1.0))], loop=(1, 3, 2))
# heads the tensor-core attention takes, one key head, more kept tokens than the window, a loop from the first layer on
RORUTAR_B = model(515, 128, 3e-6, 9.0, [
    layer(attention(4, 1, 64, 64, 0.2, 2000.0, 64, 3.0, 6.0, 21, 30), states(4, 32, 16, 2, 4, 2), 0.5, 0.8, moe(9, 2, 3, 2, 32, 2.0)),
    layer(attention(2, 2, 32, 32, 0.3, 500.0, 16, None, 12.0, 50, 5), states(8, 16, 24, 4, 3, 8), 1.1, 1.0, moe(5, 3, 1, 1, 48, 0.5)),
    layer(attention(4, 2, 128, 128, 0.12, 3000.0, 32, 1.5, 4.0, 64, 16), states(2, 64, 40, 1, 2, 2), 0.9, 0.6, moe(12, 2, 6, 2, 56, 3.0))],
    loop=(0, 2, 2))
# sizes nothing divides; a window of one token; no loop
RORUTAR_C = model(331, 72, 1e-6, 1.0, [
    layer(attention(3, 3, 10, 6, 1.1, 77.0, 10, 7.0, 2.0, 1, 1), states(3, 7, 5, 1, 5, 3), 1.0, 1.0, moe(7, 4, 1, 1, 12, 0.8)),
    layer(attention(6, 2, 22, 14, 0.6, 400.0, 2, 1.25, 9.0, 17, 2), states(5, 9, 11, 5, 3, 5), 0.8, 0.9, moe(10, 3, 5, 2, 20, 1.2)),
    layer(attention(1, 1, 6, 18, 0.9, 90.0, 4, None, 1.5, 33, 17), states(1, 15, 9, 1, 4, 1), 0.6, 0.7, None)])
RORUTAR_D = model(257, 100, 2e-6, 5.5, [
    layer(attention(5, 1, 14, 14, 0.8, 60.0, 6, None, 4.0, 5, 4), states(6, 4, 3, 3, 2, 2), 0.45, 1.3, moe(6, 1, 2, 2, 20, 0.7)),
    layer(attention(2, 2, 34, 30, 0.25, 5000.0, 20, 16.0, 7.0, 50, 1), states(2, 40, 8, 1, 4, 4), 1.2, 0.35, moe(8, 2, 4, 1, 36, 5.0))],
    loop=(1, 2, 4))
# sizes of real layers in small: heads of 128 and 64, states of 64 x 64 and 128 x 32, sixteen experts
RORUTAR_E = model(400, 384, 5e-6, 7.0, [
    layer(attention(8, 2, 64, 64, 0.15, 8000.0, 64, 4.0, 10.0, 100, 4), states(8, 64, 64, 2, 4, 2), 0.55, 0.75, moe(16, 4, 4, 2, 64, 2.5)),
    layer(attention(4, 2, 128, 128, 0.1, 20000.0, 128, None, 15.0, 80, 64), states(12, 32, 128, 4, 4, 4), 0.8, 0.8, moe(16, 3, 8, 3, 48, 1.0)),
    layer(attention(6, 3, 64, 128, 0.12, 700.0, 48, 2.0, 6.0, 130, 9), states(4, 96, 48, 1, 3, 1), 0.65, 1.0, moe(14, 4, 2, 1, 48, 4.0))],
    loop=(0, 3, 2))
CONFIGS = {"A": RORUTAR_A, "B": RORUTAR_B, "C": RORUTAR_C, "D": RORUTAR_D, "E": RORUTAR_E}


def shape_weight(name: str, t: torch.Tensor, sharp: float = 2.0) -> torch.Tensor:
    """Random weights changed so that faults show: query norms scaled (a token's attention then rests on few keys: a key lost
    or one too many moves the logits), decays from a token's memory to hundreds of tokens', step sizes around one, strong
    taps, routers sharp enough that the chosen scores differ, expert inputs that pass the clamps."""
    if name.endswith(".q.norm"):
        return t * sharp
    if name.endswith("A_log"):
        return torch.linspace(-5.0, 1.5, t.numel()).reshape(t.shape) + t
    if name.endswith("dt_bias"):
        return t * 10.0 - 0.5
    if name.endswith((".conv", ".conv.b")):
        return t * 6.0
    if name.endswith("right.D"):
        return t * 0.7
    if name.endswith("mlp.router"):
        return t * (48.0 / t.shape[1] ** 0.5)
    if name.endswith((".gate", ".up")) and ".mlp.e" in name:
        return t * (16.0 / t.shape[1] ** 0.5)
    if name == "embed":
        return t * 4.0
    return t


def write_model(path: str, cfg: dict, seed: int, dtype: torch.dtype, std: float = 0.08) -> str:
    from dinfer_b200.weights.random_init import model_declarations, random_tensor
    from dinfer_b200.weights.safetensors_io import write_safetensors
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    tensors = [(d.name, shape_weight(d.name, random_tensor(d, seed, std, 0.3, torch.float32)).to(torch.bfloat16).to(dtype))
               for d in model_declarations(cfg)]             # the same values in every dtype
    write_safetensors(os.path.join(path, "model.safetensors"), tensors, metadata={"format": "pt"})
    return path


def load_weights(model_dir: str) -> Dict[str, torch.Tensor]:
    from safetensors.torch import load_file
    return load_file(os.path.join(model_dir, "model.safetensors"))
