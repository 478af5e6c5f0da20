"""Small Pugalix models for the tests: configurations that differ in every size and option, random weights whose
scales make every mechanism matter, and model folders written from them.

The weights are drawn in float32 and rounded to bfloat16 values, so the engine in either compute type and the plain
implementation (tests/plain_pugalix.py, in float64) start from the same numbers.  The rank of a gated linear attention's
decay is the file's: `gla(..., rank)` states it for the random weights, and `write_model` leaves it out of config.json.
"""
from __future__ import annotations

import copy
import json
import math
import os
from typing import Dict, List, Optional

import numpy as np
import torch


def attention(heads, kv_heads, dim, vdim, size=0, keep=0, rot=None, base=1000.0, scale=None, kv_from=None):
    """`size` 0: no window; `rot`: rotated entries of a head (None: no rotation)."""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale if scale is not None else dim ** -0.5}
    if size:
        m["mask"] = {"size": size, "keep_first": keep}
    if rot:
        m["rot"] = {"dims": rot, "base": base}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m}


def gla(heads, dim, vdim, tau=16.0, rank=4):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau, "rank": rank}}


def mlstm(heads, dim, vdim, cap=10.0):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}}


def layer(mixer: dict, ff: Optional[int]) -> dict:
    out = copy.deepcopy(mixer)
    out["mlp"] = {"kind": "dense", "ff": ff} if ff else None
    return out


def _config(vocab, width, layers, scale=1.0, eps=1e-5):
    return {"architecture": "Pugalix", "vocab": vocab, "width": width, "embedding": {"scale": scale}, "norm": {"eps": eps}, "layers": layers}


# A: grouped-query heads, values wider than keys, a short window that keeps 5 tokens, a reader of the first layer whose
# window is longer and keeps fewer, all three kinds, layers with and without a feed-forward
CONFIG_A = _config(101, 64, [
    layer(attention(4, 2, 16, 32, size=24, keep=5, rot=8), 48),
    layer(gla(2, 16, 24, tau=16.0, rank=4), None),
    layer(mlstm(3, 8, 16, cap=12.0), 40),
    layer(attention(4, 2, 16, 32, size=40, keep=2, rot=8, kv_from=0), None),
    layer(gla(3, 24, 8, tau=4.0, rank=7), 32),
], scale=1.7)

# B: sizes that divide by nothing (a width that is no multiple of 8, heads of 12 and 20, one key/value head), no window in
# the first attention, a window of one token with one kept token, every head entry rotated, recurrences first and last
CONFIG_B = _config(77, 100, [
    layer(mlstm(5, 20, 12, cap=5.0), None),
    layer(attention(5, 1, 12, 20, rot=12, base=50.0), 52),
    layer(gla(5, 10, 30, tau=1.0, rank=3), None),
    layer(attention(3, 3, 20, 12, size=1, keep=1, scale=0.5), None),
    layer(attention(5, 1, 12, 20, size=9, keep=0, rot=12, base=50.0, kv_from=1), 28),
], scale=0.6, eps=1e-6)

# C: heads of 64 (the tcgen05 prompt and the mma.sync decode kernel) in a window that crosses key tiles and keeps more
# tokens than a page holds, as many key/value heads as heads; wide recurrences; readers of two layers
CONFIG_C = _config(211, 128, [
    layer(attention(4, 4, 64, 64, size=70, keep=19, rot=32, base=10000.0), 96),
    layer(attention(8, 2, 64, 48, size=33, keep=3, rot=64), None),
    layer(gla(2, 64, 64, tau=8.0, rank=16), 64),
    layer(attention(4, 4, 64, 64, size=70, keep=19, rot=32, base=10000.0, kv_from=0), None),
    layer(mlstm(1, 96, 128, cap=15.0), None),
    layer(attention(8, 2, 64, 48, size=100, keep=8, rot=64, kv_from=1), 64),
], scale=3.0)

# D: recurrences alone (a model without pages)
CONFIG_D = _config(59, 72, [layer(gla(4, 12, 20, tau=2.0, rank=5), 36), layer(mlstm(2, 40, 24), None), layer(gla(1, 72, 40, tau=20.0, rank=1), None)])

CONFIGS = {"A": CONFIG_A, "B": CONFIG_B, "C": CONFIG_C, "D": CONFIG_D}


def tensor_shapes(config: dict) -> Dict[str, List[int]]:
    """Every tensor of a model of this configuration, by its name in the weight file."""
    w = config["width"]
    out = {"embed": [config["vocab"], w], "final.norm": [w], "head": [config["vocab"], w]}
    for i, l in enumerate(config["layers"]):
        p, m = f"l{i}.", l["mixer"]
        x, H, d, e = p + "mix.", m["heads"], m["dim"], m["vdim"]
        out.update({p + "norm1": [w], x + "q": [H * d, w], x + "g": [H * e, w], x + "o": [w, H * e]})
        if l["type"] == "attention":
            G = m["kv_heads"]
            out[x + "q.b"] = [H * d]
            if "kv_from" not in m:
                out.update({x + "k": [G * d, w], x + "k.b": [G * d], x + "v": [G * e, w], x + "v.b": [G * e]})
        else:
            out.update({x + "k": [H * d, w], x + "v": [H * e, w]})
            if l["type"] == "gla":
                out.update({x + "norm": [e], x + "a1": [m["rank"], w], x + "a2": [H * d, m["rank"]], x + "a2.b": [H * d]})
            else:
                out.update({x + "norm": [H * e], x + "i": [H, w], x + "i.b": [H], x + "f": [H, w], x + "f.b": [H]})
        if l["mlp"]:
            ff = l["mlp"]["ff"]
            out.update({p + "norm2": [w], p + "mlp.gate": [ff, w], p + "mlp.up": [ff, w], p + "mlp.down": [w, ff]})
    return out


def make_weights(config: dict, seed: int) -> Dict[str, torch.Tensor]:
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(config).items():
        last = name.split(".")[-1]
        n = lambda std=1.0, mean=0.0: mean + std * torch.randn(shape, generator=g)
        kind = config["layers"][int(name[1:name.index(".")])]["type"] if name[0] == "l" else ""
        if name == "embed":
            t = n(0.7)
        elif name == "head":
            t = n(1.0 / math.sqrt(shape[1]))
        elif "norm" in last:
            t = n(0.2, 1.0)
        elif name.endswith("a2.b"):
            t = n(1.0, 1.0)
        elif name.endswith("i.b"):
            t = n(1.0)
        elif name.endswith("f.b"):
            t = n(1.0, 2.5)
        elif last == "b":
            t = n(0.5)
        elif last in ("q", "k") and kind == "attention":
            t = n(1.6 / math.sqrt(shape[1]))
        elif last == "g":
            t = n(1.5 / math.sqrt(shape[1]))
        elif len(shape) == 2:
            t = n(1.2 / math.sqrt(shape[1]))
        else:
            raise ValueError(name)
        out[name] = t.to(torch.bfloat16).to(torch.float32)
    return out


def write_model(config: dict, weights: Dict[str, torch.Tensor], path: str, store=torch.bfloat16, drop_rank: bool = True) -> str:
    from sandyrt_b200.weights.safetensors import write_safetensors

    os.makedirs(path, exist_ok=True)
    on_disk = copy.deepcopy(config)
    if drop_rank:
        for l in on_disk["layers"]:
            l["mixer"].pop("rank", None)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(on_disk, f, indent=1)
    write_safetensors(os.path.join(path, "model.safetensors"), {k: v.to(store) for k, v in weights.items()})
    return path


def rel_error(got: np.ndarray, want: np.ndarray) -> float:
    """Largest over the rows of: RMS over the vocabulary of the difference (mean taken off) over the RMS of the
    wanted logits (mean taken off)."""
    got, want = np.asarray(got, dtype=np.float64), np.asarray(want, dtype=np.float64)
    d = got - want
    d = d - d.mean(-1, keepdims=True)
    w = want - want.mean(-1, keepdims=True)
    return float((np.sqrt((d ** 2).mean(-1)) / np.sqrt((w ** 2).mean(-1))).max())
