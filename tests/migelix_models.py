"""Small Migelix models for the tests: configurations that differ in every size and option, random weights whose scales make
every mechanism matter, and model folders written from them.

The weights are drawn in float32 and rounded to bfloat16 values, so the engine in either compute type and the plain
implementation (tests/plain_migelix.py, in float64) start from the same numbers.  The ranks of the low-rank products are the
file's: `wkv(..., rank)` and `delta(..., rank, gate_rank)` state them for the random weights, and `write_model` leaves them out
of config.json.
"""
from __future__ import annotations

import copy
import json
import math
import os
from typing import Dict, List, Optional

import numpy as np
import torch

RANKS = ("rank", "gate_rank")


def heads_of(heads, kv_heads, dim, size=0, rot=None, base=1000.0, yarn=None, scale=None, softcap=None):
    """An attention's record.  `size` 0: no window; `rot`: rotated entries of a head (None: no rotation); yarn: (factor, original,
    fast, slow)."""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale if scale is not None else dim ** -0.5}
    if size:
        m["mask"] = {"size": size}
    if rot:
        m["rot"] = {"dims": rot, "base": base}
        if yarn:
            m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), yarn))
    if softcap:
        m["softcap"] = softcap
    return m


def attention(heads, kv_heads, dim, softcap=30.0, **kw):
    return {"type": "attention", "mixer": heads_of(heads, kv_heads, dim, softcap=softcap, **kw)}


def delta(heads, kv_heads, dim, vdim, conv=4, rank=4, gate_rank=3):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "rank": rank, "gate_rank": gate_rank}


def parallel(left, right, left_scale=0.7, right_scale=1.4):
    return {"type": "parallel", "mixer": {"left": left, "right": right, "left_scale": left_scale, "right_scale": right_scale}}


def wkv(heads, dim, rank=4):
    return {"type": "wkv", "mixer": {"heads": heads, "dim": dim, "rank": rank}}


def layer(mixer: dict, ff: Optional[int]) -> dict:
    out = copy.deepcopy(mixer)
    out["mlp"] = {"kind": "dense", "ff": ff} if ff else None
    return out


def again(layers: list, i: int) -> dict:
    """A layer that uses layer i's tensors."""
    out = copy.deepcopy(layers[i])
    out["weights_of"] = i
    return out


def _config(vocab, width, layers, eps=1e-5, cap: Optional[float] = 20.0, reuse=()):
    layers = copy.deepcopy(layers)
    for i in reuse:
        layers.append(again(layers, i))
    out = {"architecture": "Migelix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if cap:
        out["logit_softcap"] = cap
    return out


# A: all three kinds, fewer query/key heads than heads on both sides, values wider than keys in the delta rule, short windows,
# layers with and without a feed-forward, every kind once more on another layer's tensors
CONFIG_A = _config(101, 64, [
    layer(wkv(3, 16, rank=5), 40),
    layer(attention(4, 2, 16, size=24, rot=8, softcap=6.0), None),
    layer(parallel(heads_of(6, 2, 24, size=17, rot=12, base=50.0, yarn=(4.0, 30, 8.0, 1.0)), delta(4, 2, 16, 24, conv=4, rank=6, gate_rank=5)), 48),
], reuse=(2, 0, 1))

# B: sizes that divide by nothing (a width that is no multiple of 8, heads of 12 and 20 and 10), one key/value head, no window, no
# rotation, one tap, ranks of one, no cap on the logits
CONFIG_B = _config(77, 92, [
    layer(parallel(heads_of(3, 3, 12, rot=12, base=300.0), delta(3, 1, 10, 7, conv=1, rank=1, gate_rank=1), -1.1, 0.6), None),
    layer(wkv(5, 10, rank=1), None),
    layer(attention(5, 1, 20, size=9, softcap=2.5), 52),
    layer(parallel(heads_of(5, 1, 20, size=1, scale=0.5), delta(5, 5, 20, 30, conv=3, rank=9, gate_rank=11)), 28),
], eps=1e-3, cap=None)

# C: heads of 64 and 128 (the tensor-core prompt kernels and the decode kernels for them), windows that cross key tiles, wide
# recurrences, a layer run three times
CONFIG_C = _config(211, 128, [
    layer(attention(4, 4, 64, size=70, rot=32, base=10000.0, softcap=20.0), 96),
    layer(parallel(heads_of(4, 1, 128, size=33, rot=64, yarn=(8.0, 64, 16.0, 2.0)), delta(2, 2, 64, 64, conv=4, rank=16, gate_rank=16)), 64),
    layer(wkv(2, 64, rank=16), None),
    layer(parallel(heads_of(2, 2, 64, size=100, rot=64), delta(1, 1, 96, 128, conv=2, rank=20, gate_rank=24), 1.3, 0.9), None),
], reuse=(1, 1))

# D: a recurrence alone (a model without pages)
CONFIG_D = _config(59, 72, [layer(wkv(4, 12, rank=5), 36), layer(wkv(2, 40, rank=2), None)], reuse=(0,))

CONFIGS = {"A": CONFIG_A, "B": CONFIG_B, "C": CONFIG_C, "D": CONFIG_D}


def tensor_shapes(config: dict) -> Dict[str, List[int]]:
    """Every tensor of a model of this configuration, by its name in the weight file."""
    w = config["width"]
    out = {"embed": [config["vocab"], w], "final.norm": [w]}
    for i, l in enumerate(config["layers"]):
        if l.get("weights_of") is not None:
            continue
        p, m = f"l{i}.", l["mixer"]
        x = p + "mix."
        out[p + "norm1"] = [w]

        def attention_tensors(x, a, bias):
            H, G, d = a["heads"], a["kv_heads"], a["dim"]
            out.update({x + "q": [H * d, w], x + "k": [G * d, w], x + "o": [w, H * d]})
            if bias:
                out.update({x + "q.b": [H * d], x + "k.b": [G * d]})

        if l["type"] == "attention":
            attention_tensors(x, m, False)
            out[x + "g"] = [m["heads"] * m["dim"], w]
        elif l["type"] == "parallel":
            attention_tensors(x + "left.", m["left"], True)
            out[x + "left.sink"] = [m["left"]["heads"]]
            r, y = m["right"], x + "right."
            H, G, d, e, t = r["heads"], r["kv_heads"], r["dim"], r["vdim"], r["conv"]
            out.update({y + "q": [G * d, w], y + "k": [G * d, w], y + "v": [H * e, w], y + "o": [w, H * e], y + "q.conv": [G * d, t],
                        y + "k.conv": [G * d, t], y + "v.conv": [H * e, t], y + "b": [H, w], y + "A_log": [H], y + "norm": [e],
                        y + "a1": [r["rank"], w], y + "a2": [H * d, r["rank"]], y + "dt_bias": [H * d],
                        y + "g1": [r["gate_rank"], w], y + "g2": [H * e, r["gate_rank"]]})
        else:
            H, d = m["heads"], m["dim"]
            n = H * d
            out.update({x + "mu." + s: [w] for s in "rkvgw"})
            out.update({x + s: [n, w] for s in "rkvg"})
            out.update({x + "o": [w, n], x + "w1": [m["rank"], w], x + "w2": [n, m["rank"]], x + "w0": [n], x + "u": [H, d], x + "norm": [n]})
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
        flat = lambda lo, hi: lo + (hi - lo) * torch.rand(shape, generator=g)
        if name == "embed":
            t = n(0.9)
        elif last in ("norm1", "norm2") or name == "final.norm":
            t = n(0.25)                                   # stored around zero
        elif last == "norm":
            t = n(0.2, 1.0)
        elif ".mu." in name:
            t = flat(0.0, 0.9)
        elif last == "w0":
            t = flat(-6.0, 0.5)
        elif last == "u":
            t = n(0.6, 0.4)
        elif last == "A_log":
            t = flat(-3.0, 0.5)
        elif last == "dt_bias":
            t = flat(-4.0, 1.0)
        elif last == "sink":
            t = n(1.0, 1.0)
        elif last == "conv":
            t = n(0.6, 0.3)
        elif name.endswith(".b") and len(shape) == 1:
            t = n(0.5)
        elif last in ("q", "k") and ".right." not in name:
            t = n(1.6 / math.sqrt(shape[1]))
        elif last in ("g", "g2"):
            t = n(1.5 / math.sqrt(shape[1]))
        elif len(shape) == 2:
            t = n(1.2 / math.sqrt(shape[1]))
        else:
            raise ValueError(name)
        out[name] = t.to(torch.bfloat16).to(torch.float32)
    return out


def without_ranks(config: dict) -> dict:
    out = copy.deepcopy(config)
    for l in out["layers"]:
        for m in (l["mixer"], l["mixer"].get("right", {})):
            for k in RANKS:
                m.pop(k, None)
    return out


def write_model(config: dict, weights: Dict[str, torch.Tensor], path: str, store=torch.bfloat16, drop_ranks: bool = True) -> str:
    from sandyrt_b200.weights.safetensors import write_safetensors

    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(without_ranks(config) if drop_ranks else config, f, indent=1)
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
