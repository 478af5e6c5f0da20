"""A plain, slow implementation of the Migelix design: one function per mechanism, whole sequences at once, no
cache, no batching.  It shares nothing with the engine; the tests compare the engine with it.

Everything is computed in the dtype of the tensors handed in (float64 for an oracle).  A model is
`(config, weights)`: the parsed config.json and a dict name -> tensor.

Notation: T tokens, H heads, G key/value heads, d the query/key size of a head, e its value size.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

Weights = Dict[str, torch.Tensor]

# With ROUND_PRODUCTS set, every matrix product rounds its input to bfloat16 values and, unless the caller keeps the
# result in 32-bit, its output too: what an engine that multiplies in bfloat16 with 32-bit sums does.  The tests use
# this to learn how far rounding alone moves the logits of a given model.
ROUND_PRODUCTS = False


def _bf16(x: torch.Tensor) -> torch.Tensor:
    return x.to(torch.bfloat16).to(x.dtype)


def linear(w: Weights, name: str, h: torch.Tensor, bias: bool = False, keep32: bool = False) -> torch.Tensor:
    """Weights are stored [out, in]; rows of h are tokens; the bias is the tensor `name`.b."""
    y = (_bf16(h) if ROUND_PRODUCTS else h) @ w[name].to(h.dtype).t()
    if bias:
        y = y + w[name + ".b"].to(h.dtype)
    return _bf16(y) if ROUND_PRODUCTS and not keep32 else y


# ---- small pieces ----------------------------------------------------------------------------------
def rms_norm(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def centred_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    """The stored weight is the gain's distance from one."""
    return rms_norm(x, eps) * (1.0 + w.to(x.dtype))


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def softplus(z: torch.Tensor) -> torch.Tensor:
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def unit(x: torch.Tensor) -> torch.Tensor:
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


# ---- attention -------------------------------------------------------------------------------------
def yarn(dims: int, base: float, scaling: Optional[dict]):
    """The rotation's frequencies, and the factor on both its cosine and its sine."""
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return f, 1.0
    factor, original = float(scaling["factor"]), float(scaling["original"])

    def turns(n):          # the (fractional) dimension whose wavelength fits n times into the original length
        return dims * math.log(original / (2.0 * math.pi * n)) / (2.0 * math.log(base))

    lo, hi = max(math.floor(turns(scaling["fast"])), 0), min(math.ceil(turns(scaling["slow"])), dims - 1)
    out = []
    for i, x in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(x / factor * ramp + x * (1.0 - ramp))
    return out, 0.1 * math.log(factor) + 1.0


def rotate(x: torch.Tensor, positions: torch.Tensor, dims: int, base: float, scaling: Optional[dict]) -> torch.Tensor:
    """x [T, heads, d]: neighbours (2i, 2i + 1) below `dims` turn by the angle position * f_i."""
    out = x.clone()
    freq, m = yarn(dims, float(base), scaling) if dims else ([], 1.0)
    for i, f in enumerate(freq):
        a = positions.to(x.dtype) * f
        c, s = m * torch.cos(a)[:, None], m * torch.sin(a)[:, None]
        u, v = x[:, :, 2 * i], x[:, :, 2 * i + 1]
        out[:, :, 2 * i] = u * c - v * s
        out[:, :, 2 * i + 1] = v * c + u * s
    return out


def visible(T: int, size: int) -> torch.Tensor:
    """[T, T] bool: query i sees the keys i - size + 1 .. i (size 0: 0 .. i)."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) & ((i - j < size) if size else torch.ones(T, T, dtype=torch.bool))


def attention_heads(q, k, v, scale: float, seen: torch.Tensor, softcap: float = 0.0, sink: Optional[torch.Tensor] = None) -> torch.Tensor:
    """q [T, H, d], k [T, G, d], v [T, G, e] -> [T, H, e]; head h reads key/value head h // (H / G); sink [H] or None."""
    H, G = q.shape[1], k.shape[1]
    out = []
    for h in range(H):
        g = h // (H // G)
        s = q[:, h] @ k[:, g].t() * scale
        if softcap:
            s = softcap * torch.tanh(s / softcap)
        s = s.masked_fill(~seen, float("-inf"))
        if sink is not None:
            s = torch.cat([s, sink[h].to(s.dtype).expand(s.shape[0], 1)], 1)
        p = torch.softmax(s, -1)
        out.append((p[:, :-1] if sink is not None else p) @ v[:, g])
    return torch.stack(out, dim=1)


def attention_mixer(c: dict, w: Weights, pre: str, h: torch.Tensor, bias: bool, sink: bool, gate: bool) -> torch.Tensor:
    """The values are the keys before they turn."""
    H, G, d = c["heads"], c["kv_heads"], c["dim"]
    T = h.shape[0]
    at = torch.arange(T)
    rot = c.get("rot") or {"dims": 0, "base": 1.0}
    v = linear(w, pre + "k", h, bias=bias).view(T, G, d)
    q = rotate(linear(w, pre + "q", h, bias=bias).view(T, H, d), at, rot["dims"], rot["base"], rot.get("scaling"))
    k = rotate(v, at, rot["dims"], rot["base"], rot.get("scaling"))
    size = (c.get("mask") or {"size": 0})["size"]
    o = attention_heads(q, k, v, float(c["scale"]), visible(T, size), float(c.get("softcap") or 0.0), w[pre + "sink"] if sink else None)
    o = o.reshape(T, H * d)
    if gate:
        o = o * torch.sigmoid(linear(w, pre + "g", h))
    return linear(w, pre + "o", o, keep32=True)


# ---- gated delta rule with a decay per key channel -------------------------------------------------
def short_conv(x: torch.Tensor, taps: torch.Tensor) -> torch.Tensor:
    """x [T, channels], taps [channels, n]: tap n - 1 meets the token itself; zeros before the start."""
    n = taps.shape[1]
    y = torch.zeros_like(x)
    for j in range(n):
        lag = n - 1 - j
        y[lag:] += x[: x.shape[0] - lag] * taps[:, j].to(x.dtype)
    return y


def delta_rule(q, k, v, beta, log_g, S=None):
    """One head.  q, k, log_g [T, d], v [T, e], beta [T].  S <- g S by rows; u = beta (v - S^T k); S <- S + k u^T; o = S^T q."""
    if S is None:
        S = torch.zeros(q.shape[1], v.shape[1], dtype=q.dtype)
    out = []
    for t in range(q.shape[0]):
        S = torch.exp(log_g[t])[:, None] * S
        u = beta[t] * (v[t] - S.t() @ k[t])
        S = S + torch.outer(k[t], u)
        out.append(S.t() @ q[t])
    return torch.stack(out), S


def delta_mixer(c: dict, w: Weights, pre: str, h: torch.Tensor, eps: float) -> torch.Tensor:
    H, G, d, e = c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    T = h.shape[0]
    short = lambda n: silu(short_conv(linear(w, pre + n, h), w[pre + n + ".conv"]))
    q = unit(short("q").view(T, G, d)) * d ** -0.5
    k = unit(short("k").view(T, G, d))
    v = short("v").view(T, H, e)
    beta = torch.sigmoid(linear(w, pre + "b", h, keep32=True))
    z = linear(w, pre + "a1", h, keep32=True) @ w[pre + "a2"].to(h.dtype).t() + w[pre + "dt_bias"].to(h.dtype)
    log_g = -torch.exp(w[pre + "A_log"].to(h.dtype))[None, :, None] * softplus(z).view(T, H, d)
    o = torch.stack([delta_rule(q[:, j // (H // G)], k[:, j // (H // G)], v[:, j], beta[:, j], log_g[:, j])[0] for j in range(H)], dim=1)
    o = rms_norm(o, eps) * w[pre + "norm"].to(h.dtype)
    gate = torch.sigmoid(linear(w, pre + "g2", linear(w, pre + "g1", h)))
    return linear(w, pre + "o", o.reshape(T, H * e) * gate, keep32=True)


def parallel_mixer(c: dict, w: Weights, pre: str, h: torch.Tensor, eps: float, sink: bool = True) -> torch.Tensor:
    left = attention_mixer(c["left"], w, pre + "left.", h, bias=True, sink=sink, gate=False)
    right = delta_mixer(c["right"], w, pre + "right.", h, eps)
    return float(c["left_scale"]) * left + float(c["right_scale"]) * right


# ---- time mixing -----------------------------------------------------------------------------------
def wkv_rule(r, k, v, u, log_w, S=None):
    """One head.  r, k, log_w [T, d], v [T, d], u [d].  o = (S + diag(u) k v^T)^T r, then S <- diag(w) S + k v^T."""
    if S is None:
        S = torch.zeros(r.shape[1], v.shape[1], dtype=r.dtype)
    out = []
    for t in range(r.shape[0]):
        kv = torch.outer(k[t], v[t])
        out.append((S + u[:, None] * kv).t() @ r[t])
        S = torch.exp(log_w[t])[:, None] * S + kv
    return torch.stack(out), S


def wkv_mixer(c: dict, w: Weights, pre: str, h: torch.Tensor, eps: float) -> torch.Tensor:
    H, d = c["heads"], c["dim"]
    T = h.shape[0]
    before = torch.cat([torch.zeros_like(h[:1]), h[:-1]])
    mix = {n: h + (before - h) * w[pre + "mu." + n].to(h.dtype) for n in "rkvgw"}
    r, k, v = (linear(w, pre + n, mix[n]).view(T, H, d) for n in "rkv")
    gate = silu(linear(w, pre + "g", mix["g"]))
    z = torch.tanh(linear(w, pre + "w1", mix["w"], keep32=True)) @ w[pre + "w2"].to(h.dtype).t() + w[pre + "w0"].to(h.dtype)
    log_w = -torch.exp(z).view(T, H, d)
    u = w[pre + "u"].to(h.dtype)
    o = torch.stack([wkv_rule(r[:, j], k[:, j], v[:, j], u[j], log_w[:, j])[0] for j in range(H)], dim=1)
    o = rms_norm(o, eps).reshape(T, H * d) * w[pre + "norm"].to(h.dtype)
    return linear(w, pre + "o", o * gate, keep32=True)


# ---- feed-forward, layer, model --------------------------------------------------------------------
def gated_mlp(w: Weights, pre: str, h: torch.Tensor) -> torch.Tensor:
    return linear(w, pre + "down", gelu_tanh(linear(w, pre + "gate", h)) * linear(w, pre + "up", h), keep32=True)


def tensors_of(config: dict, i: int) -> int:
    """The layer whose tensors layer i uses."""
    while config["layers"][i].get("weights_of") is not None:
        i = config["layers"][i]["weights_of"]
    return i


def run_layer(config: dict, w: Weights, i: int, x: torch.Tensor, sink: bool = True) -> torch.Tensor:
    l, p, eps = config["layers"][i], f"l{tensors_of(config, i)}.", float(config["norm"]["eps"])
    h = centred_norm(x, w[p + "norm1"], eps)
    if l["type"] == "attention":
        x = x + attention_mixer(l["mixer"], w, p + "mix.", h, bias=False, sink=False, gate=True)
    elif l["type"] == "wkv":
        x = x + wkv_mixer(l["mixer"], w, p + "mix.", h, eps)
    elif l["type"] == "parallel":
        x = x + parallel_mixer(l["mixer"], w, p + "mix.", h, eps, sink)
    else:
        raise ValueError(l["type"])
    if l.get("mlp"):
        x = x + gated_mlp(w, p + "mlp.", centred_norm(x, w[p + "norm2"], eps))
    return x


def forward_with_streams(config: dict, w: Weights, tokens: List[int], dtype=torch.float64, sink: bool = True):
    """Logits [T, vocab] and the residual stream after every layer [layers, T, width]."""
    w = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in w.items()}
    x = w["embed"][torch.tensor(tokens, dtype=torch.long)]
    streams = []
    for i in range(len(config["layers"])):
        x = run_layer(config, w, i, x, sink)
        streams.append(x)
    y = centred_norm(x, w["final.norm"], float(config["norm"]["eps"]))
    logits = linear(w, "embed", y, keep32=True)
    cap = float(config.get("logit_softcap") or 0.0)
    return (cap * torch.tanh(logits / cap) if cap else logits), torch.stack(streams)


def forward(config: dict, w: Weights, tokens: List[int], dtype=torch.float64, sink: bool = True) -> torch.Tensor:
    return forward_with_streams(config, w, tokens, dtype, sink)[0]


def forward_rounded(config: dict, w: Weights, tokens: List[int], dtype=torch.float64) -> torch.Tensor:
    """`forward` with every product's operands (and results, where an engine keeps them in 16 bits) rounded to bfloat16."""
    global ROUND_PRODUCTS
    ROUND_PRODUCTS = True
    try:
        return forward(config, w, tokens, dtype)
    finally:
        ROUND_PRODUCTS = False
