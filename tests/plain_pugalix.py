"""A plain, slow implementation of the Pugalix design: one function per mechanism, whole sequences at once, no
cache, no batching.  It shares nothing with the engine; the tests compare the engine with it.

Everything is computed in the dtype of the tensors handed in (float64 for an oracle).  A model is
`(config, weights)`: the parsed config.json and a dict name -> tensor.

Notation: T tokens, H heads, G key/value heads, d the query/key size of a head, e its value size.
"""
from __future__ import annotations

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
def rms_norm(x: torch.Tensor, gain: Optional[torch.Tensor], eps: float) -> torch.Tensor:
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if gain is None else y * gain.to(x.dtype)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def log_sigmoid(z: torch.Tensor) -> torch.Tensor:
    return torch.clamp(z, max=0.0) - torch.log1p(torch.exp(-z.abs()))


# ---- attention -------------------------------------------------------------------------------------
def rotate(x: torch.Tensor, positions: torch.Tensor, dims: int, base: float) -> torch.Tensor:
    """x [T, heads, d]: neighbours (2i, 2i + 1) below `dims` turn by the angle position * base^(-2i / dims)."""
    out = x.clone()
    for i in range(dims // 2):
        a = positions.to(x.dtype) * float(base) ** (-2.0 * i / dims)
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        u, v = x[:, :, 2 * i], x[:, :, 2 * i + 1]
        out[:, :, 2 * i] = u * c - v * s
        out[:, :, 2 * i + 1] = v * c + u * s
    return out


def visible(T: int, size: int, keep_first: int) -> torch.Tensor:
    """[T, T] bool: query i sees key j when j is not behind i and lies among the last `size` positions (0: all of them)
    or among the first `keep_first` of the sequence."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    near = (i - j < size) if size else torch.ones(T, T, dtype=torch.bool)
    return (j <= i) & (near | (j < keep_first))


def softmax_with_one(s: torch.Tensor) -> torch.Tensor:
    """exp(s_j) / (1 + sum exp(s_j)) over the last axis; -inf marks what is not seen."""
    m = torch.clamp(s.max(-1, keepdim=True).values, min=0.0)
    p = torch.exp(s - m)
    return p / (torch.exp(-m) + p.sum(-1, keepdim=True))


def attention_heads(q, k, v, scale: float, seen: torch.Tensor, sink: bool = True) -> torch.Tensor:
    """q [T, H, d], k [T, G, d], v [T, G, e] -> [T, H, e]; head h reads key/value head h // (H / G)."""
    H, G = q.shape[1], k.shape[1]
    out = []
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].t() * scale).masked_fill(~seen, float("-inf"))
        p = softmax_with_one(s) if sink else torch.softmax(s, -1)
        out.append(p @ v[:, g])
    return torch.stack(out, dim=1)


def attention_mixer(c: dict, w: Weights, pre: str, h: torch.Tensor, kept: Dict[int, tuple], layer: int, sink: bool = True) -> torch.Tensor:
    """`kept`: layer -> (rotated keys, values) of the layers run so far; a layer with kv_from reads another's."""
    H, G, d, e = c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    T = h.shape[0]
    at = torch.arange(T)
    rot = c.get("rot") or {"dims": 0, "base": 1.0}
    q = rotate(linear(w, pre + "q", h, bias=True).view(T, H, d), at, rot["dims"], rot["base"])
    if c.get("kv_from") is None:
        k = rotate(linear(w, pre + "k", h, bias=True).view(T, G, d), at, rot["dims"], rot["base"])
        kept[layer] = (k, linear(w, pre + "v", h, bias=True).view(T, G, e))
    k, v = kept[layer if c.get("kv_from") is None else c["kv_from"]]
    mask = c.get("mask") or {"size": 0, "keep_first": 0}
    o = attention_heads(q, k, v, float(c["scale"]), visible(T, mask["size"], mask["keep_first"]), sink)
    o = o.reshape(T, H * e) * torch.sigmoid(linear(w, pre + "g", h))
    return linear(w, pre + "o", o, keep32=True)


# ---- gated linear attention ------------------------------------------------------------------------
def gla_rule(q, k, v, log_alpha, S=None):
    """One head.  q, k, log_alpha [T, d], v [T, e].  Token by token: row i of S fades by its own factor, then the token's
    outer product is added, then read: S <- diag(alpha) S + k v^T;  o = S^T q."""
    if S is None:
        S = torch.zeros(q.shape[1], v.shape[1], dtype=q.dtype)
    out = []
    for t in range(q.shape[0]):
        S = torch.exp(log_alpha[t])[:, None] * S + torch.outer(k[t], v[t])
        out.append(S.t() @ q[t])
    return torch.stack(out), S


def gla_mixer(c: dict, w: Weights, pre: str, h: torch.Tensor, eps: float) -> torch.Tensor:
    H, d, e = c["heads"], c["dim"], c["vdim"]
    T = h.shape[0]
    q = (linear(w, pre + "q", h) * d ** -0.5).view(T, H, d)
    k = linear(w, pre + "k", h).view(T, H, d)
    v = linear(w, pre + "v", h).view(T, H, e)
    z = linear(w, pre + "a1", h, keep32=True) @ w[pre + "a2"].to(h.dtype).t() + w[pre + "a2.b"].to(h.dtype)
    log_alpha = (log_sigmoid(z) / float(c["tau"])).view(T, H, d)
    o = torch.stack([gla_rule(q[:, j], k[:, j], v[:, j], log_alpha[:, j])[0] for j in range(H)], dim=1)
    o = rms_norm(o, w[pre + "norm"], eps).reshape(T, H * e)
    return linear(w, pre + "o", o * silu(linear(w, pre + "g", h)), keep32=True)


# ---- matrix memory (mLSTM) -------------------------------------------------------------------------
def mlstm_rule(q, k, v, log_i, log_f, state=None):
    """One head.  q, k [T, d], v [T, e], log_i, log_f [T].  The state (S [d, e], n [d], m) starts as zeros, m included:
        m' = max(log_f + m, log_i);  S, n fade by exp(log_f + m - m') and take exp(log_i - m') k v^T and exp(log_i - m') k;
        o = S^T q / (max(|n . q|, exp(-m')) + 1e-6)."""
    dt = q.dtype
    S, n, m = state or (torch.zeros(q.shape[1], v.shape[1], dtype=dt), torch.zeros(q.shape[1], dtype=dt), torch.zeros((), dtype=dt))
    out = []
    for t in range(q.shape[0]):
        m2 = torch.maximum(log_f[t] + m, log_i[t])
        fade, take = torch.exp(log_f[t] + m - m2), torch.exp(log_i[t] - m2)
        S, n, m = fade * S + take * torch.outer(k[t], v[t]), fade * n + take * k[t], m2
        out.append(S.t() @ q[t] / (torch.maximum((n @ q[t]).abs(), torch.exp(-m)) + 1e-6))
    return torch.stack(out), (S, n, m)


def mlstm_mixer(c: dict, w: Weights, pre: str, h: torch.Tensor, eps: float) -> torch.Tensor:
    H, d, e, cap = c["heads"], c["dim"], c["vdim"], float(c["gate_cap"])
    T = h.shape[0]
    q = (linear(w, pre + "q", h) * d ** -0.5).view(T, H, d)
    k = linear(w, pre + "k", h).view(T, H, d)
    v = linear(w, pre + "v", h).view(T, H, e)
    log_i = cap * torch.tanh(linear(w, pre + "i", h, bias=True, keep32=True) / cap)
    log_f = log_sigmoid(cap * torch.tanh(linear(w, pre + "f", h, bias=True, keep32=True) / cap))
    o = torch.stack([mlstm_rule(q[:, j], k[:, j], v[:, j], log_i[:, j], log_f[:, j])[0] for j in range(H)], dim=1)
    o = rms_norm(o, None, eps).reshape(T, H * e) * w[pre + "norm"].to(h.dtype)
    return linear(w, pre + "o", o * torch.sigmoid(linear(w, pre + "g", h)), keep32=True)


# ---- feed-forward, layer, model --------------------------------------------------------------------
def gated_mlp(w: Weights, pre: str, h: torch.Tensor) -> torch.Tensor:
    return linear(w, pre + "down", silu(linear(w, pre + "gate", h)) * linear(w, pre + "up", h), keep32=True)


def run_layer(config: dict, w: Weights, i: int, x: torch.Tensor, kept: Dict[int, tuple], sink: bool = True) -> torch.Tensor:
    l, p, eps = config["layers"][i], f"l{i}.", float(config["norm"]["eps"])
    h = rms_norm(x, w[p + "norm1"], eps)
    if l["type"] == "attention":
        x = x + attention_mixer(l["mixer"], w, p + "mix.", h, kept, i, sink)
    elif l["type"] == "gla":
        x = x + gla_mixer(l["mixer"], w, p + "mix.", h, eps)
    elif l["type"] == "mlstm":
        x = x + mlstm_mixer(l["mixer"], w, p + "mix.", h, eps)
    else:
        raise ValueError(l["type"])
    if l.get("mlp"):
        x = x + gated_mlp(w, p + "mlp.", rms_norm(x, w[p + "norm2"], eps))
    return x


def forward_with_streams(config: dict, w: Weights, tokens: List[int], dtype=torch.float64, sink: bool = True):
    """Logits [T, vocab] and the residual stream after every layer [layers, T, width]."""
    w = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in w.items()}
    x = w["embed"][torch.tensor(tokens, dtype=torch.long)] * float(config["embedding"]["scale"])
    kept: Dict[int, tuple] = {}
    streams = []
    for i in range(len(config["layers"])):
        x = run_layer(config, w, i, x, kept, sink)
        streams.append(x)
    y = rms_norm(x, w["final.norm"], float(config["norm"]["eps"]))
    return linear(w, "head", y, keep32=True), torch.stack(streams)


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
