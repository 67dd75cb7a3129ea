"""Plain, slow restatement of the Sirodra design in float64 PyTorch on the CPU — the yardstick the CUDA path is held against.

One function per mechanism, written from the design's equations; it shares no code with the product path (it reads the raw
config dictionary and the checkpoint's tensor names directly) and keeps no cache: a sequence is always recomputed whole.

Notation: T tokens at positions 0 .. T-1, W[name] the checkpoint tensor `name` as float64, linear weights [out, in].
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

F64 = torch.float64


# ---- element-wise pieces and norms -----------------------------------------------------------------------------------------
def sigmoid(z: torch.Tensor) -> torch.Tensor:
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * sigmoid(z)


def log_sigmoid(z: torch.Tensor) -> torch.Tensor:
    """log(1 / (1 + e^-z)) without overflow on either side."""
    return torch.minimum(z, torch.zeros_like(z)) - torch.log1p(torch.exp(-z.abs()))


def gelu_erf(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def soft_cap(z: torch.Tensor, cap: float) -> torch.Tensor:
    return cap * torch.tanh(z / cap)


def rms_unit(v: torch.Tensor, eps: float) -> torch.Tensor:
    """v / sqrt(mean(v^2) + eps) over the last axis."""
    return v / torch.sqrt((v * v).mean(-1, keepdim=True) + eps)


def centred_norm(v: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    """Layer norm with a weight and no bias: (v - mean) / sqrt(mean((v - mean)^2) + eps) * w."""
    d = v - v.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w


# ---- rotary positions ----------------------------------------------------------------------------------------------------------
def rotate(v: torch.Tensor, dims: int, base: float, factor: float = 1.0) -> torch.Tensor:
    """v [T, heads, n]: among the first `dims` entries of every head, entries (2i, 2i + 1) turn at position t by the angle
    t * base^(-2i/dims) / factor; entries from `dims` on pass unchanged."""
    out = v.clone()
    for i in range(dims // 2):
        ang = torch.arange(v.shape[0], dtype=F64) * (base ** (-2.0 * i / dims) / factor)
        c, s = torch.cos(ang)[:, None], torch.sin(ang)[:, None]
        a, b = v[..., 2 * i], v[..., 2 * i + 1]
        out[..., 2 * i], out[..., 2 * i + 1] = a * c - b * s, b * c + a * s
    return out


# ---- softmax attention over a window of tokens and the pooled blocks before it ----------------------------------------------------
def visible(i: int, window: int, pool: int):
    """What position i attends to: (first token, number of pooled blocks).  Tokens first .. i lie in the window; block b (positions
    b pool .. b pool + pool - 1) counts when its last position has left the window."""
    first = max(0, i - window + 1) if window > 0 else 0
    blocks = 0
    while window > 0 and pool > 0 and blocks * pool + pool - 1 <= i - window:
        blocks += 1
    return first, blocks


def attention(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    """h [T, width].  Query head a reads key / value head a // (H / G); queries and keys turn, then are divided by their root mean
    square; tokens of the window and pooled blocks share one softmax; every head's output is multiplied by a sigmoid gate."""
    T = h.shape[0]
    H, G, d, dv, scale = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["scale"]
    mask = m.get("mask") or {}
    window, pool = mask.get("size", 0), mask.get("pool", 0)
    q = (h @ W[p + "q"].T + W[p + "q.b"]).reshape(T, H, d)
    k = (h @ W[p + "k"].T + W[p + "k.b"]).reshape(T, G, d)
    v = (h @ W[p + "v"].T + W[p + "v.b"]).reshape(T, G, dv)
    rot = m.get("rot")
    if rot:
        factor = (rot.get("scaling") or {}).get("factor", 1.0)
        q, k = rotate(q, rot["dims"], rot["base"], factor), rotate(k, rot["dims"], rot["base"], factor)
    q, k = rms_unit(q, eps), rms_unit(k, eps)
    if pool > 0:
        nb = T // pool
        kb = k[:nb * pool].reshape(nb, pool, G, d).mean(1)
        vb = v[:nb * pool].reshape(nb, pool, G, dv).mean(1)
    gate = sigmoid(h @ W[p + "g"].T)                                   # [T, H]
    out = torch.zeros(T, H, dv, dtype=F64)
    for i in range(T):
        first, blocks = visible(i, window, pool)
        for a in range(H):
            g = a // (H // G)
            keys, vals = k[first:i + 1, g], v[first:i + 1, g]
            if blocks:
                keys, vals = torch.cat([kb[:blocks, g], keys]), torch.cat([vb[:blocks, g], vals])
            s = (keys @ q[i, a]) * scale
            e = torch.exp(s - s.max())
            out[i, a] = (e / e.sum()) @ vals * gate[i, a]
    return out.reshape(T, H * dv) @ W[p + "o"].T


# ---- linear attention whose forget gate also decides what is written ----------------------------------------------------------------
def hgrn2(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    """State S [dim, vdim] per head, zero at the start: S <- diag(f_t) S + (1 - f_t) v_t^T, o_t = S^T silu(q_t), with
    f_t = l + (1 - l) sigmoid(z_t) per head and channel.  Every head's o is RMS-normed with one weight vector; then projected."""
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    q = silu(h @ W[p + "q"].T).reshape(T, H, d)
    v = (h @ W[p + "v"].T).reshape(T, H, dv)
    low = W[p + "lower"]
    f = (low + (1.0 - low) * sigmoid(h @ W[p + "f"].T + W[p + "f.b"])).reshape(T, H, d)
    S = torch.zeros(H, d, dv, dtype=F64)
    o = torch.zeros(T, H, dv, dtype=F64)
    for t in range(T):
        S = f[t][:, :, None] * S + (1.0 - f[t])[:, :, None] * v[t][:, None, :]
        o[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return (rms_unit(o, eps) * W[p + "norm"]).reshape(T, H * dv) @ W[p + "o"].T


# ---- matrix memory with exponential gates --------------------------------------------------------------------------------------------
def mlstm(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    """Per head a memory S [dim, vdim], a normaliser n [dim] (both zero at the start) and a running maximum mx (zero at the start):
    mx' = max(lf + mx, li);  S <- e^(lf + mx - mx') S + e^(li - mx') k v^T;  n <- the same with k alone;
    o = S^T q / (max(|n . q|, e^(-mx')) + 1e-6), with capped log gates li, lf = log sigmoid.  Every head's o is divided by its root
    mean square; then norm weights, a sigmoid gate per entry, projection."""
    T = h.shape[0]
    H, d, dv, cap = m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    q = (h @ W[p + "q"].T).reshape(T, H, d) * d ** -0.5
    k = (h @ W[p + "k"].T).reshape(T, H, d)
    v = (h @ W[p + "v"].T).reshape(T, H, dv)
    li = soft_cap(h @ W[p + "i"].T + W[p + "i.b"], cap)
    lf = log_sigmoid(soft_cap(h @ W[p + "f"].T + W[p + "f.b"], cap))
    S, n, mx = torch.zeros(H, d, dv, dtype=F64), torch.zeros(H, d, dtype=F64), torch.zeros(H, dtype=F64)
    o = torch.zeros(T, H, dv, dtype=F64)
    for t in range(T):
        new = torch.maximum(lf[t] + mx, li[t])
        keep, write = torch.exp(lf[t] + mx - new), torch.exp(li[t] - new)
        S = keep[:, None, None] * S + write[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + write[:, None] * k[t]
        mx = new
        den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-mx)) + 1e-6
        o[t] = torch.einsum("hdv,hd->hv", S, q[t]) / den[:, None]
    y = rms_unit(o, eps).reshape(T, H * dv) * W[p + "norm"] * sigmoid(h @ W[p + "g"].T)
    return y @ W[p + "o"].T


# ---- feed-forward -----------------------------------------------------------------------------------------------------------------
def dense_ff(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    return gelu_erf(h @ W[p + "up"].T) @ W[p + "down"].T


# ---- the model ------------------------------------------------------------------------------------------------------------------
MIXERS = {"attention": attention, "hgrn2": hgrn2, "mlstm": mlstm}


def layer(i: int, cfg: dict, x: torch.Tensor, W: Dict[str, torch.Tensor]) -> torch.Tensor:
    L, p, eps = cfg["layers"][i], f"l{i}.", cfg["norm"]["eps"]
    x = x + MIXERS[L["type"]](centred_norm(x, W[p + "norm1"], eps), W, p + "mix.", L["mixer"], eps)
    if L.get("mlp") is not None:
        x = x + dense_ff(centred_norm(x, W[p + "norm2"], eps), W, p + "mlp.")
    return x


def forward(cfg: dict, weights: Dict[str, torch.Tensor], tokens: List[int], taps: Optional[list] = None) -> torch.Tensor:
    """Logits f64 [T, vocab].  `taps`, when given, receives the residual stream after every layer run."""
    W = {k: v.to(F64) for k, v in weights.items()}
    x0 = W["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    x = x0
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    start, stop, times = (loop["start"], loop["stop"], loop["times"]) if loop else (0, 0, 0)

    def run(i, x):
        x = layer(i, cfg, x, W)
        if taps is not None:
            taps.append(x)
        return x

    for i in range(start):
        x = run(i, x)
    for _ in range(times):
        x = torch.cat([x, x0], 1) @ W["loop.in"].T
        for i in range(start, stop):
            x = run(i, x)
    for i in range(stop, n):
        x = run(i, x)
    return centred_norm(x, W["final.norm"], cfg["norm"]["eps"]) @ W["head"].T
