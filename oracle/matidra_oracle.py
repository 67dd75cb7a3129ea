"""Plain, slow restatement of the Matidra design in float64 PyTorch on the CPU — the yardstick the CUDA path is held against.

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


def softplus(z: torch.Tensor) -> torch.Tensor:
    """log(1 + e^z) without overflow."""
    return torch.maximum(z, torch.zeros_like(z)) + torch.log1p(torch.exp(-z.abs()))


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def rms_unit(v: torch.Tensor, eps: float) -> torch.Tensor:
    """v / sqrt(mean(v^2) + eps) over the last axis."""
    return v / torch.sqrt((v * v).mean(-1, keepdim=True) + eps)


def unit(v: torch.Tensor) -> torch.Tensor:
    """v / sqrt(sum(v^2) + 1e-6) over the last axis."""
    return v / torch.sqrt((v * v).sum(-1, keepdim=True) + 1e-6)


def layer_norm(v: torch.Tensor, w: torch.Tensor, b: torch.Tensor, eps: float) -> torch.Tensor:
    d = v - v.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w + b


# ---- short causal convolution ------------------------------------------------------------------------------------------------
def time_conv(u: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """y[t, c] = sum_j w[c, j] u[t - (taps - 1) + j, c], zeros before position 0."""
    taps = w.shape[1]
    y = torch.zeros_like(u)
    for t in range(u.shape[0]):
        for j in range(taps):
            s = t - (taps - 1) + j
            if s >= 0:
                y[t] = y[t] + w[:, j] * u[s]
    return y


# ---- rotary positions ----------------------------------------------------------------------------------------------------------
def rotary_table(dims: int, base: float, scaling: Optional[dict]):
    """(frequencies [dims / 2], amplitude).  Without scaling f_i = base^(-2i/dims) and amplitude 1."""
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return f, 1.0

    def at(turns):
        return dims * math.log(scaling["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(at(scaling["fast"])), 0)
    hi = min(math.ceil(at(scaling["slow"])), dims - 1)
    out = []
    for i, fi in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / scaling["factor"] * r + fi * (1.0 - r))
    return out, 0.1 * math.log(scaling["factor"]) + 1.0


def rotate(v: torch.Tensor, dims: int, base: float, scaling: Optional[dict] = None) -> torch.Tensor:
    """v [T, heads, n]: among the first `dims` entries of every head, entries (2i, 2i + 1) turn at position t by the angle t f_i,
    cos and sin times the amplitude; entries from `dims` on pass unchanged."""
    f, amp = rotary_table(dims, base, scaling)
    out = v.clone()
    for i in range(dims // 2):
        ang = torch.arange(v.shape[0], dtype=F64) * f[i]
        c, s = amp * torch.cos(ang)[:, None], amp * torch.sin(ang)[:, None]
        a, b = v[..., 2 * i], v[..., 2 * i + 1]
        out[..., 2 * i], out[..., 2 * i + 1] = a * c - b * s, b * c + a * s
    return out


# ---- softmax attention ----------------------------------------------------------------------------------------------------------
def causal_softmax(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float) -> torch.Tensor:
    """q [T, H, d], k [T, G, d], v [T, G, dv]; query head a reads key / value head a // (H / G); position i sees j <= i."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for i in range(T):
        for a in range(H):
            g = a // (H // G)
            s = (k[:i + 1, g] @ q[i, a]) * scale
            e = torch.exp(s - s.max())
            out[i, a] = (e / e.sum()) @ v[:i + 1, g]
    return out


def temperature(T: int, coef: float, every: float) -> torch.Tensor:
    """[T]: 1 + coef ln(floor((p + 1) / every) + 1)."""
    return torch.tensor([1.0 + coef * math.log(math.floor((p + 1) / every) + 1.0) for p in range(T)], dtype=F64)


def convolved_attention(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    """Projections through a short convolution, head norms, query temperature, softmax over all earlier keys, a sigmoid gate per entry."""
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = time_conv(h @ W[p + "q"].T, W[p + "q.conv"]).reshape(T, H, d)
    k = time_conv(h @ W[p + "k"].T, W[p + "k.conv"]).reshape(T, G, d)
    v = time_conv(h @ W[p + "v"].T, W[p + "v.conv"]).reshape(T, G, dv)
    q, k = rms_unit(q, eps) * W[p + "q.norm"], rms_unit(k, eps) * W[p + "k.norm"]
    t = m.get("q_temp")
    if t:
        q = q * temperature(T, t["coef"], t["every"])[:, None, None]
    o = causal_softmax(q, k, v, m["scale"]).reshape(T, H * dv)
    return (o * sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


def keys_as_values_attention(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    """The values are the projected keys, before norm and rotation."""
    T, H, G, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = (h @ W[p + "q"].T).reshape(T, H, d)
    v = (h @ W[p + "k"].T).reshape(T, G, d)
    q, k = rms_unit(q, eps) * W[p + "q.norm"], rms_unit(v, eps) * W[p + "k.norm"]
    r = m.get("rot")
    if r:
        q, k = rotate(q, r["dims"], r["base"], r.get("scaling")), rotate(k, r["dims"], r["base"], r.get("scaling"))
    return causal_softmax(q, k, v, m["scale"]).reshape(T, H * d) @ W[p + "o"].T


# ---- delta rule with a decay per key channel ----------------------------------------------------------------------------------
def delta_walk(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, g: torch.Tensor, beta: torch.Tensor) -> torch.Tensor:
    """q, k, g [T, H, d], v [T, H, dv], beta [T, H].  State S [d, dv] per head from zero:
    S <- diag(g) S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=F64)
    o = torch.zeros_like(v)
    for t in range(T):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        o[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return o


def channel_delta_rule(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = silu(time_conv(h @ W[p + "q"].T, W[p + "q.conv"])).reshape(T, G, d)
    k = silu(time_conv(h @ W[p + "k"].T, W[p + "k.conv"])).reshape(T, G, d)
    v = silu(time_conv(h @ W[p + "v"].T, W[p + "v.conv"])).reshape(T, H, dv)
    of = torch.tensor([a // (H // G) for a in range(H)])
    q, k = (unit(q) * d ** -0.5)[:, of], unit(k)[:, of]
    beta = sigmoid(h @ W[p + "b"].T)
    z = (h @ W[p + "a1"].T @ W[p + "a2"].T + W[p + "dt_bias"]).reshape(T, H, d)
    g = torch.exp(-torch.exp(W[p + "A_log"])[None, :, None] * softplus(z))
    o = rms_unit(delta_walk(q, k, v, g, beta), eps) * W[p + "norm"]
    gate = sigmoid(h @ W[p + "g1"].T @ W[p + "g2"].T).reshape(T, H, dv)
    return (o * gate).reshape(T, H * dv) @ W[p + "o"].T


# ---- feed-forward -----------------------------------------------------------------------------------------------------------------
def dense_ff(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    return (gelu_tanh(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


# ---- the model ------------------------------------------------------------------------------------------------------------------
def mixer(L: dict, h: torch.Tensor, W: Dict[str, torch.Tensor], p: str, eps: float) -> torch.Tensor:
    m = L["mixer"]
    if L["type"] == "attention":
        return keys_as_values_attention(h, W, p, m, eps)
    left = convolved_attention(h, W, p + "left.", m["left"], eps)
    right = channel_delta_rule(h, W, p + "right.", m["right"], eps)
    return m["left_scale"] * left + m["right_scale"] * right


def layer(i: int, cfg: dict, x: torch.Tensor, W: Dict[str, torch.Tensor]) -> torch.Tensor:
    """Norms after the sums: x <- norm1(alpha x + mixer(x)), x <- norm2(alpha x + ff(x))."""
    L, p, eps, alpha = cfg["layers"][i], f"l{i}.", cfg["norm"]["eps"], cfg["postln_alpha"]
    x = layer_norm(alpha * x + mixer(L, x, W, p + "mix.", eps), W[p + "norm1"], W[p + "norm1.b"], eps)
    if L.get("mlp") is not None:
        x = layer_norm(alpha * x + dense_ff(x, W, p + "mlp."), W[p + "norm2"], W[p + "norm2.b"], eps)
    return x


def forward(cfg: dict, weights: Dict[str, torch.Tensor], tokens: List[int], taps: Optional[list] = None) -> torch.Tensor:
    """Logits f64 [T, vocab].  `taps`, when given, receives the residual stream after every layer."""
    W = {k: v.to(F64) for k, v in weights.items()}
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    for i in range(len(cfg["layers"])):
        x = layer(i, cfg, x, W)
        if taps is not None:
            taps.append(x)
    return layer_norm(x, W["final.norm"], W["final.norm.b"], cfg["norm"]["eps"]) @ W["head"].T
