"""Sirodra: a decoder-only language model lowered to op lists (seq_ops.StepBuilder) for seq_engine.SequenceEngine.

With n(v; w) = (v - mean v) / sqrt(var v + eps) * w (layer norm, no bias) a layer is
    x <- x + mixer(n(x; norm1)) ;   x <- x + ff(n(x; norm2))      (no feed-forward: the first sublayer only)
and one launch (FQ3C_SUM_NORM) closes a sublayer: it adds the sublayer's output to the stream and writes what reads the stream next
(a norm, or the operand of the product in front of a pass).  Mixers:
  * "hgrn2":     linear attention with a forget gate per channel that also decides what is written (state: S [heads * dim, vdim]);
  * "mlstm":     matrix memory with exponential gates under a running maximum (state: S and its normaliser [heads * dim, vdim + 1], m [heads]);
  * "attention": windowed softmax attention with biased projections, rotary positions (linear scaling), unit-RMS queries and keys, one
                 pooled key and value per block before the window, and a sigmoid gate per head (state: key / value cache, pooled rows).
Feed-forward: dense, erf-GELU.  A configured range of layers runs several times on the same tensors, every pass on states of its own;
in front of each pass x <- W_in [x; embedding output].  Output: n(x; final.norm), then the head.

This file only packs the checkpoint's tensors into the layouts the mechanisms take and strings the mechanisms together in the
configured order; the kernels, the state manager and the step loop are the shared ones.
"""
from __future__ import annotations

from typing import Callable, Dict, List, Optional

import torch

from .config import ForgetGateAttentionConfig, MatrixMemoryConfig, SirodraConfig, SoftmaxAttentionConfig
from .seq_ops import StepBuilder
from .seq_state import StateSpec

PAD = 8      # stacked projections are padded to a multiple of this many rows, so that their f32 outputs have 16-byte rows


def tensor_specs(cfg: SirodraConfig) -> Dict[str, tuple]:
    """name -> shape of every tensor a checkpoint of this configuration holds."""
    W = cfg.width
    out = {"embed": (cfg.vocab, W), "final.norm": (W,), "head": (cfg.vocab, W)}
    if cfg.loop is not None:
        out["loop.in"] = (W, 2 * W)
    for i, L in enumerate(cfg.layers):
        p, m = f"l{i}.", L.mixer
        q = p + "mix."
        out[p + "norm1"] = (W,)
        if isinstance(m, ForgetGateAttentionConfig):
            n = m.heads * m.dim
            out.update({q + "q": (n, W), q + "f": (n, W), q + "f.b": (n,), q + "lower": (n,), q + "v": (m.heads * m.vdim, W), q + "norm": (m.vdim,),
                        q + "o": (W, m.heads * m.vdim)})
        elif isinstance(m, MatrixMemoryConfig):
            n, nv = m.heads * m.dim, m.heads * m.vdim
            out.update({q + "q": (n, W), q + "k": (n, W), q + "v": (nv, W), q + "g": (nv, W), q + "o": (W, nv), q + "norm": (nv,)})
            for g in ("i", "f"):
                out.update({q + g: (m.heads, W), q + g + ".b": (m.heads,)})
        else:
            for n, size in (("q", m.heads * m.dim), ("k", m.kv_heads * m.dim), ("v", m.kv_heads * m.vdim)):
                out.update({q + n: (size, W), q + n + ".b": (size,)})
            out.update({q + "g": (m.heads, W), q + "o": (W, m.heads * m.vdim)})
        if L.mlp is not None:
            out.update({p + "norm2": (W,), p + "mlp.up": (L.mlp.ff, W), p + "mlp.down": (W, L.mlp.ff)})
    return out


def init_synthetic(cfg: SirodraConfig, seed: int = 0) -> Dict[str, torch.Tensor]:
    """Random bf16-representable weights of a configuration (no checkpoint offline): products scaled by 1/sqrt(fan-in)."""
    g = torch.Generator().manual_seed(seed)
    w = {}
    for name, shape in tensor_specs(cfg).items():
        last = name.rsplit(".", 1)[-1]
        if last in ("norm1", "norm2", "norm"):
            t = 1.0 + 0.1 * torch.randn(shape, generator=g)
        elif last == "lower":
            t = 0.9 * torch.rand(shape, generator=g)
        elif name.endswith("f.b"):
            t = 2.0 + torch.randn(shape, generator=g)           # forget gates mostly near one, some fast
        elif last == "b":
            t = 0.3 * torch.randn(shape, generator=g)
        elif name == "embed":
            t = torch.randn(shape, generator=g)
        else:
            t = torch.randn(shape, generator=g) / (shape[-1] ** 0.5)
        w[name] = t.to(torch.bfloat16).to(torch.float32)
    return w


def rotary_frequencies(dims: int, base: float, factor: float = 1.0) -> torch.Tensor:
    """f_i = base^(-2i/dims) / factor, i < dims / 2, in float64 (rounded once, by the caller)."""
    i = torch.arange(dims // 2, dtype=torch.float64)
    return torch.as_tensor(base, dtype=torch.float64) ** (-2.0 * i / dims) / factor


class Packer:
    """Checkpoint tensors -> the layouts the mechanisms of seq_ops.StepBuilder take.  `raw(name)` gives a CPU f32 tensor."""

    def __init__(self, raw: Callable[[str], torch.Tensor], device, f32: bool):
        self.raw, self.device, self.wdt = raw, torch.device(device), torch.float32 if f32 else torch.bfloat16

    def W(self, t):   # product operand
        return t.to(self.device, self.wdt).contiguous()

    def F(self, t):   # always-f32 parameter
        return t.to(self.device, torch.float32).contiguous()

    def stack(self, p: str, names, biased):
        """One projection out of several (zero rows up to a multiple of PAD) and its bias (zeros for the parts that have none)."""
        w = torch.cat([self.raw(p + n) for n in names], 0)
        b = torch.cat([self.raw(p + n + ".b") if n in biased else torch.zeros(self.raw(p + n).shape[0]) for n in names])
        pad = -w.shape[0] % PAD
        return self.W(torch.nn.functional.pad(w, (0, 0, 0, pad))), self.F(torch.nn.functional.pad(b, (0, pad)))

    def attention(self, p: str, m: SoftmaxAttentionConfig) -> dict:
        w, b = self.stack(p, ("q", "k", "v", "g"), ("q", "k", "v"))
        d = {"wqkv": w, "bqkv": b, "o": self.W(self.raw(p + "o")), "o_b": None, "sink": None, "r12": None, "freq": None}
        if m.rot_dims > 0:
            f = rotary_frequencies(m.rot_dims, m.rot_base, m.rot_factor)
            d["freq"] = self.F(f)
            d["freq_lo"] = self.F(f - f.to(torch.float32).to(torch.float64))
        return d

    def forget_gate(self, p: str) -> dict:
        w, b = self.stack(p, ("q", "f", "v"), ("f",))
        return {"win": w, "bin": b, "lower": self.F(self.raw(p + "lower")), "norm": self.F(self.raw(p + "norm")), "o": self.W(self.raw(p + "o"))}

    def memory(self, p: str) -> dict:
        w, b = self.stack(p, ("q", "k", "v", "g", "i", "f"), ("i", "f"))
        return {"win": w, "bin": b, "norm": self.F(self.raw(p + "norm")), "o": self.W(self.raw(p + "o"))}


class SirodraModel:
    def __init__(self, cfg: SirodraConfig, get: Callable[[str], Optional[torch.Tensor]], device, f32: bool = False):
        """`get(name)` returns a CPU tensor or None."""
        self.cfg, self.device, self.f32 = cfg, torch.device(device), bool(f32)
        self.wdt = torch.float32 if f32 else torch.bfloat16
        self.vocab, self.width = cfg.vocab, cfg.width
        specs = tensor_specs(cfg)

        def raw(name):
            t = get(name)
            if t is None:
                raise KeyError(f"tensor {name!r} is missing")
            if tuple(t.shape) != tuple(specs[name]):
                raise ValueError(f"tensor {name!r} has shape {tuple(t.shape)}, the configuration implies {tuple(specs[name])}")
            return t.to(torch.float32)

        pk = Packer(raw, self.device, self.f32)
        self.g: Dict[str, object] = {"embed": pk.W(raw("embed")), "final.norm": pk.F(raw("final.norm")), "head": pk.W(raw("head")),
                                     "ones": pk.F(torch.ones(2))}
        if cfg.loop is not None:
            self.g["loop.in"] = pk.W(raw("loop.in"))
        self.layers: List[dict] = []
        for i, L in enumerate(cfg.layers):
            p, m = f"l{i}.", L.mixer
            d: dict = {"norm1": pk.F(raw(p + "norm1"))}
            if isinstance(m, ForgetGateAttentionConfig):
                d["mix"] = pk.forget_gate(p + "mix.")
            elif isinstance(m, MatrixMemoryConfig):
                d["mix"] = pk.memory(p + "mix.")
            else:
                d["mix"] = pk.attention(p + "mix.", m)
            if L.mlp is not None:
                d["norm2"] = pk.F(raw(p + "norm2"))
                d["ff"] = {"up": pk.W(raw(p + "mlp.up")), "down": pk.W(raw(p + "mlp.down"))}
            self.layers.append(d)

    # ---- what a sequence keeps between steps ------------------------------------------------------
    def state_specs(self) -> List[StateSpec]:
        out = []
        for r, (i, _) in enumerate(self.cfg.runs):       # every layer run has a state of its own, also the later passes of a loop
            m, p = self.cfg.layers[i].mixer, f"r{r}."
            if isinstance(m, ForgetGateAttentionConfig):
                out.append(StateSpec(p + "fg", "carry", m.vdim, m.heads * m.dim, in_place=True))
            elif isinstance(m, MatrixMemoryConfig):
                out += [StateSpec(p + "mm.s", "carry", m.vdim + 1, m.heads * m.dim, in_place=True), StateSpec(p + "mm.m", "carry", m.heads)]
            else:
                for n, cols in (("k", m.kv_heads * m.dim), ("v", m.kv_heads * m.vdim)):
                    out.append(StateSpec(p + n, "append", cols, dtype=self.wdt))
                    if m.pool > 0:
                        out.append(StateSpec(p + n + ".pool", "append", cols, dtype=self.wdt, every=m.pool))
        return out

    # ---- one step of M tokens -----------------------------------------------------------------------
    def build_step(self, b: StepBuilder, ids: torch.Tensor, layer_taps: Optional[list] = None):
        """ids: device int32 [M].  Returns the f32 residual stream after the last layer, [M, width].  `layer_taps`, when given,
        receives one f32 buffer per layer run that the step also fills with the stream after that run (debugging, tests)."""
        c, M, Wd, g = self.cfg, b.M, self.cfg.width, self.g
        runs = c.runs
        parts = torch.zeros(2, M, Wd, dtype=torch.float32, device=self.device)      # [stream | the running sublayer's output]
        b.plan.keep.append(parts)
        x, y = parts[0], parts[1]
        hn = b.buf("hn", M, Wd, b.adt)        # the running sublayer's normed input
        if c.loop is not None:                # [stream | embedding output], what the product in front of a pass reads
            cat = b.buf("loop.cat", M, 2 * Wd, b.adt)
            b.embed(ids, g["embed"], x, operand=cat, operand_col=0 if runs[0][1] else Wd)
        else:
            b.embed(ids, g["embed"], x)

        def close(r, w):
            """The sublayer's output joins the stream; what reads the stream next is written in the same launch."""
            if w is not None:
                b.sum_norm(parts, 2, g["ones"], norm_w=w, norm_out=hn, eps=c.norm_eps, center=True)
            elif r + 1 < len(runs) and runs[r + 1][1]:
                b.sum_norm(parts, 2, g["ones"], norm_out=cat)
            else:
                b.sum_norm(parts, 2, g["ones"])

        for r, (i, starts_pass) in enumerate(runs):
            L, w, m, p = c.layers[i], self.layers[i], c.layers[i].mixer, f"r{r}."
            if starts_pass:
                b.linear(cat, g["loop.in"], x)
            if starts_pass or r == 0:
                b.group_norm(x, w["norm1"], 1, c.norm_eps, hn, center=True)
            if isinstance(m, ForgetGateAttentionConfig):
                b.forget_gate_attention(hn, m, w["mix"], p + "fg", c.norm_eps, y)
            elif isinstance(m, MatrixMemoryConfig):
                b.matrix_memory(hn, m, w["mix"], p + "mm", c.norm_eps, y)
            else:
                b.softmax_attention(hn, m, w["mix"], p + "k", p + "v", y, eps=c.norm_eps)
            following = self.layers[runs[r + 1][0]]["norm1"] if r + 1 < len(runs) and not runs[r + 1][1] else None
            if L.mlp is not None:
                close(r, w["norm2"])
                b.gelu_ff(hn, w["ff"], y)
            close(r, following)
            if layer_taps is not None:
                t = torch.zeros(M, Wd, dtype=torch.float32, device=self.device)
                b.plan.keep.append(t)
                b.sum_norm(parts, 1, g["ones"], out=t)
                layer_taps.append(t)
        b.commit()
        return x

    def build_head(self, b: StepBuilder, x: torch.Tensor, want: torch.Tensor) -> torch.Tensor:
        """`b` is a builder of b.M = wanted rows.  Logits f32 [b.M, vocab] of the rows of x (f32, a step's output) named by
        the device int32 index list `want`."""
        c = self.cfg
        rows = b.embed(want, x, b.buf("head.rows", b.M, c.width))
        xn = b.group_norm(rows, self.g["final.norm"], 1, c.norm_eps, b.buf("head.xn", b.M, c.width, b.adt), center=True)
        return b.linear(xn, self.g["head"], b.buf("head.logits", b.M, c.vocab))
