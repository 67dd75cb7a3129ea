"""Matidra: a decoder-only language model lowered to op lists (seq_ops.StepBuilder) for seq_engine.SequenceEngine.

With n(v; w, b) = (v - mean v) / sqrt(var v + eps) * w + b (layer norm with bias) and a configured alpha a layer is
    x <- n(alpha x + mixer(x); norm1) ;   x <- n(alpha x + ff(x); norm2)      (no feed-forward: the first sublayer only)
so the sublayers read the stream itself, and one launch (FQ3C_SUM_NORM with FQ3C_POST) closes a sublayer: the sum, the norm, the new
stream in f32 and its copy as the next product's operand.  Mixers:
  * "parallel":  left_scale * softmax attention (short convolution on q, k and v, head norms, a query temperature that grows with the
                 position, a sigmoid gate per entry; state: key / value cache) + right_scale * delta rule with a decay per key channel (short
                 convolution and silu, unit queries and keys; state: S [heads * dim, vdim]); both share the convolution's carried inputs;
  * "attention": softmax attention whose values are the projected keys (head norms, then rotary positions on neighbouring pairs with a
                 scaled table, on queries and keys only; state: key / value cache).
Feed-forward: dense, gelu_tanh(gate) * up.  Output: n(x; final.norm), then the head.

This file only packs the checkpoint's tensors into the layouts the mechanisms take and strings the mechanisms together in the
configured order; the kernels, the state manager and the step loop are the shared ones.
"""
from __future__ import annotations

from typing import Callable, Dict, List, Optional

import torch

from .config import ChannelDeltaRuleConfig, MatidraConfig, ScaledPairMixerConfig, SoftmaxAttentionConfig
from .ratizen import scaled_rotary_table
from .seq_ops import StepBuilder
from .seq_state import StateSpec

PAD = 8      # stacked projections are padded to a multiple of this many rows, so that their f32 outputs have 16-byte rows
SYNTHETIC_RANK = 64      # init_synthetic's low-rank sizes when the configuration leaves them to the tensors


def tensor_specs(cfg: MatidraConfig) -> Dict[str, tuple]:
    """name -> shape of every tensor a checkpoint of this configuration holds (None: a size only the tensor itself gives)."""
    W = cfg.width
    out = {"embed": (cfg.vocab, W), "final.norm": (W,), "final.norm.b": (W,), "head": (cfg.vocab, W)}
    for i, L in enumerate(cfg.layers):
        p, m = f"l{i}.", L.mixer
        out.update({p + "norm1": (W,), p + "norm1.b": (W,)})
        if isinstance(m, ScaledPairMixerConfig):
            a, r, q = m.left, m.right, p + "mix.left."
            for n, size in (("q", a.heads * a.dim), ("k", a.kv_heads * a.dim), ("v", a.kv_heads * a.vdim)):
                out.update({q + n: (size, W), q + n + ".conv": (size, a.conv)})
            out.update({q + "q.norm": (a.dim,), q + "k.norm": (a.dim,), q + "g": (a.heads * a.vdim, W), q + "o": (W, a.heads * a.vdim)})
            q = p + "mix.right."
            for n, size in (("q", r.kv_heads * r.dim), ("k", r.kv_heads * r.dim), ("v", r.heads * r.vdim)):
                out.update({q + n: (size, W), q + n + ".conv": (size, r.conv)})
            ra, rg = r.decay_rank or None, r.gate_rank or None
            out.update({q + "b": (r.heads, W), q + "A_log": (r.heads,), q + "dt_bias": (r.heads * r.dim,), q + "norm": (r.vdim,),
                        q + "a1": (ra, W), q + "a2": (r.heads * r.dim, ra), q + "g1": (rg, W), q + "g2": (r.heads * r.vdim, rg),
                        q + "o": (W, r.heads * r.vdim)})
        else:
            q = p + "mix."
            out.update({q + "q": (m.heads * m.dim, W), q + "k": (m.kv_heads * m.dim, W), q + "q.norm": (m.dim,), q + "k.norm": (m.dim,),
                        q + "o": (W, m.heads * m.vdim)})
        if L.mlp is not None:
            out.update({p + "norm2": (W,), p + "norm2.b": (W,), p + "mlp.gate": (L.mlp.ff, W), p + "mlp.up": (L.mlp.ff, W),
                        p + "mlp.down": (W, L.mlp.ff)})
    return out


def init_synthetic(cfg: MatidraConfig, seed: int = 0) -> Dict[str, torch.Tensor]:
    """Random bf16-representable weights of a configuration (no checkpoint offline): products scaled by 1/sqrt(fan-in)."""
    g = torch.Generator().manual_seed(seed)
    w = {}
    for name, shape in tensor_specs(cfg).items():
        shape = tuple(SYNTHETIC_RANK if s is None else s for s in shape)
        last = name.rsplit(".", 1)[-1]
        if last in ("norm1", "norm2", "norm"):
            t = 1.0 + 0.1 * torch.randn(shape, generator=g)
        elif name.endswith((".norm1.b", ".norm2.b", "final.norm.b")):
            t = 0.1 * torch.randn(shape, generator=g)
        elif last == "A_log":
            t = torch.randn(shape, generator=g) - 1.0
        elif last == "dt_bias":
            t = torch.randn(shape, generator=g) - 3.0           # decays mostly close to one, some fast
        elif name == "embed":
            t = torch.randn(shape, generator=g)
        else:
            t = torch.randn(shape, generator=g) / (shape[-1] ** 0.5)
        w[name] = t.to(torch.bfloat16).to(torch.float32)
    return w


class Packer:
    """Checkpoint tensors -> the layouts the mechanisms of seq_ops.StepBuilder take.  `raw(name)` gives a CPU f32 tensor."""

    def __init__(self, raw: Callable[[str], torch.Tensor], device, f32: bool):
        self.raw, self.device, self.wdt = raw, torch.device(device), torch.float32 if f32 else torch.bfloat16

    def W(self, t):   # product operand
        return t.to(self.device, self.wdt).contiguous()

    def F(self, t):   # always-f32 parameter
        return t.to(self.device, torch.float32).contiguous()

    def stack(self, names):
        """One projection out of several, with zero rows up to a multiple of PAD."""
        w = torch.cat([self.raw(n) for n in names], 0)
        return self.W(torch.nn.functional.pad(w, (0, 0, 0, -w.shape[0] % PAD)))

    def taps(self, names):
        """Convolution weights of several parts as one f32 [channels, taps]: shorter ones get zero taps in front."""
        parts = [self.raw(n + ".conv") for n in names]
        n = max(t.shape[1] for t in parts)
        return self.F(torch.cat([torch.nn.functional.pad(t, (n - t.shape[1], 0)) for t in parts], 0))

    def head_norms(self, p: str) -> dict:
        return {"q_norm": self.F(self.raw(p + "q.norm")), "k_norm": self.F(self.raw(p + "k.norm"))}

    def attention(self, p: str, m: SoftmaxAttentionConfig) -> dict:
        """Attention whose values are its projected keys."""
        d = {"wqkv": self.stack((p + "q", p + "k")), "o": self.W(self.raw(p + "o")), "freq": None, **self.head_norms(p)}
        if m.rot_dims > 0:
            f, d["amp"] = scaled_rotary_table(m.rot_dims, m.rot_base, m.rot_scaling)
            d["freq"] = self.F(f)
            d["freq_lo"] = self.F(f - f.to(torch.float32).to(torch.float64))
        return d

    def convolved_attention(self, p: str) -> dict:
        """Attention with short convolutions and a gate per entry, on its own."""
        names = [p + n for n in ("q", "k", "v")]
        return {"wqkv": self.stack(names + [p + "g"]), "conv": self.taps(names), "o": self.W(self.raw(p + "o")), **self.head_norms(p)}

    def delta_parts(self, p: str, scale: float = 1.0) -> dict:
        """What the channel-decay delta rule takes between its convolution and its output product; scale multiplies its result."""
        a1, a2, g1, g2 = (self.raw(p + n) for n in ("a1", "a2", "g1", "g2"))
        if a1.shape[0] != a2.shape[1] or g1.shape[0] != g2.shape[1]:
            raise ValueError(f"{p}: the two factors of a low-rank projection disagree on their inner size")
        return {"a2": self.W(a2.T), "g2": self.W(g2.T), "dt_bias": self.F(self.raw(p + "dt_bias")), "A_log": self.F(self.raw(p + "A_log")),
                "norm": self.F(self.raw(p + "norm").to(torch.float64) * scale)}

    def channel_delta(self, p: str) -> dict:
        """The channel-decay delta rule on its own."""
        names = [p + n for n in ("q", "k", "v")]
        return {"win": self.stack(names + [p + n for n in ("b", "a1", "g1")]), "conv": self.taps(names), "o": self.W(self.raw(p + "o")),
                **self.delta_parts(p)}

    def pair(self, p: str, right_scale: float) -> dict:
        """Both side by side: one projection, one convolution, one output product on the concatenated heads."""
        lp, rp = p + "left.", p + "right."
        conv = [lp + n for n in ("q", "k", "v")] + [rp + n for n in ("q", "k", "v")]
        return {"win": self.stack(conv + [lp + "g"] + [rp + n for n in ("b", "a1", "g1")]), "conv": self.taps(conv),
                "o": self.W(torch.cat([self.raw(lp + "o"), self.raw(rp + "o")], 1)), "left": self.head_norms(lp),
                "right": self.delta_parts(rp, right_scale)}


class MatidraModel:
    def __init__(self, cfg: MatidraConfig, get: Callable[[str], Optional[torch.Tensor]], device, f32: bool = False):
        """`get(name)` returns a CPU tensor or None."""
        self.cfg, self.device, self.f32 = cfg, torch.device(device), bool(f32)
        self.wdt = torch.float32 if f32 else torch.bfloat16
        self.vocab, self.width = cfg.vocab, cfg.width
        specs = tensor_specs(cfg)

        def raw(name):
            t = get(name)
            if t is None:
                raise KeyError(f"tensor {name!r} is missing")
            want = specs[name]
            if len(t.shape) != len(want) or any(b is not None and a != b for a, b in zip(t.shape, want)):
                raise ValueError(f"tensor {name!r} has shape {tuple(t.shape)}, the configuration implies {tuple(want)}")
            return t.to(torch.float32)

        pk = Packer(raw, self.device, self.f32)
        self.g: Dict[str, object] = {"embed": pk.W(raw("embed")), "final.norm": pk.F(raw("final.norm")), "final.norm.b": pk.F(raw("final.norm.b")),
                                     "head": pk.W(raw("head")), "sum": pk.F(torch.tensor([cfg.alpha, 1.0], dtype=torch.float64)),
                                     "one": pk.F(torch.ones(1))}
        self.layers: List[dict] = []
        for i, L in enumerate(cfg.layers):
            p, m = f"l{i}.", L.mixer
            d: dict = {n: pk.F(raw(p + n)) for n in ("norm1", "norm1.b")}
            d["mix"] = pk.pair(p + "mix.", m.right_scale) if isinstance(m, ScaledPairMixerConfig) else pk.attention(p + "mix.", m)
            if L.mlp is not None:
                d.update({n: pk.F(raw(p + n)) for n in ("norm2", "norm2.b")})
                gate_up = torch.stack([raw(p + "mlp.gate"), raw(p + "mlp.up")], 1).reshape(2 * L.mlp.ff, cfg.width)
                d["ff"] = {"gate_up": pk.W(gate_up), "down": pk.W(raw(p + "mlp.down"))}
            self.layers.append(d)

    # ---- what a sequence keeps between steps ------------------------------------------------------
    def state_specs(self) -> List[StateSpec]:
        out = []

        def cache(i, m: SoftmaxAttentionConfig):
            out.append(StateSpec(f"l{i}.k", "append", m.kv_heads * m.dim, dtype=self.wdt))
            out.append(StateSpec(f"l{i}.v", "append", m.kv_heads * m.vdim, dtype=self.wdt))

        for i, L in enumerate(self.cfg.layers):
            m = L.mixer
            if isinstance(m, ScaledPairMixerConfig):
                r: ChannelDeltaRuleConfig = m.right
                cache(i, m.left)
                channels, taps = self.layers[i]["mix"]["conv"].shape
                out.append(StateSpec(f"l{i}.kd.conv", "carry", channels, taps - 1))
                out.append(StateSpec(f"l{i}.kd.s", "carry", r.vdim, r.heads * r.dim, in_place=True))
            else:
                cache(i, m)
        return out

    # ---- one step of M tokens -----------------------------------------------------------------------
    def build_step(self, b: StepBuilder, ids: torch.Tensor, layer_taps: Optional[list] = None):
        """ids: device int32 [M].  Returns the f32 residual stream after the last layer, [M, width].  `layer_taps`, when given,
        receives one f32 buffer per layer that the step also fills with the stream after that layer (debugging, tests)."""
        c, M, Wd, g = self.cfg, b.M, self.cfg.width, self.g
        parts = torch.zeros(2, M, Wd, dtype=torch.float32, device=self.device)      # [stream | the running sublayer's output]
        b.plan.keep.append(parts)
        x, y = parts[0], parts[1]
        h = x if b.f32 else b.buf("h", M, Wd, b.adt)        # the stream as a product operand
        b.embed(ids, g["embed"], x, operand=None if b.f32 else h)

        def close(w, n):
            b.sum_norm(parts, 2, g["sum"], norm_w=w[n], norm_b=w[n + ".b"], norm_out=None if b.f32 else h, eps=c.norm_eps, center=True, post=True)

        for i, (L, w) in enumerate(zip(c.layers, self.layers)):
            m = L.mixer
            if isinstance(m, ScaledPairMixerConfig):
                b.attention_beside_delta_rule(h, m.left, m.right, w["mix"], f"l{i}.k", f"l{i}.v", f"l{i}.kd", c.norm_eps, y, left_scale=m.left_scale)
            else:
                b.softmax_attention(h, m, w["mix"], f"l{i}.k", f"l{i}.v", y, eps=c.norm_eps)
            close(w, "norm1")
            if L.mlp is not None:
                b.gelu_glu_ff(h, w["ff"], y)
                close(w, "norm2")
            if layer_taps is not None:
                t = torch.zeros(M, Wd, dtype=torch.float32, device=self.device)
                b.plan.keep.append(t)
                b.sum_norm(parts, 1, g["one"], out=t)
                layer_taps.append(t)
        b.commit()
        return x

    def build_head(self, b: StepBuilder, x: torch.Tensor, want: torch.Tensor) -> torch.Tensor:
        """`b` is a builder of b.M = wanted rows.  Logits f32 [b.M, vocab] of the rows of x (f32, a step's output) named by
        the device int32 index list `want`."""
        c = self.cfg
        rows = b.embed(want, x, b.buf("head.rows", b.M, c.width))
        xn = b.group_norm(rows, self.g["final.norm"], 1, c.norm_eps, b.buf("head.xn", b.M, c.width, b.adt), center=True, bias=self.g["final.norm.b"])
        return b.linear(xn, self.g["head"], b.buf("head.logits", b.M, c.vocab))
