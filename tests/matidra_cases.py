"""Small Matidra configurations and random checkpoints for the tests (raw config dictionaries, as a config.json holds them)."""
import torch

from sidalorn_cases import save_checkpoint, tokens  # noqa: F401  (same checkpoint format and token draws)


def left(heads, kv_heads, dim, vdim, conv, scale, temp=None):
    """temp: (coef, every) or None for no query temperature."""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "scale": scale}
    if temp:
        m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    return m


def right(heads, kv_heads, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def pair(a, b, left_scale, right_scale):
    return {"type": "parallel", "mixer": {"left": a, "right": b, "left_scale": left_scale, "right_scale": right_scale}}


def attn(heads, kv_heads, dim, scale, rot_dims=0, base=10000.0, scaling=None):
    """rot_dims 0: no positions; scaling: (factor, original, fast, slow) or None."""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale}
    if rot_dims:
        m["rot"] = {"dims": rot_dims, "base": base}
        if scaling:
            m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"type": "attention", "mixer": m}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def layer(mixer, mlp=None):
    return dict(mixer, mlp=mlp)


def config(vocab, width, layers, alpha=1.7, eps=1e-6):
    return {"architecture": "Matidra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "postln_alpha": alpha, "layers": layers}


def odd():
    """Sizes that are multiples of nothing convenient, convolutions of different lengths side by side, grouped heads on every side,
    feed-forwards on some layers only."""
    return config(61, 44, [
        layer(pair(left(4, 2, 10, 7, 3, 0.4, (0.6, 5)), right(6, 2, 6, 9, 5), 0.7, 1.6), dense(30)),
        layer(attn(3, 1, 14, 0.3, 10, 300.0, (3.0, 64, 4.0, 1.5))),
        layer(pair(left(2, 1, 6, 11, 4, 0.5, (0.25, 17)), right(3, 3, 13, 5, 2), 1.3, 0.5)),
        layer(attn(4, 4, 6, 0.5, 6, 50.0), dense(21)),
        layer(pair(left(3, 3, 8, 8, 1, 0.35), right(2, 1, 9, 18, 1), 1.0, 1.0), dense(10)),
    ], alpha=1.4, eps=1e-2)      # eps large enough that a norm ignoring it fails


def unaligned():
    """Width not a multiple of 8 (no tensor-core product takes it); no rotation in one attention, all of a head in the other."""
    return config(29, 36, [
        layer(attn(2, 2, 10, 0.5)),
        layer(pair(left(2, 2, 9, 5, 2, 0.4, (1.0, 3)), right(2, 2, 5, 6, 3), 0.9, 1.1), dense(14)),
        layer(attn(6, 2, 8, 0.4, 8, 100.0, (2.0, 40, 3.0, 1.0)), dense(18)),
    ], alpha=1.0)


def aligned():
    """Sizes the tensor-core kernels take (multiples of 16 / 64)."""
    return config(320, 128, [
        layer(pair(left(4, 2, 32, 64, 4, 0.2, (0.3, 50)), right(4, 2, 32, 48, 4), 0.8, 1.2), dense(192)),
        layer(attn(8, 2, 32, 0.2, 16, 5000.0, (4.0, 256, 16.0, 2.0)), dense(128)),
        layer(pair(left(2, 2, 64, 32, 3, 0.15, (0.2, 64)), right(2, 2, 64, 64, 4), 1.1, 0.6), dense(320)),
    ], alpha=2.2, eps=1e-5)


def weights(cfg, seed=0, decay_rank=5, gate_rank=7):
    """Random weights rounded to bf16 (so that bf16 and f32 runs hold the same numbers).  Queries and keys are normed per head, so a
    test that wants peaked attention rows raises the configuration's `scale`."""
    g = torch.Generator().manual_seed(seed)

    def rnd(*shape, s=1.0):
        return s * torch.randn(*shape, generator=g)

    W, width = {}, cfg["width"]

    def norm(name, n):
        W[name], W[name + ".b"] = 1.0 + rnd(n, s=0.2), rnd(n, s=0.2)

    def heads(q, m):
        W[q + "q.norm"], W[q + "k.norm"] = 1.0 + rnd(m["dim"], s=0.3), 1.0 + rnd(m["dim"], s=0.3)

    W["embed"] = rnd(cfg["vocab"], width)
    W["head"] = rnd(cfg["vocab"], width, s=width ** -0.5)
    norm("final.norm", width)
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        norm(p + "norm1", width)
        if L["type"] == "parallel":
            a, r, q = m["left"], m["right"], p + "mix.left."
            H, G, d, dv = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            for n, size in (("q", H * d), ("k", G * d), ("v", G * dv)):
                W[q + n], W[q + n + ".conv"] = rnd(size, width, s=width ** -0.5), rnd(size, a["conv"], s=a["conv"] ** -0.5)
            heads(q, a)
            W[q + "g"] = rnd(H * dv, width, s=2.0 * width ** -0.5)
            W[q + "o"] = rnd(width, H * dv, s=2.0 * (H * dv) ** -0.5)
            q = p + "mix.right."
            H, G, d, dv = r["heads"], r["kv_heads"], r["dim"], r["vdim"]
            for n, size in (("q", G * d), ("k", G * d), ("v", H * dv)):
                W[q + n], W[q + n + ".conv"] = rnd(size, width, s=width ** -0.5), rnd(size, r["conv"], s=r["conv"] ** -0.5)
            W[q + "b"] = rnd(H, width, s=2.0 * width ** -0.5)
            W[q + "A_log"], W[q + "dt_bias"] = rnd(H, s=0.7) - 0.5, rnd(H * d) - 2.0
            W[q + "a1"], W[q + "a2"] = rnd(decay_rank, width, s=width ** -0.5), rnd(H * d, decay_rank, s=1.5 * decay_rank ** -0.5)
            W[q + "g1"], W[q + "g2"] = rnd(gate_rank, width, s=width ** -0.5), rnd(H * dv, gate_rank, s=2.0 * gate_rank ** -0.5)
            W[q + "norm"] = 1.0 + rnd(dv, s=0.2)
            W[q + "o"] = rnd(width, H * dv, s=2.0 * (H * dv) ** -0.5)
        else:
            q = p + "mix."
            H, G, d = m["heads"], m["kv_heads"], m["dim"]
            W[q + "q"], W[q + "k"] = rnd(H * d, width, s=width ** -0.5), rnd(G * d, width, s=width ** -0.5)
            heads(q, m)
            W[q + "o"] = rnd(width, H * d, s=(H * d) ** -0.5)
        f = L.get("mlp")
        if f is not None:
            norm(p + "norm2", width)
            W[p + "mlp.gate"], W[p + "mlp.up"] = rnd(f["ff"], width, s=2.0 * width ** -0.5), rnd(f["ff"], width, s=width ** -0.5)
            W[p + "mlp.down"] = rnd(width, f["ff"], s=f["ff"] ** -0.5)
    return {k: v.to(torch.bfloat16).to(torch.float32) for k, v in W.items()}      # what a bf16 checkpoint holds
