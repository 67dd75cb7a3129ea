"""Small Sirodra configurations and random checkpoints for the tests (raw config dictionaries, as a config.json holds them)."""
import torch

from sidalorn_cases import save_checkpoint, tokens  # noqa: F401  (same checkpoint format and token draws)


def hgrn(heads, dim, vdim):
    return {"type": "hgrn2", "mixer": {"heads": heads, "dim": dim, "vdim": vdim}}


def mlstm(heads, dim, vdim, cap):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}}


def attn(heads, kv_heads, dim, vdim, window, pool, scale, rot_dims=0, base=10000.0, factor=None):
    """window 0: no mask at all; pool 0: a plain sliding window; rot_dims 0: no positions; factor None: no scaling entry."""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if window:
        m["mask"] = {"size": window}
        if pool:
            m["mask"]["pool"] = pool
    if rot_dims:
        m["rot"] = {"dims": rot_dims, "base": base}
        if factor is not None:
            m["rot"]["scaling"] = {"factor": factor}
    return {"type": "attention", "mixer": m}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def layer(mixer, mlp=None):
    return dict(mixer, mlp=mlp)


def config(vocab, width, layers, loop=None, eps=1e-6):
    out = {"architecture": "Sirodra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if loop:
        out["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return out


def odd():
    """Sizes that are multiples of nothing convenient, layers before and after a loop of three passes, a window that no pool size
    divides, a pool wider than its window, feed-forwards on every kind of mixer."""
    return config(61, 44, [
        layer(attn(3, 1, 10, 7, 11, 4, 0.5, 6, base=300.0, factor=3.0), dense(30)),
        layer(mlstm(3, 6, 5, 2.5)),
        layer(hgrn(5, 6, 9), dense(21)),
        layer(attn(4, 2, 6, 9, 5, 8, 0.6, 6, base=50.0, factor=0.5)),
        layer(mlstm(1, 13, 18, 6.0), dense(10)),
        layer(hgrn(1, 11, 4)),
    ], loop=(1, 4, 3), eps=1e-2)      # eps large enough that a norm ignoring it fails


def unaligned():
    """Width not a multiple of 8 (no tensor-core product takes it), no loop, no rotation in one attention and no scaling in the
    other, neither window nor pooled blocks in one, a window without pooled blocks in the other."""
    return config(29, 36, [
        layer(attn(2, 2, 10, 6, 0, 0, 0.7)),
        layer(hgrn(2, 9, 5), dense(14)),
        layer(attn(6, 2, 8, 10, 9, 0, 0.5, 4, base=100.0), dense(18)),
        layer(mlstm(2, 4, 3, 15.0)),
    ])


def aligned():
    """Sizes the tensor-core kernels take (multiples of 16 / 64); the whole stack in a loop of two passes."""
    return config(320, 128, [
        layer(hgrn(4, 32, 48)),
        layer(attn(8, 2, 32, 64, 40, 8, 0.4, 16, base=5000.0, factor=2.0), dense(192)),
        layer(mlstm(4, 32, 64, 10.0), dense(128)),
        layer(attn(4, 4, 64, 32, 33, 3, 0.3, 64, factor=1.0)),
    ], loop=(0, 4, 2), eps=1e-5)


def once():
    """A loop of a single pass over the last layers, pooled blocks of one position and a window of one."""
    return config(37, 24, [
        layer(attn(2, 1, 8, 6, 1, 1, 0.6, 8, base=40.0, factor=1.5)),
        layer(mlstm(2, 6, 7, 3.0)),
        layer(attn(2, 2, 6, 5, 7, 1, 0.5, 2), dense(9)),
    ], loop=(1, 3, 1), eps=1e-4)


def weights(cfg, seed=0):
    """Random weights rounded to bf16 (so that bf16 and f32 runs hold the same numbers).  Queries and keys are normed per head, so a
    test that wants peaked attention rows raises the configuration's `scale`."""
    g = torch.Generator().manual_seed(seed)

    def rnd(*shape, s=1.0):
        return (s * torch.randn(*shape, generator=g)).to(torch.bfloat16).to(torch.float32)

    W, width = {}, cfg["width"]
    W["embed"] = rnd(cfg["vocab"], width)
    W["head"] = rnd(cfg["vocab"], width, s=width ** -0.5)
    W["final.norm"] = 1.0 + rnd(width, s=0.2)
    if cfg.get("loop"):
        W["loop.in"] = rnd(width, 2 * width, s=(2 * width) ** -0.5)
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        q = p + "mix."
        W[p + "norm1"] = 1.0 + rnd(width, s=0.2)
        H, d, dv = m["heads"], m["dim"], m["vdim"]
        if L["type"] == "hgrn2":
            W[q + "q"], W[q + "v"] = rnd(H * d, width, s=width ** -0.5), rnd(H * dv, width, s=width ** -0.5)
            W[q + "f"], W[q + "f.b"] = rnd(H * d, width, s=width ** -0.5), 1.0 + rnd(H * d, s=1.5)
            W[q + "lower"] = torch.rand(H * d, generator=g) * 0.95
            W[q + "norm"] = 1.0 + rnd(dv, s=0.2)
        elif L["type"] == "mlstm":
            for n, size in (("q", H * d), ("k", H * d), ("v", H * dv), ("g", H * dv)):
                W[q + n] = rnd(size, width, s=(2.0 if n == "g" else 1.0) * width ** -0.5)
            W[q + "i"], W[q + "i.b"] = rnd(H, width, s=1.5 * width ** -0.5), rnd(H, s=1.0)
            W[q + "f"], W[q + "f.b"] = rnd(H, width, s=1.5 * width ** -0.5), 2.0 + rnd(H, s=1.0)
            W[q + "norm"] = 1.0 + rnd(H * dv, s=0.2)
        else:
            G = m["kv_heads"]
            for n, size in (("q", H * d), ("k", G * d), ("v", G * dv)):
                W[q + n], W[q + n + ".b"] = rnd(size, width, s=width ** -0.5), rnd(size, s=0.3)
            W[q + "g"] = rnd(H, width, s=2.0 * width ** -0.5)
        W[q + "o"] = rnd(width, H * dv, s=(H * dv) ** -0.5)
        f = L.get("mlp")
        if f is not None:
            W[p + "norm2"] = 1.0 + rnd(width, s=0.2)
            W[p + "mlp.up"] = rnd(f["ff"], width, s=2.0 * width ** -0.5)
            W[p + "mlp.down"] = rnd(width, f["ff"], s=f["ff"] ** -0.5)
    return {k: v.to(torch.bfloat16).to(torch.float32) for k, v in W.items()}      # what a bf16 checkpoint holds
