"""Host-side parts of the Sirodra sequence model (no GPU): configuration reader, tensor inventory, packing, state declaration, and
the float64 oracle's own consistency (oracle/sirodra_oracle.py)."""
import json
import math

import pytest
import torch

import sirodra_cases as cases
from oracle import sirodra_oracle as so
from qwen3_tts_cuda_graphs_b200.config import (DenseFFConfig, ForgetGateAttentionConfig, LoopConfig, MatrixMemoryConfig,
                                               SEQUENCE_ARCHITECTURES, SoftmaxAttentionConfig, sequence_config_from_dict)

F64 = torch.float64


def test_config_reader_takes_every_size_and_constant_from_the_dictionary():
    c = sequence_config_from_dict(json.loads(json.dumps(cases.odd())))
    assert (c.vocab, c.width, c.norm_eps, len(c.layers)) == (61, 44, 1e-2, 6)
    assert c.loop == LoopConfig(1, 4, 3)
    assert [i for i, _ in c.runs] == [0] + [1, 2, 3] * 3 + [4, 5]
    assert [r for r, (_, first) in enumerate(c.runs) if first] == [1, 4, 7]
    assert c.layers[0].mixer == SoftmaxAttentionConfig(3, 1, 10, 7, 0.5, rot_dims=6, rot_base=300.0, window=11, gate=True, bias=True, out_bias=False,
                                                       rot_factor=3.0, qk_unit=True, pool=4)
    assert c.layers[0].mlp == DenseFFConfig(30) and c.layers[1].mlp is None
    assert c.layers[1].mixer == MatrixMemoryConfig(3, 6, 5, 2.5)
    assert c.layers[2].mixer == ForgetGateAttentionConfig(5, 6, 9)
    plain = sequence_config_from_dict(cases.unaligned())       # defaults of what the dictionary leaves out
    a, b = plain.layers[0].mixer, plain.layers[2].mixer
    assert plain.loop is None and plain.runs == ((0, False), (1, False), (2, False), (3, False)) and plain.norm_eps == 1e-6
    assert (a.window, a.pool, a.rot_dims) == (0, 0, 0) and (b.window, b.pool, b.rot_dims, b.rot_factor) == (9, 0, 4, 1.0)
    one = sequence_config_from_dict(cases.once())
    assert one.runs == ((0, False), (1, True), (2, False))
    mha = cases.unaligned()
    del mha["layers"][0]["mixer"]["kv_heads"]
    assert sequence_config_from_dict(mha).layers[0].mixer.kv_heads == 2
    assert "Sirodra" in SEQUENCE_ARCHITECTURES
    for breakit in (lambda d: d["layers"][3]["mixer"].update(kv_heads=3), lambda d: d["layers"][0].update(type="other"),
                    lambda d: d["layers"][0]["mixer"]["rot"].update(dims=12), lambda d: d["layers"][0]["mixer"]["rot"].update(dims=3),
                    lambda d: d["layers"][0]["mixer"]["rot"]["scaling"].update(factor=0.0), lambda d: d["layers"][0]["mixer"]["mask"].pop("size"),
                    lambda d: d["layers"][1]["mixer"].update(gate_cap=0.0), lambda d: d["layers"][0]["mlp"].update(kind="other"),
                    lambda d: d["loop"].update(stop=7), lambda d: d["loop"].update(start=4), lambda d: d["loop"].update(times=0)):
        bad = cases.odd()
        breakit(bad)
        with pytest.raises(ValueError):
            sequence_config_from_dict(bad)


def test_model_declares_the_tensors_the_test_checkpoint_holds():
    from qwen3_tts_cuda_graphs_b200.sirodra import init_synthetic, tensor_specs

    for make in (cases.odd, cases.unaligned, cases.aligned, cases.once):
        cfg = make()
        W = cases.weights(cfg)
        specs = tensor_specs(sequence_config_from_dict(cfg))
        assert set(W) == set(specs)
        assert all(tuple(W[k].shape) == tuple(specs[k]) for k in W)
        S = init_synthetic(sequence_config_from_dict(cfg))
        assert set(S) == set(specs) and all(tuple(S[k].shape) == tuple(specs[k]) for k in S)
        assert ("loop.in" in specs) == ("loop" in cfg)


def test_packing_and_state_declaration_follow_the_layer_runs():
    from qwen3_tts_cuda_graphs_b200.seq_state import SequenceStateManager
    from qwen3_tts_cuda_graphs_b200.sirodra import SirodraModel

    cfg = cases.odd()
    W = cases.weights(cfg)
    m = SirodraModel(sequence_config_from_dict(cfg), W.get, "cpu", f32=True)
    specs = {s.name: s for s in m.state_specs()}
    want = {"r0.k", "r0.v", "r0.k.pool", "r0.v.pool", "r10.mm.s", "r10.mm.m", "r11.fg"}
    for r in (1, 4, 7):      # three passes, each with states of its own
        want |= {f"r{r}.mm.s", f"r{r}.mm.m", f"r{r + 1}.fg"} | {f"r{r + 2}.{n}" for n in ("k", "v", "k.pool", "v.pool")}
    assert set(specs) == want
    assert (specs["r0.k"].cols, specs["r0.v"].cols, specs["r3.k"].cols, specs["r3.v"].cols) == (10, 7, 12, 18)
    assert (specs["r0.k.pool"].every, specs["r6.v.pool"].every, specs["r6.v.pool"].cols) == (4, 8, 18)
    s, mx, fg = specs["r4.mm.s"], specs["r4.mm.m"], specs["r5.fg"]
    assert (s.kind, s.rows, s.cols) == ("carry", 18, 6) and (mx.kind, mx.rows, mx.cols) == ("carry", 1, 3) and (fg.rows, fg.cols) == (30, 9)
    slot = SequenceStateManager(m.state_specs(), 43, "cpu", 1).acquire("a")
    assert slot.cur["r0.k"].shape == (43, 10) and slot.cur["r0.k.pool"].shape == (10, 10) and slot.cur["r3.v.pool"].shape == (5, 18)
    att = m.layers[0]["mix"]
    rows = 30 + 10 + 7 + 3
    assert att["wqkv"].shape == (56, 44) and torch.equal(att["wqkv"][:rows], torch.cat([W[f"l0.mix.{n}"] for n in "qkvg"]))
    assert not att["wqkv"][rows:].any()                       # padding rows
    assert torch.equal(att["bqkv"][:47], torch.cat([W[f"l0.mix.{n}.b"] for n in "qkv"])) and not att["bqkv"][47:].any() and att["o_b"] is None
    assert torch.allclose(att["freq"].to(F64), torch.tensor([300.0 ** (-2.0 * i / 6) / 3.0 for i in range(3)], dtype=F64), rtol=1e-6)
    mem = m.layers[1]["mix"]
    assert torch.equal(mem["win"][:72], torch.cat([W[f"l1.mix.{n}"] for n in "qkvgif"])) and mem["win"].shape == (72, 44)
    assert torch.equal(mem["bin"], torch.cat([torch.zeros(66), W["l1.mix.i.b"], W["l1.mix.f.b"]]))
    fgw = m.layers[2]["mix"]
    assert torch.equal(fgw["win"][:105], torch.cat([W[f"l2.mix.{n}"] for n in "qfv"])) and fgw["win"].shape == (112, 44)
    assert torch.equal(fgw["bin"][30:60], W["l2.mix.f.b"]) and not fgw["bin"][:30].any() and not fgw["bin"][60:].any()
    assert torch.equal(fgw["lower"], W["l2.mix.lower"])
    assert "ff" not in m.layers[1] and m.layers[0]["ff"]["up"].shape == (30, 44)
    assert torch.equal(m.g["loop.in"], W["loop.in"]) and torch.equal(m.g["head"], W["head"])
    with pytest.raises(ValueError):
        SirodraModel(sequence_config_from_dict(cfg), {**W, "l0.mix.q": W["l0.mix.q"][:-1]}.get, "cpu")
    with pytest.raises(KeyError):
        SirodraModel(sequence_config_from_dict(cfg), {k: v for k, v in W.items() if k != "loop.in"}.get, "cpu")
    bare = SirodraModel(sequence_config_from_dict(cases.unaligned()), cases.weights(cases.unaligned()).get, "cpu")
    assert bare.layers[0]["mix"]["freq"] is None and "loop.in" not in bare.g
    assert not any(".pool" in s.name for s in bare.state_specs())


def test_oracle_norms_and_activations():
    torch.manual_seed(0)
    x = torch.randn(3, 10, dtype=F64) + 5.0
    w = torch.randn(10, dtype=F64)
    assert torch.allclose(so.centred_norm(x, w, 1e-3), torch.nn.functional.layer_norm(x, (10,), w, None, 1e-3))
    assert torch.allclose(so.rms_unit(x, 0.0).pow(2).mean(-1), torch.ones(3, dtype=F64))
    z = torch.linspace(-40.0, 40.0, 33, dtype=F64)
    assert torch.allclose(so.log_sigmoid(z), torch.nn.functional.logsigmoid(z))
    assert torch.allclose(so.gelu_erf(z), torch.nn.functional.gelu(z)) and torch.allclose(so.silu(z), torch.nn.functional.silu(z))
    assert float(so.soft_cap(z, 3.0).abs().max()) <= 3.0 and abs(float(so.soft_cap(torch.tensor(0.01, dtype=F64), 3.0)) - 0.01) < 1e-6


def test_oracle_rotation():
    torch.manual_seed(1)
    v = torch.randn(6, 2, 10, dtype=F64)
    r = so.rotate(v, 6, 100.0, 4.0)
    assert torch.allclose(r[0], v[0]) and torch.allclose(r[..., 6:], v[..., 6:]) and torch.allclose((r * r).sum(-1), (v * v).sum(-1))
    c, s = math.cos(3.0 / 4.0), math.sin(3.0 / 4.0)           # pair 0 at position 3: frequency 1, divided by the factor
    assert torch.allclose(r[3, 0, 0], v[3, 0, 0] * c - v[3, 0, 1] * s) and torch.allclose(r[3, 0, 1], v[3, 0, 1] * c + v[3, 0, 0] * s)
    f1 = 100.0 ** (-2.0 / 6) / 4.0
    c, s = math.cos(5 * f1), math.sin(5 * f1)
    assert torch.allclose(r[5, 1, 2], v[5, 1, 2] * c - v[5, 1, 3] * s)
    # a rotation keeps the root mean square of a head: the unit norm may come before or after it
    assert torch.allclose(so.rms_unit(r, 1e-3), so.rotate(so.rms_unit(v, 1e-3), 6, 100.0, 4.0))


def test_oracle_visible_tokens_and_blocks():
    # window 5, blocks of 3: block b (positions 3b .. 3b + 2) from position 3b + 2 + 5 on
    assert [so.visible(i, 5, 3) for i in (0, 4, 6, 7, 9, 10, 13)] == [(0, 0), (0, 0), (2, 0), (3, 1), (5, 1), (6, 2), (9, 3)]
    assert so.visible(9, 1, 1) == (9, 9)                      # everything is seen, one by one
    assert so.visible(9, 0, 0) == (0, 0) and so.visible(9, 4, 0) == (6, 0)
    torch.manual_seed(2)
    cfg = cases.config(8, 12, [cases.layer(cases.attn(2, 1, 4, 3, 5, 3, 1.0, 2))])
    W = {k[len("l0.mix."):]: v.to(F64) for k, v in cases.weights(cfg, seed=2).items() if k.startswith("l0.mix.")}
    m = cfg["layers"][0]["mixer"]
    h = torch.randn(16, 12, dtype=F64)
    base = so.attention(h, W, "", m, 1e-6)
    h2 = h.clone()
    h2[1] += 1.0        # position 1 (block 0): in the window of 1 .. 5, unseen at 6, in its block from 7 on
    out = so.attention(h2, W, "", m, 1e-6)
    moved = [not torch.allclose(out[i], base[i], atol=1e-9) for i in range(16)]
    assert moved == [False] + [True] * 5 + [False] + [True] * 9
    # a block enters as the mean of its keys and values: equal inputs make it one more copy of a token's key
    same = h[:1].expand(16, 12).clone()
    m0 = {k: v for k, v in m.items() if k != "rot"}
    o = so.attention(same, W, "", m0, 1e-6)
    assert torch.allclose(o, o[:1].expand_as(o))


def test_oracle_recurrences_against_their_sums():
    torch.manual_seed(3)
    T, width = 7, 8
    h = torch.randn(T, width, dtype=F64)
    r = lambda *s: torch.randn(*s, dtype=F64)     # noqa: E731
    W = {"q": r(4, width), "f": r(4, width), "f.b": r(4), "lower": torch.rand(4, dtype=F64), "v": r(3, width), "norm": r(3), "o": torch.eye(3, dtype=F64)}
    got = so.hgrn2(h, W, "", {"heads": 1, "dim": 4, "vdim": 3}, 1e-6)
    f = W["lower"] + (1 - W["lower"]) * torch.sigmoid(h @ W["f"].T + W["f.b"])
    q, v = torch.nn.functional.silu(h @ W["q"].T), h @ W["v"].T
    for t in range(T):
        o = torch.zeros(3, dtype=F64)
        for j in range(t + 1):
            o = o + (q[t] * (1 - f[j]) * f[j + 1:t + 1].prod(0)).sum() * v[j]
        assert torch.allclose(got[t], so.rms_unit(o, 1e-6) * W["norm"])
    W = {"q": r(4, width), "k": r(4, width), "v": r(3, width), "g": r(3, width), "i": r(1, width), "i.b": r(1), "f": r(1, width), "f.b": r(1),
         "norm": r(3), "o": torch.eye(3, dtype=F64)}
    got = so.mlstm(h, W, "", {"heads": 1, "dim": 4, "vdim": 3, "gate_cap": 2.0}, 1e-6)
    q, k, v = h @ W["q"].T / 2.0, h @ W["k"].T, h @ W["v"].T
    li = 2.0 * torch.tanh((h @ W["i"].T + W["i.b"]) / 2.0)[:, 0]
    lf = torch.nn.functional.logsigmoid(2.0 * torch.tanh((h @ W["f"].T + W["f.b"]) / 2.0))[:, 0]
    for t in range(T):       # without the maximum: weights e^(li_j + sum of later lf), the divisor's floor is 1 (plus 1e-6 at its scale)
        a = [(torch.exp(li[j] + lf[j + 1:t + 1].sum()) * (q[t] @ k[j])) for j in range(t + 1)]
        mx = max([float(lf[:t + 1].sum())] + [float(li[j] + lf[j + 1:t + 1].sum()) for j in range(t + 1)])
        o = sum(a[j] * v[j] for j in range(t + 1)) / (max(abs(float(sum(a))), 1.0) + 1e-6 * math.exp(mx))
        assert torch.allclose(got[t], so.rms_unit(o, 1e-6) * W["norm"] * torch.sigmoid(h[t] @ W["g"].T), atol=1e-10)


def test_oracle_loops_and_skips_absent_feed_forwards():
    cfg = cases.odd()
    W = cases.weights(cfg, seed=5)
    toks = cases.tokens(cfg, 12)
    taps = []
    out = so.forward(cfg, W, toks, taps)
    assert out.shape == (12, 61) and len(taps) == 12
    other = list(toks)
    other[8] = (other[8] + 1) % 61            # causal: a later token changes nothing before it
    assert torch.allclose(so.forward(cfg, W, other)[:8], out[:8])
    # a loop unrolled by hand: the pass mixes the embedding output in, then runs the layers
    W64 = {k: v.to(F64) for k, v in W.items()}
    x0 = W64["embed"][torch.as_tensor(toks)]
    x = so.layer(0, cfg, x0, W64)
    for _ in range(3):
        x = x @ W64["loop.in"][:, :44].T + x0 @ W64["loop.in"][:, 44:].T
        for i in (1, 2, 3):
            x = so.layer(i, cfg, x, W64)
    assert torch.allclose(taps[9], x)
