"""Host-side parts of the Matidra sequence model (no GPU): configuration reader, tensor inventory, packing, state declaration, and
the float64 oracle's own consistency (oracle/matidra_oracle.py)."""
import json
import math

import pytest
import torch

import matidra_cases as cases
from oracle import matidra_oracle as mo
from qwen3_tts_cuda_graphs_b200.config import (ChannelDeltaRuleConfig, DenseFFConfig, SEQUENCE_ARCHITECTURES, ScaledPairMixerConfig,
                                               SoftmaxAttentionConfig, sequence_config_from_dict)

F64 = torch.float64


def test_config_reader_takes_every_size_and_constant_from_the_dictionary():
    c = sequence_config_from_dict(json.loads(json.dumps(cases.odd())))
    assert (c.vocab, c.width, c.norm_eps, c.alpha, len(c.layers)) == (61, 44, 1e-2, 1.4, 5)
    m = c.layers[0].mixer
    assert m == ScaledPairMixerConfig(SoftmaxAttentionConfig(4, 2, 10, 7, 0.4, qk_norm=True, conv=3, q_temp=(0.6, 5.0), entry_gate=True),
                                      ChannelDeltaRuleConfig(6, 2, 6, 9, 5), 0.7, 1.6)
    assert c.layers[0].mlp == DenseFFConfig(30) and c.layers[1].mlp is None
    assert c.layers[1].mixer == SoftmaxAttentionConfig(3, 1, 14, 14, 0.3, rot_dims=10, rot_base=300.0, rot_scaling=(3.0, 64.0, 4.0, 1.5),
                                                       qk_norm=True, keys_as_values=True)
    assert c.layers[3].mixer.rot_scaling is None and c.layers[3].mixer.rot_dims == 6
    assert c.layers[4].mixer.left.q_temp is None and c.layers[4].mixer.left.conv == 1
    d = cases.unaligned()       # defaults of what the dictionary leaves out
    del d["layers"][0]["mixer"]["kv_heads"], d["layers"][1]["mixer"]["left"]["kv_heads"], d["layers"][1]["mixer"]["right"]["kv_heads"]
    c = sequence_config_from_dict(d)
    assert c.layers[0].mixer.kv_heads == 2 and c.layers[0].mixer.rot_dims == 0
    assert c.layers[1].mixer.left.kv_heads == 2 and c.layers[1].mixer.right.kv_heads == 2
    assert "Matidra" in SEQUENCE_ARCHITECTURES
    for breakit in (lambda d: d["layers"][1]["mixer"].update(kv_heads=2), lambda d: d["layers"][0].update(type="other"),
                    lambda d: d["layers"][1]["mixer"]["rot"].update(dims=16), lambda d: d["layers"][1]["mixer"]["rot"].update(dims=3),
                    lambda d: d["layers"][1]["mixer"]["rot"]["scaling"].update(factor=0.0), lambda d: d["layers"][1]["mixer"].update(vdim=13),
                    lambda d: d["layers"][0]["mixer"]["left"].update(kv_heads=3), lambda d: d["layers"][0]["mixer"]["right"].update(kv_heads=4),
                    lambda d: d["layers"][0]["mixer"]["left"].update(conv=0), lambda d: d["layers"][0]["mixer"]["left"]["q_temp"].update(every=0),
                    lambda d: d["layers"][0]["mlp"].update(kind="other")):
        bad = cases.odd()
        breakit(bad)
        with pytest.raises(ValueError):
            sequence_config_from_dict(bad)


def test_model_declares_the_tensors_the_test_checkpoint_holds():
    from qwen3_tts_cuda_graphs_b200.matidra import init_synthetic, tensor_specs

    for make in (cases.odd, cases.unaligned, cases.aligned):
        cfg = make()
        W = cases.weights(cfg)
        specs = tensor_specs(sequence_config_from_dict(cfg))
        assert set(W) == set(specs)
        assert all(all(b is None or a == b for a, b in zip(W[k].shape, specs[k])) and len(W[k].shape) == len(specs[k]) for k in W)
        S = init_synthetic(sequence_config_from_dict(cfg))
        assert set(S) == set(specs) and all(all(b is None or a == b for a, b in zip(S[k].shape, specs[k])) for k in S)


def test_packing_and_state_declaration():
    from qwen3_tts_cuda_graphs_b200.matidra import MatidraModel
    from qwen3_tts_cuda_graphs_b200.seq_state import SequenceStateManager

    cfg = cases.odd()
    W = cases.weights(cfg)
    m = MatidraModel(sequence_config_from_dict(cfg), W.get, "cpu", f32=True)
    specs = {s.name: s for s in m.state_specs()}
    assert set(specs) == {f"l{i}.{n}" for i in range(5) for n in ("k", "v")} | {f"l{i}.kd.{n}" for i in (0, 2, 4) for n in ("conv", "s")}
    nl, nr = 4 * 10 + 2 * 10 + 2 * 7, 2 * 2 * 6 + 6 * 9
    c, s = specs["l0.kd.conv"], specs["l0.kd.s"]
    assert (c.rows, c.cols, c.in_place) == (4, nl + nr, False) and (s.rows, s.cols, s.in_place) == (36, 9, True)
    assert specs["l4.kd.conv"].rows == 0                      # a single tap carries nothing
    assert (specs["l0.k"].cols, specs["l0.v"].cols, specs["l1.k"].cols, specs["l1.v"].cols) == (20, 14, 14, 14)
    slot = SequenceStateManager(m.state_specs(), 43, "cpu", 1).acquire("a")
    assert slot.cur["l1.v"].shape == (43, 14) and "l4.kd.conv" not in slot.cur and slot.cur["l0.kd.s"] is slot.next["l0.kd.s"]
    mix = m.layers[0]["mix"]
    order = [f"l0.mix.left.{n}" for n in "qkv"] + [f"l0.mix.right.{n}" for n in "qkv"]
    rest = ["l0.mix.left.g"] + [f"l0.mix.right.{n}" for n in ("b", "a1", "g1")]
    rows = nl + nr + 28 + 6 + 5 + 7
    assert mix["win"].shape == (-(-rows // 8) * 8, 44) and torch.equal(mix["win"][:rows], torch.cat([W[n] for n in order + rest]))
    assert not mix["win"][rows:].any()
    assert mix["conv"].shape == (nl + nr, 5) and not mix["conv"][:nl, :2].any()          # three taps beside five: zeros in front
    assert torch.equal(mix["conv"][:40, 2:], W["l0.mix.left.q.conv"]) and torch.equal(mix["conv"][nl:nl + 12], W["l0.mix.right.q.conv"])
    assert torch.equal(mix["o"], torch.cat([W["l0.mix.left.o"], W["l0.mix.right.o"]], 1))
    assert torch.allclose(mix["right"]["norm"], 1.6 * W["l0.mix.right.norm"])
    att = m.layers[1]["mix"]
    assert torch.equal(att["wqkv"][:56], torch.cat([W["l1.mix.q"], W["l1.mix.k"]])) and att["wqkv"].shape == (56, 44)
    f, amp = mo.rotary_table(10, 300.0, cfg["layers"][1]["mixer"]["rot"]["scaling"])
    assert torch.allclose(att["freq"].to(F64) + att["freq_lo"].to(F64), torch.tensor(f, dtype=F64), rtol=1e-12) and abs(att["amp"] - amp) < 1e-15
    ff = m.layers[0]["ff"]["gate_up"]
    assert torch.equal(ff[0::2], W["l0.mlp.gate"]) and torch.equal(ff[1::2], W["l0.mlp.up"])
    assert "ff" not in m.layers[1] and torch.equal(m.g["sum"], torch.tensor([1.4, 1.0]))
    with pytest.raises(ValueError):
        MatidraModel(sequence_config_from_dict(cfg), {**W, "l0.mix.left.q": W["l0.mix.left.q"][:-1]}.get, "cpu")
    with pytest.raises(ValueError):      # the low-rank factors disagree
        MatidraModel(sequence_config_from_dict(cfg), {**W, "l0.mix.right.a1": W["l0.mix.right.a1"][:-1]}.get, "cpu")
    with pytest.raises(KeyError):
        MatidraModel(sequence_config_from_dict(cfg), {k: v for k, v in W.items() if k != "final.norm.b"}.get, "cpu")


def test_oracle_norms_activations_and_convolution():
    torch.manual_seed(0)
    x = torch.randn(3, 10, dtype=F64) + 5.0
    w, b = torch.randn(10, dtype=F64), torch.randn(10, dtype=F64)
    assert torch.allclose(mo.layer_norm(x, w, b, 1e-3), torch.nn.functional.layer_norm(x, (10,), w, b, 1e-3))
    assert torch.allclose(mo.rms_unit(x, 0.0).pow(2).mean(-1), torch.ones(3, dtype=F64))
    assert torch.allclose(mo.unit(x).pow(2).sum(-1), torch.ones(3, dtype=F64), atol=1e-6)
    z = torch.linspace(-40.0, 40.0, 33, dtype=F64)
    assert torch.allclose(mo.softplus(z), torch.nn.functional.softplus(z)) and torch.allclose(mo.silu(z), torch.nn.functional.silu(z))
    assert torch.allclose(mo.gelu_tanh(z), torch.nn.functional.gelu(z, approximate="tanh"))
    u, k = torch.randn(9, 4, dtype=F64), torch.randn(4, 3, dtype=F64)
    want = torch.nn.functional.conv1d(torch.nn.functional.pad(u.T, (2, 0)), k[:, None], groups=4).T
    assert torch.allclose(mo.time_conv(u, k), want) and torch.allclose(mo.time_conv(u, k[:, 2:]), u * k[:, 2])


def test_oracle_rotation_and_its_scaled_table():
    torch.manual_seed(1)
    v = torch.randn(6, 2, 10, dtype=F64)
    r = mo.rotate(v, 6, 100.0)
    assert torch.allclose(r[0], v[0]) and torch.allclose(r[..., 6:], v[..., 6:]) and torch.allclose((r * r).sum(-1), (v * v).sum(-1))
    c, s = math.cos(3.0), math.sin(3.0)
    assert torch.allclose(r[3, 0, 0], v[3, 0, 0] * c - v[3, 0, 1] * s) and torch.allclose(r[3, 0, 1], v[3, 0, 1] * c + v[3, 0, 0] * s)
    # a table of eight frequencies, base e^2: entry n(t) = 16 ln(128 / (2 pi t)) / 4; fast 4 -> 6.5.., slow 1 -> 12.06..
    sc = {"factor": 5.0, "original": 128, "fast": 4.0, "slow": 1.0}
    f, amp = mo.rotary_table(16, math.e ** 2, sc)
    plain, one = mo.rotary_table(16, math.e ** 2, None)
    assert one == 1.0 and abs(amp - (0.1 * math.log(5.0) + 1.0)) < 1e-15
    lo = math.floor(16 * math.log(128 / (8 * math.pi)) / 4)
    hi = math.ceil(16 * math.log(128 / (2 * math.pi)) / 4)
    assert (lo, hi) == (6, 13)
    assert f[:7] == plain[:7]                                 # at and below the fast end: unchanged
    assert abs(f[7] - (plain[7] / 5.0 / 7.0 + plain[7] * 6.0 / 7.0)) < 1e-15
    scaled = mo.rotate(v, 6, 100.0, {"factor": 3.0, "original": 64, "fast": 2.0, "slow": 1.0})
    a = 0.1 * math.log(3.0) + 1.0
    assert torch.allclose(scaled[0, :, :6], a * v[0, :, :6]) and torch.allclose(scaled[..., 6:], v[..., 6:])


def test_oracle_attention_and_temperature():
    torch.manual_seed(2)
    q, k, v = torch.randn(7, 4, 5, dtype=F64), torch.randn(7, 2, 5, dtype=F64), torch.randn(7, 2, 3, dtype=F64)
    got = mo.causal_softmax(q, k, v, 0.7)
    kk, vv = k.repeat_interleave(2, 1), v.repeat_interleave(2, 1)
    want = torch.nn.functional.scaled_dot_product_attention(q.transpose(0, 1), kk.transpose(0, 1), vv.transpose(0, 1), is_causal=True, scale=0.7).transpose(0, 1)
    assert torch.allclose(got, want)
    t = mo.temperature(12, 0.5, 4)
    assert torch.equal(t[:3], torch.ones(3, dtype=F64)) and torch.allclose(t[3:7], torch.tensor(1 + 0.5 * math.log(2.0), dtype=F64))
    assert abs(float(t[11]) - (1 + 0.5 * math.log(4.0))) < 1e-15


def test_oracle_delta_walk_against_its_definition():
    """With orthonormal keys, write strength one and no decay the state is an exact associative memory; a decay acts on its own row only."""
    d = 4
    k = torch.eye(d, dtype=F64)[:, None, :]
    v = torch.randn(d, 1, 3, dtype=F64)
    ones = torch.ones(d, 1, d, dtype=F64)
    o = mo.delta_walk(k, k, v, ones, torch.ones(d, 1, dtype=F64))
    assert torch.allclose(o, v)                               # the read-out sees the current token's write
    kk, vv = torch.cat([k, k]), torch.cat([v, torch.zeros_like(v)])
    g = torch.cat([ones, ones])
    g[d:, :, 2] = 0.5
    o = mo.delta_walk(kk, kk, vv, g, torch.cat([torch.ones(d, 1, dtype=F64), torch.zeros(d, 1, dtype=F64)]))
    assert torch.allclose(o[d + 1], v[1]) and torch.allclose(o[d + 2], 0.125 * v[2]) and torch.allclose(o[d + 3], v[3])
    # the correction reads the decayed state: writing v over half of v with strength one leaves v
    o = mo.delta_walk(k[[2, 2]], k[[2, 2]], v[[2, 2]], g[[d, d]], torch.ones(2, 1, dtype=F64))
    assert torch.allclose(o[1], v[2])


def test_oracle_model_is_causal_and_norms_come_behind_the_sums():
    cfg = cases.odd()
    W = cases.weights(cfg, seed=5)
    toks = cases.tokens(cfg, 12)
    taps = []
    out = mo.forward(cfg, W, toks, taps)
    assert out.shape == (12, 61) and len(taps) == 5
    other = list(toks)
    other[8] = (other[8] + 1) % 61
    assert torch.allclose(mo.forward(cfg, W, other)[:8], out[:8])
    W64 = {k: v.to(F64) for k, v in W.items()}
    x = W64["embed"][torch.as_tensor(toks)]
    m = cfg["layers"][0]["mixer"]
    mixed = 0.7 * mo.convolved_attention(x, W64, "l0.mix.left.", m["left"], 1e-2) + 1.6 * mo.channel_delta_rule(x, W64, "l0.mix.right.", m["right"], 1e-2)
    x = torch.nn.functional.layer_norm(1.4 * x + mixed, (44,), W64["l0.norm1"], W64["l0.norm1.b"], 1e-2)
    z = torch.nn.functional.gelu(x @ W64["l0.mlp.gate"].T, approximate="tanh") * (x @ W64["l0.mlp.up"].T) @ W64["l0.mlp.down"].T
    x = torch.nn.functional.layer_norm(1.4 * x + z, (44,), W64["l0.norm2"], W64["l0.norm2.b"], 1e-2)
    assert torch.allclose(taps[0], x)
