"""The Matidra sequence model on the CUDA op-list path against the float64 oracle (oracle/matidra_oracle.py).

Mechanisms alone (seq_ops.StepBuilder fragments), then whole models: prompts, prompts in portions down to two tokens, token by
token decoding through the caches and carried states, slots that are given back and used again, requests that take turns, keys far
back and on both sides of the kernels' tiles, positions at which the query temperature steps, long decoding, sizes that are multiples
of nothing, and greedy generation through the engine's entry point, the scheduler and the command line.
"""
import pytest
import torch

import matidra_cases as cases
from oracle import matidra_oracle as mo

pytestmark = pytest.mark.gpu

F64 = torch.float64
DEV = "cuda"
TOL = {True: 3e-4, False: 6e-2}      # true 32-bit / bf16 products


def make_engine(cfg, W, f32=True, max_tokens=700, max_slots=2):
    from qwen3_tts_cuda_graphs_b200.config import sequence_config_from_dict
    from qwen3_tts_cuda_graphs_b200.seq_engine import SequenceEngine, model_class

    model = model_class(cfg["architecture"])(sequence_config_from_dict(cfg), W.get, DEV, f32=f32)
    return SequenceEngine(model, max_tokens, max_slots)


def row_errors(got, want):
    """Per row: RMS of the mean-free difference, relative to the RMS of the wanted row."""
    got, want = got.to(F64).cpu(), want.to(F64)
    d = got - want
    d = d - d.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / want.pow(2).mean(-1).sqrt().clamp_min(1e-9)


def close_enough(got, want, f32):
    """True 32-bit: every row within the tolerance.  bf16 products: rounding noise grows at a few positions of these tiny random
    models (a peaked softmax's near-tie, a read-out that nearly vanishes before its norm), so nine rows in ten must be within the
    tolerance and the typical one well within it; a wrong key, a wrong position or a lost state moves far more."""
    e = row_errors(got, want)
    if f32:
        return float(e.max()) < TOL[True]
    return float(e.quantile(0.9)) < TOL[False] and float(e.median()) < TOL[False] / 2


def run_schedule(eng, toks, portions, name="r"):
    """Feed toks in the given portions (the rest one by one); logits of every position, [T, vocab]."""
    rows, at = [], 0
    for n in list(portions) + [1] * (len(toks) - sum(portions)):
        part = toks[at:at + n]
        rows.append(eng.step(name, part, list(range(len(part)))).clone())
        at += n
    eng.close(name)
    return torch.cat(rows, 0)


class Bench:
    """A StepBuilder around hand-made state: runs one mechanism for a sequence of portions."""

    def __init__(self, specs, f32=True, max_pos=700):
        from qwen3_tts_cuda_graphs_b200 import codec
        from qwen3_tts_cuda_graphs_b200.seq_state import SequenceStateManager

        self.codec, self.f32 = codec, f32
        self.lib = codec.load_lib()
        self.mgr = SequenceStateManager(specs, max_pos, torch.device(DEV), 1)
        self.slot = self.mgr.acquire("t")

    def run(self, M, build):
        from qwen3_tts_cuda_graphs_b200.seq_ops import StepBuilder

        b = StepBuilder(torch.device(DEV), M, self.slot, self.f32)
        out = build(b)
        b.commit()
        self.codec.run_op_plan(self.lib, b.finish(), False)
        torch.cuda.synchronize()
        return out

    def portions(self, h, sizes, build, width):
        rows, at, T = [], 0, h.shape[0]
        for n in list(sizes) + [1] * (T - sum(sizes)):
            part = h[at:at + n].to(DEV, torch.float32 if self.f32 else torch.bfloat16).contiguous()
            out = torch.zeros(n, width, device=DEV)
            self.run(n, lambda b: build(b, part, out))
            rows.append(out.cpu())
            at += n
        return torch.cat(rows)


def cuda(t, dtype=torch.float32):
    return t.to(DEV, dtype).contiguous()


def bf(t):
    return t.to(torch.bfloat16).to(torch.float32)


def packer(W, f32=True):
    from qwen3_tts_cuda_graphs_b200.matidra import Packer

    return Packer(lambda n: W[n].to(torch.float32), DEV, f32)


def sub_weights(cfg, prefix, seed, **kw):
    return {k[len(prefix):]: v for k, v in cases.weights(cfg, seed=seed, **kw).items() if k.startswith(prefix)}


def wide(W):
    return {k: v.to(F64) for k, v in W.items()}


def layer_config(cfg, i=0):
    from qwen3_tts_cuda_graphs_b200.config import sequence_config_from_dict

    return sequence_config_from_dict(cfg).layers[i]


def kv_specs(G, d, dv, f32):
    from qwen3_tts_cuda_graphs_b200.seq_state import StateSpec

    dt = torch.float32 if f32 else torch.bfloat16
    return [StateSpec("k", "append", G * d, dtype=dt), StateSpec("v", "append", G * dv, dtype=dt)]


# ---------------------------------------------------------------------------------------------------------------------------
# mechanisms alone
# ---------------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("M,N", [(1, 36), (3, 64), (7, 37), (40, 1028), (5, 4500)])
def test_norm_behind_the_sum(M, N, f32):
    """The stream becomes the normed row; its copy as an operand is the same row rounded once.  Widths with and without 16-byte rows,
    and one that does not fit a block's registers."""
    torch.manual_seed(N)
    eps, dt = 1e-1, torch.float32 if f32 else torch.bfloat16
    parts, w, nw, nb = torch.randn(3, M, N) + 2.0, torch.tensor([1.3, -0.4, 0.7]), torch.randn(N), torch.randn(N)
    want = mo.layer_norm((w.to(F64)[:, None, None] * parts.to(F64)).sum(0), nw.to(F64), nb.to(F64), eps)
    for with_copy in (True, False):
        p, copy = cuda(parts), torch.zeros(M, N, device=DEV, dtype=dt)
        Bench([], f32).run(M, lambda b: b.sum_norm(p, 3, cuda(w), norm_w=cuda(nw), norm_b=cuda(nb), norm_out=copy if with_copy else None, eps=eps,
                                                   center=True, post=True))
        assert torch.allclose(p[0].cpu().to(F64), want, atol=2e-5) and torch.equal(p[1:].cpu(), parts[1:])
        if with_copy:
            assert torch.equal(copy, p[0].to(dt))
    # in front of a sublayer: the sum stays, the copy is normed with the bias
    p, copy = cuda(parts), torch.zeros(M, N, device=DEV)
    Bench([], True).run(M, lambda b: b.sum_norm(p, 3, cuda(w), norm_w=cuda(nw), norm_b=cuda(nb), norm_out=copy, eps=eps, center=True))
    assert torch.allclose(copy.cpu().to(F64), want, atol=2e-5)
    assert torch.allclose(p[0].cpu().to(F64), (w.to(F64)[:, None, None] * parts.to(F64)).sum(0), atol=2e-5)


@pytest.mark.parametrize("M,groups,size", [(3, 1, 36), (5, 3, 7), (300, 4, 64)])
def test_group_norm_with_a_bias_and_an_output_column(M, groups, size):
    torch.manual_seed(size)
    N, eps = groups * size, 1e-2
    x, w, b = torch.randn(M, N) * 3 + 1, torch.randn(N), torch.randn(N)
    unit = mo.layer_norm(x.to(F64).reshape(M, groups, size), torch.ones(size, dtype=F64), torch.zeros(size, dtype=F64), eps).reshape(M, N)
    out = torch.full((M, N + 12), 7.0, device=DEV)
    Bench([]).run(M, lambda sb: sb.group_norm(cuda(x), cuda(w), groups, eps, out, center=True, bias=cuda(b), out_col=8))
    assert torch.allclose(out[:, 8:8 + N].cpu().to(F64), unit * w.to(F64) + b.to(F64), atol=2e-5)
    assert (out[:, :8] == 7.0).all() and (out[:, 8 + N:] == 7.0).all()


@pytest.mark.parametrize("taps,N,split", [(1, 20, 8), (2, 13, 5), (3, 24, 12), (4, 64, 0), (5, 32, 32), (8, 16, 4), (11, 12, 4)])
def test_short_convolution_with_and_without_silu(taps, N, split):
    """Columns below `split` pass plainly, the others through silu; portions on both sides of the many-rows kernel."""
    from qwen3_tts_cuda_graphs_b200.seq_state import StateSpec

    torch.manual_seed(taps)
    T = 230
    u, w = torch.randn(T, N), torch.randn(N, taps)
    want = mo.time_conv(u.to(F64), w.to(F64))
    want[:, split:] = mo.silu(want[:, split:])
    for sizes in ([T], [64, 2, 65, 3], [5, 1, 130, 80], [2] * 20):
        bench = Bench([StateSpec("c", "carry", N, taps - 1)])
        got = bench.portions(u, sizes, lambda b, rows, out: b.time_conv(rows, cuda(w), "c", out, silu=True, silu_from=split), N)
        assert torch.allclose(got.to(F64), want, atol=1e-5), sizes


@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("M,width,ff", [(1, 36, 20), (3, 64, 128), (6, 48, 64), (200, 128, 192), (300, 64, 96), (50, 20, 7), (130, 72, 129)])
def test_dense_gated_gelu_feed_forward(M, width, ff, f32):
    torch.manual_seed(M)
    x = bf(torch.randn(M, width) * 1.5)
    W = {n: bf(torch.randn(ff, width) * 2 * width ** -0.5) for n in ("gate", "up")}
    W["down"] = bf(torch.randn(width, ff) * ff ** -0.5)
    want = mo.dense_ff(x.to(F64), wide(W), "")
    dt = torch.float32 if f32 else torch.bfloat16
    packed = {"gate_up": cuda(torch.stack([W["gate"], W["up"]], 1).reshape(2 * ff, width), dt), "down": cuda(W["down"], dt)}
    out = torch.zeros(M, width, device=DEV)
    Bench([], f32).run(M, lambda b: b.gelu_glu_ff(cuda(x, dt), packed, out))
    e = row_errors(out, want)
    assert float(e.max()) < (1e-5 if f32 else 2e-2)


ATTN_CASES = {
    # name: (H, G, d, rot_dims, base, scaling, scale, width, T, portions)
    "no_positions": (3, 1, 10, 0, 1.0, None, 0.6, 24, 60, [41, 2]),
    "whole_heads_turn": (4, 4, 6, 6, 40.0, None, 0.8, 20, 70, [2, 3, 50]),
    "part_of_a_head_scaled": (6, 2, 14, 8, 200.0, (3.0, 48, 6.0, 1.5), 0.5, 36, 90, [33, 31, 2]),
    "scaled_below_one_turn": (2, 1, 12, 12, 90.0, (2.5, 20, 1.0, 0.3), 0.5, 28, 50, [1, 48]),
    "scaled_ends_meet": (2, 2, 8, 4, 30.0, (2.0, 10, 40.0, 39.0), 0.5, 16, 40, [40]),
    "tensor_core_sizes": (8, 2, 32, 16, 3000.0, (4.0, 128, 8.0, 1.0), 0.4, 64, 200, [64, 66, 2, 40]),
    "wide_heads": (2, 1, 112, 64, 1000.0, (8.0, 512, 12.0, 2.0), 0.2, 48, 150, [130]),
    "five_heads_a_group": (5, 1, 48, 32, 500.0, (1.5, 100, 5.0, 1.0), 0.3, 48, 120, [100, 2]),
}


@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("case", list(ATTN_CASES))
def test_attention_on_keys_as_values_alone(case, f32):
    H, G, d, rd, base, scaling, scale, width, T, portions = ATTN_CASES[case]
    eps = 1e-2
    cfg = cases.config(8, width, [cases.layer(cases.attn(H, G, d, scale, rd, base, scaling))], eps=eps)
    W = sub_weights(cfg, "l0.mix.", seed=len(case))
    m, c = cfg["layers"][0]["mixer"], layer_config(cfg).mixer
    torch.manual_seed(5)
    h = bf(torch.randn(T, width))
    want = mo.keys_as_values_attention(h.to(F64), wide(W), "", m, eps)
    bench = Bench(kv_specs(G, d, d, f32), f32, max_pos=T + 3)
    w = packer(W, f32).attention("", c)
    got = bench.portions(h, portions, lambda b, rows, out: b.softmax_attention(rows, c, w, "k", "v", out, eps=eps), width)
    assert close_enough(got, want, f32), float(row_errors(got, want).max())
    if f32:
        v = bench.slot.cur["v"][:T].cpu()
        assert torch.allclose(v.to(F64), (h.to(F64) @ W["k"].to(F64).T), atol=1e-4)        # values are the keys as projected
        # the premises: without the table's scaling, or with a tenth of a turn more or less, it is another function
        if scaling:
            for other in (dict(m, rot=dict(m["rot"], scaling=None)), dict(m, rot=dict(m["rot"], scaling=dict(m["rot"]["scaling"], factor=scaling[0] * 1.2)))):
                assert float(row_errors(mo.keys_as_values_attention(h.to(F64), wide(W), "", other, eps), want).max()) > 10 * TOL[True]


def test_angles_stay_exact_thousands_of_positions_on():
    """Scores of +-60 between keys that turn fast, 2400 positions in: an angle only as good as one 32-bit product would show."""
    H, G, d, width, T = 1, 1, 32, 16, 2400
    cfg = cases.config(8, width, [cases.layer(cases.attn(H, G, d, 2.0, 32, 7.0, (0.7, 100, 9.0, 1.0)))])
    W = sub_weights(cfg, "l0.mix.", seed=31)
    torch.manual_seed(14)
    h = bf(torch.randn(T, width))
    want = mo.keys_as_values_attention(h.to(F64), wide(W), "", cfg["layers"][0]["mixer"], 1e-6)
    c = layer_config(cfg).mixer
    bench = Bench(kv_specs(G, d, d, True), True, max_pos=T)
    w = packer(W, True).attention("", c)
    got = bench.portions(h, [2390, 2], lambda b, rows, out: b.softmax_attention(rows, c, w, "k", "v", out, eps=1e-6), width)
    assert float(row_errors(got, want).max()) < 1e-4, float(row_errors(got, want).max())


CONV_CASES = {
    # name: (H, G, d, dv, taps, temp, scale, width, T, portions)
    "grouped_three_taps": (4, 2, 10, 7, 3, (0.7, 6), 0.5, 24, 70, [2, 3, 1, 40]),
    "one_tap_no_temperature": (2, 2, 6, 9, 1, None, 0.7, 20, 50, [50]),
    "eleven_taps": (3, 1, 8, 12, 11, (0.4, 1), 0.5, 20, 60, [4, 2, 5, 30]),
    "tensor_core_sizes": (4, 2, 32, 64, 4, (0.3, 40), 0.3, 64, 220, [63, 3, 100, 2]),
    "values_wider_than_keys": (6, 6, 16, 112, 4, (0.5, 33), 0.4, 48, 150, [129]),
    "three_heads_a_group": (6, 2, 48, 32, 2, (0.9, 100), 0.25, 48, 205, [200]),
}


def conv_specs(G, d, dv, channels, taps, f32):
    from qwen3_tts_cuda_graphs_b200.seq_state import StateSpec

    return kv_specs(G, d, dv, f32) + [StateSpec("k.conv", "carry", channels, taps - 1)]


@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("case", list(CONV_CASES))
def test_convolved_attention_with_temperature_and_entry_gates_alone(case, f32):
    H, G, d, dv, taps, temp, scale, width, T, portions = CONV_CASES[case]
    eps = 1e-2
    m = cases.left(H, G, d, dv, taps, scale, temp)
    cfg = cases.config(8, width, [cases.layer(cases.pair(m, cases.right(1, 1, 4, 4, 1), 1.0, 1.0))], eps=eps)
    W = sub_weights(cfg, "l0.mix.left.", seed=len(case))
    c = layer_config(cfg).mixer.left
    torch.manual_seed(6)
    h = bf(torch.randn(T, width))
    want = mo.convolved_attention(h.to(F64), wide(W), "", m, eps)
    bench = Bench(conv_specs(G, d, dv, (H + G) * d + G * dv, taps, f32), f32, max_pos=T + 3)
    w = packer(W, f32).convolved_attention("")
    got = bench.portions(h, portions, lambda b, rows, out: b.softmax_attention(rows, c, w, "k", "v", out, eps=eps), width)
    assert close_enough(got, want, f32), float(row_errors(got, want).max())
    if f32:
        one = {**W, "g": W["g"].reshape(H, dv, width)[:, :1].expand(H, dv, width).reshape(H * dv, width)}        # a gate per head is not the same
        assert float(row_errors(mo.convolved_attention(h.to(F64), wide(one), "", m, eps), want).median()) > 10 * TOL[True]


@pytest.mark.parametrize("f32", [True, False])
def test_query_temperature_steps_at_the_right_position(f32):
    """Two kinds of keys whose scores differ: the softmax between them shows the temperature of each position.  It steps when p + 1
    reaches a multiple of `every`, in prompts and in decoding."""
    H, d, dv, width, T, every = 1, 16, 16, 16, 150, 37
    m = cases.left(H, 1, d, dv, 1, 0.025, (2.0, every))
    cfg = cases.config(8, width, [cases.layer(cases.pair(m, cases.right(1, 1, 4, 4, 1), 1.0, 1.0))])
    c = layer_config(cfg).mixer.left
    W = {"q": torch.zeros(d, width), "k": torch.zeros(d, width), "v": torch.zeros(dv, width), "g": torch.zeros(dv, width), "o": torch.eye(width),
         "q.norm": torch.ones(d), "k.norm": torch.ones(d), "q.conv": torch.ones(d, 1), "k.conv": torch.ones(d, 1), "v.conv": torch.ones(dv, 1)}
    W["q"][0, 0], W["k"][0, 1], W["k"][1, 2] = 1.0, 1.0, 1.0           # keys lie along the query's axis (channel 1) or across it (channel 2)
    W["v"][0, 1], W["v"][1, 2] = 1.0, 1.0
    h = torch.zeros(T, width)
    h[:, 0] = 1.0
    h[0::2, 1], h[1::2, 2] = 1.0, 1.0
    want = mo.convolved_attention(h.to(F64), wide(W), "", m, 1e-6)
    share = want[:, 0] / (want[:, 0] + want[:, 1])
    for edge in range(every - 1, T, every):      # the premise: a step of the temperature moves an output far more than the tolerance
        assert abs(float(share[edge] - share[edge - 2])) > 2e-2
    for portions in ([T], [every - 1, 2, 34], [every, 36, 2], [70, 2, 2]):
        bench = Bench(conv_specs(1, d, dv, 2 * d + dv, 1, f32), f32, max_pos=T)
        w = packer(W, f32).convolved_attention("")
        got = bench.portions(h, portions, lambda b, rows, out: b.softmax_attention(rows, c, w, "k", "v", out, eps=1e-6), width)
        assert float((got.to(F64) - want).abs().max()) < (1e-5 if f32 else 4e-3), portions


@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("at", [0, 31, 32, 63, 64, 127, 200])
def test_a_single_key_far_back_takes_the_softmax(at, f32):
    """One key answers every later query, hundreds of positions on, wherever it lies in the kernels' 32- and 64-key tiles; its value
    alone comes out, prompt or decoding, also right at the position itself and never before it."""
    H, G, d, dv, width, T = 4, 2, 32, 16, 16, 420
    m = cases.left(H, G, d, dv, 1, 2.0, (0.1, 64))
    cfg = cases.config(8, width, [cases.layer(cases.pair(m, cases.right(1, 1, 4, 4, 1), 1.0, 1.0))])
    c = layer_config(cfg).mixer.left
    torch.manual_seed(at)
    W = {"q": torch.zeros(H * d, width), "k": torch.zeros(G * d, width), "v": bf(torch.randn(G * dv, width) * 0.3), "o": bf(torch.randn(width, H * dv) * 0.3),
         "g": torch.zeros(H * dv, width), "q.norm": torch.ones(d), "k.norm": torch.ones(d), "q.conv": torch.ones(H * d, 1), "k.conv": torch.ones(G * d, 1),
         "v.conv": torch.ones(G * dv, 1)}
    W["q"][0::d, 2], W["k"][0::d, 0], W["k"][1::d, 1] = 1.0, 1.0, 1.0
    h = bf(torch.randn(T, width) * 0.5)
    h[:, 2], h[:, 0], h[:, 1] = 1.0, 0.0, 1.0
    h[at, 0], h[at, 1] = 1.0, 0.0
    want = mo.convolved_attention(h.to(F64), wide(W), "", m, 1e-6)
    marker = 0.5 * (h[at].to(F64) @ W["v"].to(F64).T).reshape(G, 1, dv).expand(G, H // G, dv).reshape(-1) @ W["o"].to(F64).T
    takes = row_errors(want, marker.expand(T, width)) < 1e-2
    assert [i for i in range(T) if takes[i]] == list(range(at, T))
    for portions in ([T], [at + 1], [max(at, 1), 2, 180], [390]):
        bench = Bench(conv_specs(G, d, dv, (H + G) * d + G * dv, 1, f32), f32, max_pos=T)
        w = packer(W, f32).convolved_attention("")
        got = bench.portions(h, portions, lambda b, rows, out: b.softmax_attention(rows, c, w, "k", "v", out, eps=1e-6), width)
        assert float(row_errors(got, want).max()) < (TOL[True] if f32 else TOL[False]), portions


DELTA_CASES = {
    # name: (H, G, d, dv, taps, decay rank, gate rank, width, T, portions)
    "three_heads_a_key_head": (6, 2, 6, 9, 3, 5, 7, 24, 70, [1, 2, 40, 17]),
    "one_head_wide_values_one_tap": (1, 1, 9, 37, 1, 3, 2, 20, 45, [45]),
    "key_size_not_a_multiple_of_four": (3, 3, 10, 16, 5, 8, 16, 16, 33, [2, 2, 2]),
    "rank_one": (2, 1, 12, 8, 2, 1, 1, 16, 40, [30]),
    "wide_keys_many_value_tiles": (2, 2, 136, 40, 4, 24, 24, 64, 90, [64, 2, 20]),
    "keys_of_264_rows": (1, 1, 264, 8, 4, 16, 8, 32, 40, [17, 2]),
    "around_one_round_of_tokens": (2, 2, 12, 20, 4, 8, 8, 24, 70, [16, 17, 15, 18]),
    "long_prompt": (4, 2, 32, 64, 4, 16, 32, 64, 400, [330, 2, 50]),
    "portions_of_whole_and_broken_blocks": (2, 2, 64, 48, 4, 16, 16, 48, 420, [64, 65, 63, 96, 128]),
    "key_size_128": (3, 1, 128, 128, 4, 32, 64, 96, 300, [257, 2]),
    "long_prompt_odd_sizes": (3, 3, 20, 24, 4, 8, 8, 32, 700, [130, 560]),
    "key_size_96": (2, 1, 96, 36, 3, 16, 16, 40, 200, [190]),
}


def delta_bench(H, G, d, dv, taps, T, f32):
    from qwen3_tts_cuda_graphs_b200.seq_state import StateSpec

    return Bench([StateSpec("s.conv", "carry", 2 * G * d + H * dv, taps - 1), StateSpec("s.s", "carry", dv, H * d, in_place=True)], f32, max_pos=T + 3)


def delta_setup(H, G, d, dv, taps, ra, rg, width, seed, eps):
    m = cases.right(H, G, d, dv, taps)
    cfg = cases.config(8, width, [cases.layer(cases.pair(cases.left(1, 1, 4, 4, 1, 1.0), m, 1.0, 1.0))], eps=eps)
    return m, layer_config(cfg).mixer.right, sub_weights(cfg, "l0.mix.right.", seed=seed, decay_rank=ra, gate_rank=rg)


@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("case", list(DELTA_CASES))
def test_channel_delta_rule_alone(case, f32):
    H, G, d, dv, taps, ra, rg, width, T, portions = DELTA_CASES[case]
    eps = 1e-4
    m, c, W = delta_setup(H, G, d, dv, taps, ra, rg, width, len(case), eps)
    torch.manual_seed(3)
    h = bf(torch.randn(T, width))
    want = mo.channel_delta_rule(h.to(F64), wide(W), "", m, eps)
    w = packer(W, f32).channel_delta("")
    for sizes in (portions, [T]):
        bench = delta_bench(H, G, d, dv, taps, T, f32)
        got = bench.portions(h, sizes, lambda b, rows, out: b.channel_delta_rule(rows, c, w, "s", eps, out), width)
        assert close_enough(got, want, f32), (sizes, float(row_errors(got, want).max()))
    if f32:
        # the premises: without dt_bias, with one decay per head, or with every head's rate equal it is a different function
        same = W["dt_bias"].reshape(H, d)[:, :1].expand(H, d).reshape(-1)
        for name, t in (("dt_bias", torch.zeros_like(W["dt_bias"])), ("dt_bias", same), ("A_log", W["A_log"] + 0.3)):
            other = mo.channel_delta_rule(h.to(F64), {**wide(W), name: t.to(F64)}, "", m, eps)
            assert float(row_errors(other, want).median()) > 10 * TOL[True], name


@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("corner", ["keeps_everything", "forgets_at_once", "some_channels_each", "strong_writes", "no_writes"])
def test_channel_decays_and_write_strengths_at_their_ends(corner, f32):
    """Decays within 1e-6 of one, decays that vanish (products over a run of tokens underflow), both side by side in one head; write
    strengths near one on nearly equal keys (corrections that cancel) and near zero."""
    H, G, d, dv, taps, width, T, eps = 2, 1, 32, 24, 2, 24, 300, 1e-4
    m, c, W = delta_setup(H, G, d, dv, taps, 6, 6, width, 77, eps)
    if corner == "keeps_everything":
        W["dt_bias"] -= 12.0
    elif corner == "forgets_at_once":
        W["dt_bias"] += 9.0
        W["A_log"] += 2.0
    elif corner == "some_channels_each":
        W["dt_bias"][0::3] = 20.0
        W["dt_bias"][1::3] = -14.0
        W["A_log"] += 1.5
    torch.manual_seed(4)
    h = bf(torch.randn(T, width))
    if corner == "strong_writes":      # inputs that repeat with small changes: keys nearly parallel, strengths near one
        h = bf(h[:1] + 0.1 * h)
        W["b"] = bf(h[:1] / (h[0] @ h[0]) * 6.0).expand(H, width).clone()
    elif corner == "no_writes":
        W["b"] = bf(-h.mean(0, keepdim=True)).expand(H, width).clone()
        h = bf(h + 4.0)
        W["b"] = torch.full((H, width), -0.06)
    W = {k: bf(v) for k, v in W.items()}
    want = mo.channel_delta_rule(h.to(F64), wide(W), "", m, eps)
    assert torch.isfinite(want).all()
    w = packer(W, f32).channel_delta("")
    for sizes in ([T], [37, 2, 200], [2, 2, 64]):
        bench = delta_bench(H, G, d, dv, taps, T, f32)
        got = bench.portions(h, sizes, lambda b, rows, out: b.channel_delta_rule(rows, c, w, "s", eps, out), width)
        assert torch.isfinite(got).all() and close_enough(got, want, f32), (sizes, float(row_errors(got, want).max()))


@pytest.mark.parametrize("f32", [True, False])
def test_a_token_written_long_ago_is_read_back(f32):
    """A channel that keeps everything holds one token's value for hundreds of tokens that write along other keys; a lost or misplaced
    state, or a decay on the wrong channel, loses it."""
    H, d, dv, width, T, at = 1, 8, 8, 16, 500, 70
    m = cases.right(H, 1, d, dv, 1)
    cfg = cases.config(8, width, [cases.layer(cases.pair(cases.left(1, 1, 4, 4, 1, 1.0), m, 1.0, 1.0))])
    c = layer_config(cfg).mixer.right
    z = torch.zeros
    W = {"q": z(d, width), "k": z(d, width), "v": z(dv, width), "b": z(H, width), "A_log": z(H), "dt_bias": torch.full((H * d,), 1.0), "norm": torch.ones(dv),
         "a1": z(1, width), "a2": z(H * d, 1), "g1": z(1, width), "g2": z(H * dv, 1), "o": bf(torch.randn(width, dv, generator=torch.Generator().manual_seed(1)))}
    for n, size in (("q", d), ("k", d), ("v", dv)):
        W[n + ".conv"] = torch.ones(size, 1)
    W["dt_bias"][3] = -24.0                                  # key channel 3 keeps everything
    W["q"][3, 0] = 4.0                                       # every query asks along channel 3
    W["k"][3, 1], W["k"][5, 2] = 4.0, 4.0                    # one token writes along channel 3, the others along 5 (decaying)
    W["b"][0, 0] = 5.0
    W["v"][:, 8:] = torch.eye(dv)
    torch.manual_seed(9)
    h = z(T, width)
    h[:, 0], h[:, 2] = 1.0, 1.0
    h[at, 1], h[at, 2] = 1.0, 0.0
    h[:, 8:] = bf(torch.randn(T, 8))
    want = mo.channel_delta_rule(h.to(F64), wide(W), "", m, 1e-6)
    v = mo.silu(h[at, 8:].to(F64))
    marker = (mo.rms_unit(v, 1e-6) * 0.5) @ W["o"].to(F64).T
    assert float(row_errors(want[at:], marker.expand(T - at, width)).max()) < 1e-4
    w = packer(W, f32).channel_delta("")
    for sizes in ([T], [at, 2, 300], [at + 1, 64, 64], [2] * 60):
        bench = delta_bench(H, 1, d, dv, 1, T, f32)
        got = bench.portions(h, sizes, lambda b, rows, out: b.channel_delta_rule(rows, c, w, "s", 1e-6, out), width)
        assert float(row_errors(got[at:], marker.expand(T - at, width)).max()) < (TOL[True] if f32 else 2e-2), sizes


@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("taps", [(3, 5), (4, 2), (1, 1), (1, 4)])
def test_both_mixers_on_one_projection(taps, f32):
    """Convolutions of different lengths share one launch and one carried history; the scales act on their own side."""
    from qwen3_tts_cuda_graphs_b200.seq_state import StateSpec

    width, T, eps = 28, 120, 1e-3
    a, r = cases.left(4, 2, 10, 7, taps[0], 0.4, (0.5, 9)), cases.right(6, 3, 6, 8, taps[1])
    cfg = cases.config(8, width, [cases.layer(cases.pair(a, r, 0.6, 1.7))], eps=eps)
    W = sub_weights(cfg, "l0.mix.", seed=sum(taps))
    mix = layer_config(cfg).mixer
    torch.manual_seed(2)
    h = bf(torch.randn(T, width))
    lo, ro = mo.convolved_attention(h.to(F64), wide(W), "left.", a, eps), mo.channel_delta_rule(h.to(F64), wide(W), "right.", r, eps)
    want = 0.6 * lo + 1.7 * ro
    w = packer(W, f32).pair("", mix.right_scale)
    channels = w["conv"].shape[0]
    for sizes in ([T], [2, 3, 1, 70], [97, 2]):
        bench = Bench(kv_specs(2, 10, 7, f32) + [StateSpec("s.conv", "carry", channels, max(taps) - 1), StateSpec("s.s", "carry", 8, 36, in_place=True)],
                      f32, max_pos=T + 3)
        got = bench.portions(h, sizes, lambda b, rows, out: b.attention_beside_delta_rule(rows, mix.left, mix.right, w, "k", "v", "s", eps, out,
                                                                                          left_scale=mix.left_scale), width)
        assert close_enough(got, want, f32), (sizes, float(row_errors(got, want).max()))


def test_two_parts_of_a_list_side_by_side():
    """A side stream sees what was launched before it, the main stream sees its results behind the join; a list may end with the side
    stream open; the same list captured as a graph gives the same."""
    from qwen3_tts_cuda_graphs_b200.seq_ops import StepBuilder

    torch.manual_seed(1)
    M, N = 700, 256
    bench = Bench([], True)
    x, one = cuda(torch.randn(1, M, N)), cuda(torch.ones(2))
    for ending in (True, False):
        b = StepBuilder(torch.device(DEV), M, bench.slot, True)
        a, parts, out = torch.zeros(M, N, device=DEV), torch.zeros(2, M, N, device=DEV), torch.zeros(M, N, device=DEV)
        b.sum_norm(x, 1, cuda(torch.tensor([2.0])), out=a)                     # before both: a = 2 x
        b.branch(0)
        for _ in range(6):
            b.sum_norm(a[None], 1, cuda(torch.tensor([3.0])), out=parts[0])     # side: 6 x
        b.branch(1)
        b.sum_norm(a[None], 1, cuda(torch.tensor([5.0])), out=parts[1])         # main: 10 x
        if ending:
            b.branch(2)
            b.sum_norm(parts, 2, one, out=out)
        plan = b.finish()
        for _ in range(4):          # launched, then captured and replayed
            parts.zero_()
            out.zero_()
            bench.codec.run_op_plan(bench.lib, plan, True)
            total = out if ending else parts[0] + parts[1]
            assert torch.allclose(total, 16.0 * x[0], rtol=1e-5)
        assert getattr(plan, "graph", None) is not None
        bench.lib.fq3c_graph_destroy(plan.graph)
    b = StepBuilder(torch.device(DEV), M, bench.slot, True)       # a second side stream inside the first is refused
    b.branch(0)
    b.branch(0)
    with pytest.raises(Exception, match="one side stream"):
        bench.codec.run_op_plan(bench.lib, b.finish(), False)


# ---------------------------------------------------------------------------------------------------------------------------
# whole models
# ---------------------------------------------------------------------------------------------------------------------------
CASES = {"odd": cases.odd, "unaligned": cases.unaligned, "aligned": cases.aligned}


@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("case", list(CASES))
def test_prompt_portions_and_decoding_agree_with_the_oracle(case, f32):
    cfg = CASES[case]()
    W = cases.weights(cfg, seed=7)
    T = 150 if case == "aligned" else 90
    toks = cases.tokens(cfg, T)
    taps = []
    want = mo.forward(cfg, W, toks, taps)
    eng = make_engine(cfg, W, f32)
    whole = run_schedule(eng, toks, [T])
    assert close_enough(whole, want, f32), float(row_errors(whole, want).max())
    # the slot of the request above is used again by each of these
    for portions in ([2, 3, 1, 5, 2, 37, 2, 33], [60], [1] * 20, [T - 1]):
        got = run_schedule(eng, toks, portions)
        assert close_enough(got, want, f32), portions
        assert close_enough(got, whole.cpu(), f32), portions
    if f32:   # the residual stream after every layer
        eng.step("taps", toks, [], layer_taps=True)
        assert len(eng.last_taps) == len(taps)
        for i, (a, b) in enumerate(zip(eng.last_taps, taps)):
            assert float(row_errors(a, b).max()) < TOL[True], i
        eng.close("taps")
        # the premises: the stream's factor, the norms' biases and the mixers' scales all count
        for other in (dict(cfg, postln_alpha=cfg["postln_alpha"] * 1.1), dict(cfg, norm={"eps": cfg["norm"]["eps"] * 3 + 1e-2})):
            assert float(row_errors(mo.forward(other, W, toks[:40]), want[:40]).median()) > 10 * TOL[True]
        bare = {k: torch.zeros_like(v) if k.endswith(("norm1.b", "norm2.b")) else v for k, v in W.items()}
        assert float(row_errors(mo.forward(cfg, bare, toks[:40]), want[:40]).median()) > 10 * TOL[True]
    eng.close_all()


@pytest.mark.parametrize("f32", [True, False])
def test_peaked_attention_over_hundreds_of_positions(f32):
    """Large scales put each row's mass on single keys; positions on both sides of the kernels' 32- and 64-key tiles and of their
    key-range splits come both inside a prompt portion and decoded alone."""
    s = 1.2 if f32 else 0.5          # bf16 products: milder peaks, fewer near-ties
    cfg = cases.config(64, 64, [
        cases.layer(cases.attn(4, 2, 16, s, 8, 2000.0, (2.0, 100, 8.0, 1.0)), cases.dense(96)),
        cases.layer(cases.pair(cases.left(4, 1, 16, 32, 3, s * 0.8, (0.2, 100)), cases.right(2, 2, 16, 16, 3), 1.0, 0.7)),
        cases.layer(cases.attn(2, 1, 16, s, 16, 500.0)),
    ])
    W = cases.weights(cfg, seed=9)
    T = 330
    toks = cases.tokens(cfg, T)
    want = mo.forward(cfg, W, toks)
    eng = make_engine(cfg, W, f32, max_tokens=T)
    for portions in ([T], [31, 33, 2, 36, 154, 2, 22]):       # portions end at 31, 64, 66, 102, 256, 258, 280; the rest decoded
        got = run_schedule(eng, toks, portions)
        assert close_enough(got, want, f32), float(row_errors(got, want).max())
    eng.close_all()


def test_requests_take_turns_in_two_slots_and_slots_are_reused():
    cfg = cases.odd()
    W = cases.weights(cfg, seed=10)
    eng = make_engine(cfg, W, True, max_slots=2)
    reqs = {n: cases.tokens(cfg, L, seed=i) for i, (n, L) in enumerate([("a", 23), ("b", 9), ("c", 41), ("d", 2)])}
    want = {n: mo.forward(cfg, W, t) for n, t in reqs.items()}
    got = {n: [] for n in reqs}
    at = {n: 0 for n in reqs}
    # a and b interleaved with unequal portions; when b ends, c takes its slot (caches, convolution inputs and states of b in it)
    # while a is still running; then d
    plan = [("a", 5), ("b", 2), ("a", 1), ("b", 7), ("c", 30), ("a", 10), ("c", 1), ("a", 7), ("d", 2), ("c", 10)]
    for n, k in plan:
        part = reqs[n][at[n]:at[n] + k]
        got[n].append(eng.step(n, part, list(range(k))).clone())
        at[n] += k
        if at[n] == len(reqs[n]):
            eng.close(n)
    assert len(eng.states.slots) == 2
    for n in reqs:
        assert float(row_errors(torch.cat(got[n]), want[n]).max()) < TOL[True], n
    eng.close_all()


def test_long_decoding():
    cfg = cases.odd()
    W = cases.weights(cfg, seed=11)
    toks = cases.tokens(cfg, 240)
    want = mo.forward(cfg, W, toks)
    for f32 in (True, False):
        eng = make_engine(cfg, W, f32)
        got = run_schedule(eng, toks, [3])          # 237 tokens one by one through the caches and states
        assert close_enough(got, want, f32)
        eng.close_all()


def test_first_tokens_of_a_sequence():
    """One-token and two-token sequences, and the first positions of a longer one: shorter than every convolution, states at zero."""
    for make in (cases.unaligned, cases.odd):
        cfg = make()
        W = cases.weights(cfg, seed=13)
        eng = make_engine(cfg, W, True, max_tokens=6)
        for n in (1, 2, 5):
            toks = cases.tokens(cfg, n, seed=n)
            assert float(row_errors(run_schedule(eng, toks, [n]), mo.forward(cfg, W, toks)).max()) < TOL[True]
            assert float(row_errors(run_schedule(eng, toks, []), mo.forward(cfg, W, toks)).max()) < TOL[True]
        eng.close_all()


def test_no_layers_and_no_feed_forward():
    """A model without layers is the embedding, the output norm and the head."""
    for layers in ([], [cases.layer(cases.attn(1, 1, 6, 0.5, 2, 30.0))]):
        cfg = cases.config(23, 12, layers)
        W = cases.weights(cfg, seed=15)
        eng = make_engine(cfg, W, True)
        few = cases.tokens(cfg, 9)
        assert float(row_errors(run_schedule(eng, few, [4]), mo.forward(cfg, W, few)).max()) < TOL[True]
        eng.close_all()


def test_capacity_and_bad_input_are_refused():
    cfg = cases.unaligned()
    eng = make_engine(cfg, cases.weights(cfg), True, max_tokens=10, max_slots=1)
    eng.step("a", [1, 2, 3, 4, 5, 6], [])
    with pytest.raises(RuntimeError):
        eng.step("a", [1, 2, 3, 4, 5], [])
    with pytest.raises(RuntimeError):
        eng.open("b")                                # the only slot is taken
    with pytest.raises(ValueError):
        eng.step("a", [cfg["vocab"]], [])
    eng.close("a")
    eng.step("b", [1, 2], [1])
    eng.close_all()


def _oracle_greedy(cfg, W, prompt, n):
    """Greedy continuation by the oracle, with the margin between the two best logits of every choice."""
    toks, margins = list(prompt), []
    for _ in range(n):
        lg = mo.forward(cfg, W, toks)[-1]
        top = torch.topk(lg, 2).values
        margins.append(float(top[0] - top[1]))
        toks.append(int(lg.argmax()))
    return toks[len(prompt):], margins


def _greedy_cases():
    cfg = cases.odd()
    W = cases.weights(cfg, seed=13)
    return cfg, W, [cases.tokens(cfg, L, seed=20 + i) for i, L in enumerate((12, 3, 27))]


def test_greedy_generation_through_engine_and_scheduler():
    from qwen3_tts_cuda_graphs_b200.serving import TokenRequest, TokenScheduler

    cfg, W, prompts = _greedy_cases()
    n_new = 10
    eng = make_engine(cfg, W, True, max_tokens=64, max_slots=2)
    want = []
    for p in prompts:
        ids, margins = _oracle_greedy(cfg, W, p, n_new)
        cut = next((i for i, m in enumerate(margins) if m < 1e-3), n_new)     # compare up to the first near-tie
        want.append(ids[:cut])
        assert cut >= 3
    for p, w in zip(prompts, want):
        assert eng.generate(p, n_new, prefill_chunk=5)[:len(w)] == w
    sched = TokenScheduler(eng, prefill_chunk=4)       # three requests, two slots: the third waits for a slot
    handles = [sched.submit(TokenRequest(p, n_new)) for p in prompts]
    sched.run()
    for h, w in zip(handles, want):
        assert h.done and h.reason == "length" and h.result()[:len(w)] == w
    eng.close_all()


def test_command_line_continues_prompts_greedily_and_by_sampling(tmp_path, capsys):
    """`cli lm` on a checkpoint on disk: greedy ids equal the oracle's argmax chain; the framework's sampler with top-k 1 is greedy,
    and with a seed it repeats itself."""
    import json

    from qwen3_tts_cuda_graphs_b200 import cli

    cfg, W, prompts = _greedy_cases()
    cases.save_checkpoint(str(tmp_path), cfg, W)
    n_new = 8
    base = ["--dtype", "fp32", "lm", "--model", str(tmp_path), "--max-new-tokens", str(n_new), "--concurrency", "2", "--prefill-chunk", "5"]
    for p in prompts:
        base += ["--tokens", " ".join(str(t) for t in p)]

    def run(extra):
        capsys.readouterr()
        cli.main(base + extra)
        lines = [json.loads(ln) for ln in capsys.readouterr().out.splitlines() if ln.startswith("{")]
        assert len(lines) == len(prompts) and all(d["finish"] == "length" and len(d["tokens"]) == n_new for d in lines)
        return [d["tokens"] for d in lines]

    greedy = run(["--greedy"])
    for p, got in zip(prompts, greedy):
        ids, margins = _oracle_greedy(cfg, W, p, n_new)
        cut = next((i for i, m in enumerate(margins) if m < 1e-3), n_new)
        assert cut >= 3 and got[:cut] == ids[:cut]
    assert run(["--top-k", "1", "--seed", "5"]) == greedy
    hot = run(["--temperature", "1.5", "--seed", "7"])
    assert hot == run(["--temperature", "1.5", "--seed", "7"]) and all(0 <= t < cfg["vocab"] for row in hot for t in row)
    assert hot != greedy


def test_replayer_reads_a_checkpoint_from_disk_and_writes_the_wanted_logits(tmp_path):
    """bin/trace_run as a child process: the model class comes from config.json; a finished request's slot goes to the next."""
    import json
    import os
    import subprocess
    import sys

    import numpy as np

    cfg = cases.odd()
    W = cases.weights(cfg, seed=21)
    model_dir, out_dir = tmp_path / "model", tmp_path / "out"
    model_dir.mkdir()
    cases.save_checkpoint(str(model_dir), cfg, W)
    a, b = cases.tokens(cfg, 24, seed=5), cases.tokens(cfg, 6, seed=6)
    steps = [
        {"step": 0, "entries": [{"id": "a", "tokens": a[:19], "want": [0, 3, 18]}], "end": []},
        {"step": 1, "entries": [{"id": "a", "tokens": a[19:21], "want": []}], "end": []},
        {"step": 2, "entries": [{"id": "a", "tokens": a[21:22], "want": [0]}], "end": []},
        {"step": 3, "entries": [{"id": "a", "tokens": a[22:24], "want": [1, 0]}], "end": ["a"]},
        {"step": 4, "entries": [{"id": "b", "tokens": b, "want": [5]}], "end": ["b"]},
    ]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    for dtype, tol in (("float32", TOL[True]), ("bfloat16", TOL[False])):
        p = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", str(model_dir), "--dtype", dtype,
                            "--out", str(out_dir / dtype), "--max-tokens", "32", "--max-slots", "1"],
                           input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600)
        assert p.returncode == 0, p.stderr[-2000:]
        assert [ln for ln in p.stdout.splitlines() if ln.startswith("done ")] == [f"done {i}" for i in range(5)]
        assert not (out_dir / dtype / "1.f32").exists()
        ref_a, ref_b = mo.forward(cfg, W, a), mo.forward(cfg, W, b)
        for step, ref, places in ((0, ref_a, [0, 3, 18]), (2, ref_a, [21]), (3, ref_a, [23, 22]), (4, ref_b, [5])):
            got = torch.from_numpy(np.fromfile(out_dir / dtype / f"{step}.f32", dtype="<f4").reshape(len(places), cfg["vocab"]))
            assert float(row_errors(got, ref[places]).max()) < tol, (dtype, step)
