"""The Sirodra sequence model on the CUDA op-list path against the float64 oracle (oracle/sirodra_oracle.py).

Mechanisms alone (seq_ops.StepBuilder fragments), then whole models: prompts, prompts in portions down to two tokens, token by
token decoding through the caches, pooled rows and carried states, slots that are given back and used again, requests that take
turns, keys far back inside pooled blocks, tokens just inside and just outside a window, blocks that are just seen or not yet, long
decoding, loops of one, two and three passes, sizes that are multiples of nothing, and greedy generation through the engine's entry
point, the scheduler and the command line.
"""
import pytest
import torch

import sirodra_cases as cases
from oracle import sirodra_oracle as so

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
    models (a peaked softmax's near-tie, a read-out whose divisor is nearly zero), so nine rows in ten must be within the tolerance
    and the typical one well within it; a wrong key, a window edge or a lost state moves far more."""
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
    from qwen3_tts_cuda_graphs_b200.sirodra import Packer

    return Packer(lambda n: W[n].to(torch.float32), DEV, f32)


def sub_weights(cfg, prefix, seed):
    return {k[len(prefix):]: v for k, v in cases.weights(cfg, seed=seed).items() if k.startswith(prefix)}


def layer_config(cfg, i=0):
    from qwen3_tts_cuda_graphs_b200.config import sequence_config_from_dict

    return sequence_config_from_dict(cfg).layers[i]


# ---------------------------------------------------------------------------------------------------------------------------
# mechanisms alone
# ---------------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("groups,size", [(1, 36), (3, 7), (4, 130)])
def test_group_norm_with_divisors_and_a_sigmoid_gate(groups, size):
    torch.manual_seed(size)
    M, N, eps = 5, groups * size, 1e-2
    x, gate, w = torch.randn(M, N) * 3, torch.randn(M, N + 6), 1.0 + 0.2 * torch.randn(N)
    den = torch.rand(M, groups) * 20 + 0.05
    unit = so.rms_unit(x.to(F64).reshape(M, groups, size) / den.to(F64)[..., None], eps).reshape(M, N)
    want = unit * w.to(F64) * so.sigmoid(gate.to(F64)[:, 6:])
    out, low = torch.zeros(M, N, device=DEV), torch.zeros(M, N, device=DEV, dtype=torch.bfloat16)
    for dst in (out, low):
        Bench([]).run(M, lambda b: b.group_norm(cuda(x), cuda(w), groups, eps, dst, gate=cuda(gate), gate_col=6, gate_sigmoid=True, divisor=cuda(den)))
    assert torch.allclose(out.cpu().to(F64), want, atol=2e-5)
    assert torch.allclose(low.float().cpu().to(F64), want, atol=3e-2, rtol=1e-2)
    # the premise: with this eps the divisor changes the result
    plain = so.rms_unit(x.to(F64).reshape(M, groups, size), eps).reshape(M, N) * w.to(F64) * so.sigmoid(gate.to(F64)[:, 6:])
    assert float((plain - want).abs().max()) > 0.02
    # a sigmoid gate in front of the statistics
    Bench([]).run(M, lambda b: b.group_norm(cuda(x), cuda(w), groups, eps, out, gate=cuda(gate), gate_col=6, gate_sigmoid=True, gate_first=True))
    pre = so.rms_unit((x.to(F64) * so.sigmoid(gate.to(F64)[:, 6:])).reshape(M, groups, size), eps).reshape(M, N) * w.to(F64)
    assert torch.allclose(out.cpu().to(F64), pre, atol=2e-5)


@pytest.mark.parametrize("f32", [True, False])
def test_the_stream_and_the_embedding_as_product_operands(f32):
    torch.manual_seed(4)
    M, N, V = 7, 52, 11
    dt = torch.float32 if f32 else torch.bfloat16
    parts, table = cuda(torch.randn(2, M, N)), cuda(torch.randn(V, N), dt)
    ids = torch.tensor([3, 0, 10, 3, 7, 1, 2])
    cat, x = torch.zeros(M, 2 * N, device=DEV, dtype=dt), torch.zeros(M, N, device=DEV)
    before = parts.cpu().clone()
    bench = Bench([], f32)
    bench.run(M, lambda b: b.embed(ids.to(DEV, torch.int32), table, x, operand=cat))
    assert torch.equal(cat[:, :N], table[ids]) and torch.equal(cat[:, N:], table[ids]) and torch.equal(x, table[ids].float())
    cat.zero_()
    bench.run(M, lambda b: b.embed(ids.to(DEV, torch.int32), table, x, operand=cat, operand_col=N))
    assert not cat[:, :N].any() and torch.equal(cat[:, N:], table[ids])
    bench.run(M, lambda b: b.sum_norm(parts, 2, cuda(torch.ones(2)), norm_out=cat))
    assert torch.equal(parts[0].cpu(), before[0] + before[1])
    assert torch.equal(cat[:, :N], parts[0].to(dt)) and torch.equal(cat[:, N:], table[ids])
    w = torch.randn(N, 2 * N) * 0.1
    out = torch.zeros(M, N, device=DEV)
    bench.run(M, lambda b: b.linear(cat, cuda(w, dt), out))
    want = cat.cpu().to(F64) @ w.to(dt).to(F64).T
    assert float(row_errors(out, want).max()) < 1e-5


@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("M,width,ff", [(1, 36, 20), (3, 64, 128), (200, 128, 192), (50, 20, 7)])
def test_dense_gelu_feed_forward(M, width, ff, f32):
    torch.manual_seed(M)
    x = bf(torch.randn(M, width) * 1.5)
    W = {"up": bf(torch.randn(ff, width) * 2 * width ** -0.5), "down": bf(torch.randn(width, ff) * ff ** -0.5)}
    want = so.dense_ff(x.to(F64), {k: v.to(F64) for k, v in W.items()}, "")
    dt = torch.float32 if f32 else torch.bfloat16
    out = torch.zeros(M, width, device=DEV)
    Bench([], f32).run(M, lambda b: b.gelu_ff(cuda(x, dt), {k: cuda(v, dt) for k, v in W.items()}, out))
    e = row_errors(out, want)
    assert float(e.max()) < (1e-5 if f32 else 2e-2)


GATE_CASES = {
    # name: (H, d, dv, width, T, portions)
    "five_heads_key_size_six": (5, 6, 3, 24, 70, [1, 2, 40, 17]),
    "one_head_wide_values": (1, 9, 37, 20, 45, [45]),
    "key_size_not_a_multiple_of_four": (3, 10, 16, 16, 33, [2, 2, 2]),
    "two_rounds_of_state_rows": (2, 44, 24, 32, 120, [100, 3]),
    "wide_keys_many_value_tiles": (2, 136, 40, 64, 90, [64, 2, 20]),
    "keys_of_264_rows": (1, 264, 8, 32, 40, [17, 2]),
    "around_one_round_of_tokens": (2, 12, 20, 24, 70, [16, 17, 15, 18]),
    "long_prompt": (4, 32, 64, 64, 400, [330, 2, 50]),
    # portions of 512 rows and more are walked in pieces (side by side, from start states a carry pass provides)
    "nine_pieces_ragged_tail_after_a_short_portion": (2, 20, 24, 32, 1300, [40, 1200, 2]),
    "four_pieces_then_four_again": (3, 36, 8, 24, 1160, [600, 2, 550]),
    "sixteen_pieces": (1, 12, 20, 16, 2200, [2150]),
}


@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("case", list(GATE_CASES))
def test_forget_gate_linear_attention_alone(case, f32):
    from qwen3_tts_cuda_graphs_b200.seq_state import StateSpec

    H, d, dv, width, T, portions = GATE_CASES[case]
    eps = 1e-3
    cfg = cases.config(8, width, [cases.layer(cases.hgrn(H, d, dv))], eps=eps)
    W = sub_weights(cfg, "l0.mix.", seed=len(case))
    W["lower"][::3] = bf(torch.tensor(0.99))                  # some channels that keep long, some that do not have a bound at all
    W["lower"][1::3] = 0.0
    m, c = cfg["layers"][0]["mixer"], layer_config(cfg).mixer
    torch.manual_seed(3)
    h = bf(torch.randn(T, width))
    W64 = {k: v.to(F64) for k, v in W.items()}
    want = so.hgrn2(h.to(F64), W64, "", m, eps)
    bench = Bench([StateSpec("s", "carry", dv, H * d)], f32, max_pos=T + 3)
    w = packer(W, f32).forget_gate("")
    got = bench.portions(h, portions, lambda b, rows, out: b.forget_gate_attention(rows, c, w, "s", eps, out), width)
    assert close_enough(got, want, f32), float(row_errors(got, want).max())
    if f32:
        # the premises: without the lower bound, or without the gate's bias, it is a different function
        for name in ("lower", "f.b"):
            other = so.hgrn2(h.to(F64), {**W64, name: torch.zeros_like(W64[name])}, "", m, eps)
            assert float(row_errors(other, want).median()) > 10 * TOL[True], name


def test_forget_gates_at_their_ends():
    """Gates that are (nearly) one keep the state and write next to nothing; the written part 1 - f must keep its relative precision:
    a gate of 1 - 2^-20 rounded in 32-bit and subtracted from one would be off by several per cent, and the unit read-out shows it."""
    from qwen3_tts_cuda_graphs_b200.seq_state import StateSpec

    H, d, dv, width, T, eps = 1, 4, 6, 8, 30, 0.0
    cfg = cases.config(8, width, [cases.layer(cases.hgrn(H, d, dv))])
    W = sub_weights(cfg, "l0.mix.", seed=2)
    W["f"] *= 0.25
    W["f.b"] = torch.tensor([14.0, 15.0, 16.5, 17.5])
    W["lower"] = torch.tensor([0.0, 0.5, 0.0, 0.25])
    torch.manual_seed(8)
    h = bf(torch.randn(T, width))
    W64 = {k: v.to(F64) for k, v in W.items()}
    want = so.hgrn2(h.to(F64), W64, "", cfg["layers"][0]["mixer"], eps)
    for portions in ([T], [2, 20], []):
        bench = Bench([StateSpec("s", "carry", dv, H * d)], True)
        w = packer(W, True).forget_gate("")
        c = layer_config(cfg).mixer
        got = bench.portions(h, portions, lambda b, rows, out: b.forget_gate_attention(rows, c, w, "s", eps, out), width)
        assert float(row_errors(got, want).max()) < 2e-5, portions


MEMORY_CASES = {
    # name: (H, d, dv, cap, width, T, portions)
    "three_heads_small_cap": (3, 6, 5, 1.5, 24, 70, [1, 2, 40, 17]),
    "one_head_one_value": (1, 9, 1, 4.0, 20, 45, [45]),
    "fifteen_values_share_a_tile_with_the_normaliser": (2, 10, 15, 8.0, 16, 33, [2, 2, 2]),
    "sixteen_values_put_it_into_a_tile_of_its_own": (2, 12, 16, 8.0, 16, 33, [20, 2]),
    "two_rounds_of_state_rows": (2, 44, 24, 12.0, 32, 120, [100, 3]),
    "wide_keys_many_value_tiles": (2, 136, 40, 15.0, 64, 90, [64, 2, 20]),
    "keys_of_264_rows": (1, 264, 8, 6.0, 32, 40, [17, 2]),
    "around_one_round_of_tokens": (2, 12, 20, 5.0, 24, 70, [16, 17, 15, 18]),
    "long_prompt": (4, 32, 64, 30.0, 64, 400, [330, 2, 50]),
    "nine_pieces_ragged_tail_after_a_short_portion": (2, 20, 24, 10.0, 32, 1300, [40, 1200, 2]),
    "four_pieces_then_four_again": (3, 36, 8, 3.0, 24, 1160, [600, 2, 550]),
    "sixteen_pieces": (1, 12, 20, 20.0, 16, 2200, [2150]),
}


def _memory_specs(H, d, dv):
    from qwen3_tts_cuda_graphs_b200.seq_state import StateSpec

    return [StateSpec("s.s", "carry", dv + 1, H * d), StateSpec("s.m", "carry", H)]


@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("case", list(MEMORY_CASES))
def test_matrix_memory_alone(case, f32):
    H, d, dv, cap, width, T, portions = MEMORY_CASES[case]
    eps = 1e-3
    cfg = cases.config(8, width, [cases.layer(cases.mlstm(H, d, dv, cap))], eps=eps)
    W = sub_weights(cfg, "l0.mix.", seed=len(case))
    m, c = cfg["layers"][0]["mixer"], layer_config(cfg).mixer
    torch.manual_seed(3)
    h = bf(torch.randn(T, width))
    W64 = {k: v.to(F64) for k, v in W.items()}
    want = so.mlstm(h.to(F64), W64, "", m, eps)
    bench = Bench(_memory_specs(H, d, dv), f32, max_pos=T + 3)
    w = packer(W, f32).memory("")
    got = bench.portions(h, portions, lambda b, rows, out: b.matrix_memory(rows, c, w, "s", eps, out), width)
    assert close_enough(got, want, f32), float(row_errors(got, want).max())
    if f32:      # the premises: another cap, no biases, no output gate: a different function
        assert cap > 8.0 or float(row_errors(so.mlstm(h.to(F64), W64, "", dict(m, gate_cap=2.0 * cap), eps), want).median()) > 10 * TOL[True]
        for name in ("f.b", "g"):
            other = so.mlstm(h.to(F64), {**W64, name: torch.zeros_like(W64[name])}, "", m, eps)
            assert float(row_errors(other, want).median()) > 10 * TOL[True], name


@pytest.mark.parametrize("bias", [-9.0, 0.0, 9.0])
@pytest.mark.parametrize("forget", [-6.0, 0.5, 8.0])
def test_matrix_memory_gates_at_their_ends(bias, forget):
    """Input gates far down (the maximum comes from its start at zero and decays with the forget gates, and the read-out is divided by
    e^-m, not by the normaliser), far up, forget gates that keep everything or nothing; in one step, in portions and one by one."""
    H, d, dv, cap, width, T, eps = 2, 6, 5, 12.0, 16, 600, 0.3       # an eps that the read-out's size, and so its divisor, shows against
    cfg = cases.config(8, width, [cases.layer(cases.mlstm(H, d, dv, cap))])
    W = sub_weights(cfg, "l0.mix.", seed=5)
    W["i.b"], W["f.b"] = torch.tensor([bias, bias + 1.0]), torch.tensor([forget, forget - 0.5])
    c, m = layer_config(cfg).mixer, cfg["layers"][0]["mixer"]
    torch.manual_seed(9)
    h = bf(torch.randn(T, width))
    W64 = {k: v.to(F64) for k, v in W.items()}
    want = so.mlstm(h.to(F64), W64, "", m, eps)
    if bias != 0.0:      # the premise: the input gates' level shows
        assert float(row_errors(so.mlstm(h.to(F64), {**W64, "i.b": torch.zeros(H, dtype=F64)}, "", m, eps), want).max()) > 10 * TOL[True]
    for portions in ([T], [2, 530, 40], [T - 30]):
        bench = Bench(_memory_specs(H, d, dv), True)
        w = packer(W, True).memory("")
        got = bench.portions(h, portions, lambda b, rows, out: b.matrix_memory(rows, c, w, "s", eps, out), width)
        assert float(row_errors(got, want).max()) < TOL[True], (portions, float(row_errors(got, want).max()))


ATTENTION_CASES = {
    # name: (H, G, d, dv, window, pool, rot_dims, factor, width, T, portions, scale)
    "grouped_heads_pool_smaller_than_the_window": (6, 2, 10, 7, 9, 4, 6, 2.0, 24, 70, [1, 2, 40, 17], 1.2),
    "pool_wider_than_the_window": (4, 1, 6, 10, 5, 13, 6, 0.5, 20, 75, [45], 1.5),
    "window_of_one_blocks_of_one": (2, 2, 6, 5, 1, 1, 2, 3.0, 16, 33, [2, 2, 2], 1.0),
    "window_of_one_blocks_of_three": (2, 1, 6, 5, 1, 3, 0, 1.0, 16, 40, [10, 2], 1.0),
    "window_wider_than_the_sequence": (3, 3, 4, 6, 400, 8, 4, 2.0, 16, 40, [40], 1.0),
    "no_blocks_at_all": (3, 1, 8, 6, 11, 0, 4, 4.0, 16, 50, [40], 1.0),
    "no_mask_at_all": (4, 2, 16, 16, 0, 0, 8, 2.0, 32, 90, [70, 2], 1.0),
    "many_tiles_and_splits": (8, 2, 64, 32, 100, 2, 20, 2.0, 64, 430, [400, 2, 17], 0.6),
    "block_ends_inside_tiles_and_portions": (4, 4, 16, 16, 37, 5, 16, 1.0, 32, 300, [36, 2, 91, 150], 1.0),
    "three_heads_per_key_head_no_rotation": (6, 2, 32, 16, 64, 16, 0, 1.0, 48, 230, [150, 2, 63], 0.8),
    "more_blocks_than_a_tile_holds": (2, 2, 16, 128, 20, 1, 16, 2.0, 32, 280, [200, 2, 60], 1.0),
    "one_block_per_portion": (2, 1, 32, 64, 16, 32, 8, 2.0, 32, 200, [32, 31, 33, 32, 32], 0.8),
}


@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("case", list(ATTENTION_CASES))
def test_windowed_attention_with_pooled_blocks_alone(case, f32):
    from qwen3_tts_cuda_graphs_b200.seq_state import StateSpec

    H, G, d, dv, window, pool, rot_dims, factor, width, T, portions, scale = ATTENTION_CASES[case]
    eps = 1e-3
    cfg = cases.config(8, width, [cases.layer(cases.attn(H, G, d, dv, window, pool, scale, rot_dims, base=200.0, factor=factor))], eps=eps)
    W = sub_weights(cfg, "l0.mix.", seed=len(case))
    m, c = cfg["layers"][0]["mixer"], layer_config(cfg).mixer
    torch.manual_seed(5)
    h = bf(torch.randn(T, width))
    W64 = {k: v.to(F64) for k, v in W.items()}
    want = so.attention(h.to(F64), W64, "", m, eps)
    dt = torch.float32 if f32 else torch.bfloat16
    specs = [StateSpec("k", "append", G * d, dtype=dt), StateSpec("v", "append", G * dv, dtype=dt)]
    if pool:
        specs += [StateSpec("k.pool", "append", G * d, dtype=dt, every=pool), StateSpec("v.pool", "append", G * dv, dtype=dt, every=pool)]
    bench = Bench(specs, f32, max_pos=T + 3)
    w = packer(W, f32).attention("", c)
    got = bench.portions(h, portions, lambda b, rows, out: b.softmax_attention(rows, c, w, "k", "v", out, eps=eps), width)
    assert close_enough(got, want, f32), float(row_errors(got, want).max())
    if pool:      # the pooled rows are the means of the very rows the caches hold, every complete block once
        nb = T // pool
        for n in ("k", "v"):
            cache = bench.slot.cur[n][:nb * pool].float()
            mean = cache.reshape(nb, pool, -1).mean(1)
            assert torch.allclose(bench.slot.cur[n + ".pool"][:nb].float(), mean, atol=1e-5 if f32 else 1e-2, rtol=1e-2)
    if f32:
        def differs(other, by=10 * TOL[True]):
            return float(row_errors(other, want).max()) > by

        if 0 < window < T:      # a window one position wider or narrower, blocks one position longer or left out: different functions
            for size in (window + 1, max(window - 1, 1)):
                if size != window and not (pool == 1):      # blocks of one position: any window sees everything
                    assert differs(so.attention(h.to(F64), W64, "", dict(m, mask=dict(m["mask"], size=size)), eps))
            if pool:
                assert differs(so.attention(h.to(F64), W64, "", dict(m, mask=dict(m["mask"], pool=pool + 1)), eps))
                assert differs(so.attention(h.to(F64), W64, "", dict(m, mask={"size": window}), eps))
        if rot_dims:
            assert differs(so.attention(h.to(F64), W64, "", dict(m, rot=dict(m["rot"], scaling={"factor": 1.5 * factor})), eps))
        for name in ("q.b", "k.b", "v.b", "g"):
            assert differs(so.attention(h.to(F64), {**W64, name: torch.zeros_like(W64[name])}, "", m, eps)), name


@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("dims", [(6, 5), (32, 64)])
def test_a_block_is_seen_from_the_very_position_its_last_token_has_left_the_window(dims, f32):
    """Every key points one way except a run of P equal ones that answer the queries: first as tokens of the window, then for a while
    as nothing (the block's first tokens have left, its last has not), then as one pooled key, hundreds of positions on.  The run
    alone takes the softmax when it is seen, so the position at which it appears or disappears is plain in the output."""
    from qwen3_tts_cuda_graphs_b200.seq_state import StateSpec

    d, dv = dims
    H, G, width, T, window, P, blk = 2, 1, 16, 430, 23, 6, 20
    lo, hi = blk * P, blk * P + P - 1
    cfg = cases.config(8, width, [cases.layer(cases.attn(H, G, d, dv, window, P, 40.0 / d))])
    m, c = cfg["layers"][0]["mixer"], layer_config(cfg).mixer
    torch.manual_seed(11)
    W = {"q": torch.zeros(H * d, width), "k": torch.zeros(G * d, width), "v": bf(torch.randn(G * dv, width) * 0.3), "o": bf(torch.randn(width, H * dv) * 0.3),
         "g": torch.zeros(H, width), "q.b": torch.zeros(H * d), "k.b": torch.zeros(G * d), "v.b": torch.zeros(G * dv)}
    W["q.b"][0::d] = 1.0                       # every query: the first axis
    W["k"][0, 0], W["k"][1, 1] = 1.0, 1.0      # a key lies along its input's channel 0 (answers) or 1 (does not)
    h = bf(torch.randn(T, width) * 0.5)
    h[:, 0], h[:, 1] = 0.0, 1.0
    h[lo:hi + 1, 0], h[lo:hi + 1, 1] = 1.0, 0.0
    h[lo:hi + 1, 2:] = bf(torch.randn(width - 2) * 3)          # equal values: the block's mean is the tokens' value
    W64 = {k: v.to(F64) for k, v in W.items()}
    want = so.attention(h.to(F64), W64, "", m, 1e-6)
    marker = 0.5 * (h[lo].to(F64) @ W64["v"].T).repeat(H) @ W64["o"].T
    takes = row_errors(want, marker.expand(T, width)) < 1e-2
    assert [i for i in range(T) if takes[i]] == [i for i in range(T) if lo <= i <= hi + window - 1 or i >= hi + window]       # never unseen in between ...
    # ... because its last token leaves the window exactly when the block appears; without blocks it is gone, a position more it comes late
    late = row_errors(so.attention(h.to(F64), W64, "", dict(m, mask={"size": window}), 1e-6), marker.expand(T, width)) < 1e-2
    assert [i for i in range(T) if late[i]] == list(range(lo, hi + window))
    dt = torch.float32 if f32 else torch.bfloat16
    edge = hi + window
    for portions in ([T], [130, 2, 250], [edge], [edge - 1], [edge + 1], [edge - 1, 2, 200], [lo + 2, 2, 140]):
        bench = Bench([StateSpec("k", "append", G * d, dtype=dt), StateSpec("v", "append", G * dv, dtype=dt),
                       StateSpec("k.pool", "append", G * d, dtype=dt, every=P), StateSpec("v.pool", "append", G * dv, dtype=dt, every=P)], f32, max_pos=T)
        w = packer(W, f32).attention("", c)
        got = bench.portions(h, portions, lambda b, rows, out: b.softmax_attention(rows, c, w, "k", "v", out, eps=1e-6), width)
        assert float(row_errors(got, want).max()) < (TOL[True] if f32 else TOL[False]), portions


@pytest.mark.parametrize("f32", [True, False])
def test_a_single_token_just_inside_and_just_outside_the_window(f32):
    """One key that answers every query, in a block whose other keys do not: inside the window it takes the softmax; when it has left
    and its block is not yet seen it contributes nothing; afterwards a sixth of it comes back with the block's mean."""
    from qwen3_tts_cuda_graphs_b200.seq_state import StateSpec

    H, G, d, dv, width, T, window, P, j = 2, 2, 16, 16, 16, 120, 30, 6, 37        # position 37 lies in block 6 = 36 .. 41
    cfg = cases.config(8, width, [cases.layer(cases.attn(H, G, d, dv, window, P, 1.5))])
    m, c = cfg["layers"][0]["mixer"], layer_config(cfg).mixer
    torch.manual_seed(12)
    W = {"q": torch.zeros(H * d, width), "k": torch.zeros(G * d, width), "v": bf(torch.randn(G * dv, width) * 0.3), "o": bf(torch.randn(width, H * dv) * 0.3),
         "g": torch.zeros(H, width), "q.b": torch.zeros(H * d), "k.b": torch.zeros(G * d), "v.b": torch.zeros(G * dv)}
    W["q.b"][0::d] = 1.0
    W["k"][0::d, 0], W["k"][1::d, 1] = 1.0, 1.0
    h = bf(torch.randn(T, width) * 0.5)
    h[:, 0], h[:, 1] = 0.0, 1.0
    h[j, 0], h[j, 1] = 1.0, 0.0
    W64 = {k: v.to(F64) for k, v in W.items()}
    want = so.attention(h.to(F64), W64, "", m, 1e-6)
    h2 = h.clone()
    h2[j, 2:] += 2.0
    moved = (so.attention(h2.to(F64), W64, "", m, 1e-6) - want).abs().max(-1).values
    first_block = 41 + window
    assert all(float(moved[i]) > 0.1 for i in range(j, j + window)) and not moved[j + window:first_block].any() and float(moved[first_block]) > 1e-3
    dt = torch.float32 if f32 else torch.bfloat16
    for portions in ([T], [j + window], [j + window - 1, 2, 3], [first_block, 2], []):
        bench = Bench([StateSpec("k", "append", G * d, dtype=dt), StateSpec("v", "append", G * dv, dtype=dt),
                       StateSpec("k.pool", "append", G * d, dtype=dt, every=P), StateSpec("v.pool", "append", G * dv, dtype=dt, every=P)], f32, max_pos=T)
        w = packer(W, f32).attention("", c)
        got = bench.portions(h, portions, lambda b, rows, out: b.softmax_attention(rows, c, w, "k", "v", out, eps=1e-6), width)
        assert float(row_errors(got, want).max()) < (TOL[True] if f32 else TOL[False]), portions


def test_angles_stay_exact_thousands_of_positions_on():
    """Scores of +-60 between keys that turn fast, 2400 positions in: an angle that is only as good as one 32-bit product (an error of
    1e-4 at 2400 rad) would show tenfold above the tolerance, in the window and in the pooled keys far away."""
    from qwen3_tts_cuda_graphs_b200.seq_state import StateSpec

    H, G, d, dv, width, T, window, pool = 1, 1, 32, 8, 16, 2400, 40, 2
    cfg = cases.config(8, width, [cases.layer(cases.attn(H, G, d, dv, window, pool, 2.0, 32, base=7.0, factor=0.7))])
    W = sub_weights(cfg, "l0.mix.", seed=31)
    torch.manual_seed(14)
    h = bf(torch.randn(T, width))
    want = so.attention(h.to(F64), {k: v.to(F64) for k, v in W.items()}, "", cfg["layers"][0]["mixer"], 1e-6)
    c = layer_config(cfg).mixer
    bench = Bench([StateSpec("k", "append", G * d), StateSpec("v", "append", G * dv),
                   StateSpec("k.pool", "append", G * d, every=pool), StateSpec("v.pool", "append", G * dv, every=pool)], True, max_pos=T)
    w = packer(W, True).attention("", c)
    got = bench.portions(h, [2390, 2], lambda b, rows, out: b.softmax_attention(rows, c, w, "k", "v", out, eps=1e-6), width)
    assert float(row_errors(got, want).max()) < 1e-4, float(row_errors(got, want).max())


# ---------------------------------------------------------------------------------------------------------------------------
# whole models
# ---------------------------------------------------------------------------------------------------------------------------
CASES = {"odd": cases.odd, "unaligned": cases.unaligned, "aligned": cases.aligned, "once": cases.once}


@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("case", list(CASES))
def test_prompt_portions_and_decoding_agree_with_the_oracle(case, f32):
    cfg = CASES[case]()
    W = cases.weights(cfg, seed=7)
    T = 150 if case == "aligned" else 90
    toks = cases.tokens(cfg, T)
    taps = []
    want = so.forward(cfg, W, toks, taps)
    eng = make_engine(cfg, W, f32)
    whole = run_schedule(eng, toks, [T])
    assert close_enough(whole, want, f32), float(row_errors(whole, want).max())
    # the slot of the request above is used again by each of these
    for portions in ([2, 3, 1, 5, 2, 37, 2, 33], [60], [1] * 20, [T - 1]):
        got = run_schedule(eng, toks, portions)
        assert close_enough(got, want, f32), portions
        assert close_enough(got, whole.cpu(), f32), portions
    if f32:   # the residual stream after every layer run
        eng.step("taps", toks, [], layer_taps=True)
        assert len(eng.last_taps) == len(taps)
        for i, (a, b) in enumerate(zip(eng.last_taps, taps)):
            assert float(row_errors(a, b).max()) < TOL[True], i
        eng.close("taps")
    eng.close_all()


def test_every_pass_of_a_loop_keeps_states_of_its_own_and_mixes_the_embedding_in():
    cfg = cases.odd()
    W = cases.weights(cfg, seed=8)
    toks = cases.tokens(cfg, 40)
    want = so.forward(cfg, W, toks)
    eng = make_engine(cfg, W, True)
    got = run_schedule(eng, toks, [17, 2])
    assert float(row_errors(got, want).max()) < TOL[True]
    eng.close_all()
    for loop in ((1, 4, 2), (1, 3, 3), (2, 4, 3), None):      # the premises: other loops over the same tensors are other functions
        other = dict(cfg)
        other["loop"] = dict(zip(("start", "stop", "times"), loop)) if loop else None
        assert float(row_errors(so.forward(other, W, toks), want).median()) > 30 * TOL[True], loop
    half = dict(W)
    half["loop.in"] = W["loop.in"].clone()
    half["loop.in"][:, 44:] = 0.0
    assert float(row_errors(so.forward(cfg, half, toks), want).median()) > 30 * TOL[True]
    # one pass over everything, many passes over one layer, and a loop that ends with the stack
    for loop in ((0, 6, 1), (2, 3, 5), (3, 6, 2)):
        c2 = dict(cfg, loop=dict(zip(("start", "stop", "times"), loop)))
        eng = make_engine(c2, W, True)
        assert float(row_errors(run_schedule(eng, toks[:25], [11, 2]), so.forward(c2, W, toks[:25])).max()) < TOL[True], loop
        eng.close_all()


def _peaky_model(scale):
    return cases.config(64, 64, [
        cases.layer(cases.attn(4, 2, 16, 16, 41, 4, scale, 8, base=2000.0, factor=2.0), cases.dense(96)),
        cases.layer(cases.mlstm(2, 16, 16, 9.0)),
        cases.layer(cases.attn(4, 1, 16, 8, 100, 9, scale, 16, factor=1.3)),
        cases.layer(cases.hgrn(2, 16, 16)),
    ], loop=(0, 2, 2))


@pytest.mark.parametrize("f32", [True, False])
def test_peaked_attention_over_windows_and_blocks(f32):
    """Peaked attention (large scale on unit-RMS queries and keys) puts each row's mass on single keys and blocks.  Positions on both
    sides of the kernels' 32- and 64-key tiles, of their key-range splits, of the window edges and of block ends come both inside a
    prompt portion and decoded alone."""
    scale = 1.5 if f32 else 0.6          # bf16 products: milder peaks, fewer near-ties
    cfg = _peaky_model(scale)
    W = cases.weights(cfg, seed=9)
    T = 330
    toks = cases.tokens(cfg, T)
    want = so.forward(cfg, W, toks)
    eng = make_engine(cfg, W, f32, max_tokens=T)
    got_a = run_schedule(eng, toks, [T])
    got_b = run_schedule(eng, toks, [31, 33, 2, 36, 154, 2, 22])       # portions end at 31, 64, 66, 102, 256, 258, 280; the rest decoded
    for got in (got_a, got_b):
        assert close_enough(got, want, f32), float(row_errors(got, want).max())
    if f32:
        # the premises: a window one position longer, or blocks one position longer, answers differently by far more than the tolerance
        for li, mask in ((0, {"size": 42, "pool": 4}), (0, {"size": 41, "pool": 5}), (2, {"size": 101, "pool": 9}), (2, {"size": 100, "pool": 10})):
            c2 = _peaky_model(scale)
            c2["layers"][li]["mixer"]["mask"] = mask
            assert float(row_errors(so.forward(c2, W, toks[:200])[45:], want[45:200]).max()) > 10 * TOL[True], (li, mask)
    eng.close_all()


def test_requests_take_turns_in_two_slots_and_slots_are_reused():
    cfg = cases.odd()
    W = cases.weights(cfg, seed=10)
    eng = make_engine(cfg, W, True, max_slots=2)
    reqs = {n: cases.tokens(cfg, L, seed=i) for i, (n, L) in enumerate([("a", 23), ("b", 9), ("c", 41), ("d", 2)])}
    want = {n: so.forward(cfg, W, t) for n, t in reqs.items()}
    got = {n: [] for n in reqs}
    at = {n: 0 for n in reqs}
    # a and b interleaved with unequal portions; when b ends, c takes its slot (caches, pooled rows and carried states of b in it)
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


def test_long_decoding_past_windows_and_blocks():
    cfg = cases.odd()
    W = cases.weights(cfg, seed=11)
    toks = cases.tokens(cfg, 240)
    want = so.forward(cfg, W, toks)
    for f32 in (True, False):
        eng = make_engine(cfg, W, f32)
        got = run_schedule(eng, toks, [3])          # 237 tokens one by one through the caches, pooled rows and states
        assert close_enough(got, want, f32)
        eng.close_all()


def test_first_tokens_of_a_sequence():
    """One-token and two-token sequences, and the first positions of a longer one: shorter than every window, states at zero."""
    for make in (cases.unaligned, cases.odd, cases.once):
        cfg = make()
        W = cases.weights(cfg, seed=13)
        eng = make_engine(cfg, W, True, max_tokens=6)      # a capacity below a block's size is fine
        for n in (1, 2, 5):
            toks = cases.tokens(cfg, n, seed=n)
            assert float(row_errors(run_schedule(eng, toks, [n]), so.forward(cfg, W, toks)).max()) < TOL[True]
            assert float(row_errors(run_schedule(eng, toks, []), so.forward(cfg, W, toks)).max()) < TOL[True]
        eng.close_all()


def test_no_layers_and_a_single_layer():
    """A model without layers is the embedding, the output norm and the head."""
    bare = cases.config(23, 12, [])
    Wb = cases.weights(bare, seed=15)
    eng = make_engine(bare, Wb, True)
    few = cases.tokens(bare, 9)
    assert float(row_errors(run_schedule(eng, few, [4]), so.forward(bare, Wb, few)).max()) < TOL[True]
    eng.close_all()
    one = cases.config(23, 12, [cases.layer(cases.hgrn(1, 4, 6), cases.dense(5))], loop=(0, 1, 4))
    Wo = cases.weights(one, seed=16)
    eng = make_engine(one, Wo, True)
    assert float(row_errors(run_schedule(eng, few, [4]), so.forward(one, Wo, few)).max()) < TOL[True]
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
        lg = so.forward(cfg, W, toks)[-1]
        top = torch.topk(lg, 2).values
        margins.append(float(top[0] - top[1]))
        toks.append(int(lg.argmax()))
    return toks[len(prompt):], margins


def _greedy_cases():
    cfg = cases.odd()
    W = cases.weights(cfg, seed=12)
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
        ref_a, ref_b = so.forward(cfg, W, a), so.forward(cfg, W, b)
        for step, ref, places in ((0, ref_a, [0, 3, 18]), (2, ref_a, [21]), (3, ref_a, [23, 22]), (4, ref_b, [5])):
            got = torch.from_numpy(np.fromfile(out_dir / dtype / f"{step}.f32", dtype="<f4").reshape(len(places), cfg["vocab"]))
            assert float(row_errors(got, ref[places]).max()) < tol, (dtype, step)
