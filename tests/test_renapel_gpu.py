"""Renapel on the GPU: every new kernel and kernel option beside its plain statement (also with weights and inputs made so
that one key, one distance, a sink or a lost state shows), and the model through the engine, the generation entry point
and the trace-replay program against the plain whole-sequence implementation, in 32-bit and in bfloat16."""
import json
import math
import subprocess
import sys
from pathlib import Path

import pytest
import torch

import plain_ops
import plain_renapel as plain
from test_duvozen_gpu import EXPANDED_CASES, LATENT_CASES, off
from test_mefolorn_gpu import BATCHES, Batch, _close, only_generic
from tiny_renapel import CONFIGS, make_folder, random_tokens

pytestmark = pytest.mark.gpu

PAGE = 64
DEV = "cuda:0"


def _ops():
    from llm_b200 import ops
    return ops


# ----------------------------------------------------------------------------- residual streams

@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("case", [(36, 1, 1), (97, 2, 3), (128, 3, 8), (260, 4, 1), (2048, 4, 8), (4100, 3, 2), (64, 5, 4), (132, 16, 1), (4096, 6, 3)])
def test_streams(dtype, case):
    ops = _ops()
    width, S, terms = case
    gen = torch.Generator().manual_seed(width + S)
    new = lambda *shape: torch.randn(shape, generator=gen).to(DEV)
    for n in (1, 9, 300):
        X, y, write, read, gain = new(n, S, width), new(n * terms, width), new(S + S * S), new(S), 1.0 + 0.3 * new(width)
        for wanted in (True, False):
            got, want = X.clone(), X.clone()
            out = torch.zeros((n, width), dtype=dtype, device=DEV) if wanted else None
            other = out.clone() if wanted else None
            extra = (read, gain, 1e-3) if wanted else ()
            ops.streams_update_(got, y, terms, write, *extra, **({"out": out} if wanted else {}))
            plain_ops.streams_update_(want, y, terms, write, *extra, **({"out": other} if wanted else {}))
            _close(got, want, torch.float32, (case, n))
            if wanted:
                _close(out, other, dtype, (case, n, "input"))
        rows = torch.tensor([n - 1, 0], dtype=torch.int32, device=DEV)
        for weights in (read, None):
            for which in (None, rows):
                _close(ops.streams_read(X, weights, gain, 1e-3, dtype, rows=which),
                       plain_ops.streams_read(X, weights, gain, 1e-3, dtype, rows=which), dtype, (case, "read"))
        tokens = torch.randint(0, 50, (n,), generator=gen).to(torch.int32).to(DEV)
        table = new(50, width).to(dtype)
        assert torch.equal(ops.streams_embed(tokens, table, S, 0.5), plain_ops.streams_embed(tokens, table, S, 0.5))


@pytest.mark.parametrize("width", [2048, 4096, 6148])
def test_streams_give_a_token_the_same_bits_in_any_step(width):
    """Steps of few and of many tokens take different launches: a token's streams and its input are equal to the last bit."""
    ops = _ops()
    S, n = 4, 300
    gen = torch.Generator().manual_seed(width)
    new = lambda *shape: torch.randn(shape, generator=gen).to(DEV)
    X, y, write, read, gain = new(n, S, width), new(n * 2, width), new(S + S * S), new(S), new(width)
    whole, part = X.clone(), X[:7].clone()
    out, few = torch.zeros((n, width), device=DEV), torch.zeros((7, width), device=DEV)
    ops.streams_update_(whole, y, 2, write, read, gain, 1e-5, out)
    ops.streams_update_(part, y[:14].contiguous(), 2, write, read, gain, 1e-5, few)
    assert torch.equal(whole[:7], part) and torch.equal(out[:7], few)
    assert torch.equal(ops.streams_read(whole, read, gain, 1e-5, torch.float32), out)


def test_streams_mix_from_the_first_index_to_the_second():
    """One entry of the mixture, one of the spread: the right stream gets the right share, alone."""
    ops = _ops()
    S, width = 3, 64
    gen = torch.Generator().manual_seed(1)
    X, y = torch.randn((2, S, width), generator=gen).to(DEV), torch.randn((2, width), generator=gen).to(DEV)
    for source in range(S):
        for target in range(S):
            write = torch.zeros(S + S * S, device=DEV)
            write[S + source * S + target] = 2.0
            write[source] = 3.0
            got = X.clone()
            ops.streams_update_(got, y, 1, write)
            want = torch.zeros_like(X)
            want[:, target] += 2.0 * X[:, source]
            want[:, source] += 3.0 * y
            assert torch.allclose(got, want, atol=1e-6), (source, target)


# ----------------------------------------------------------------------------- the recurrence with fixed decays

def _recurrence_inputs(H, D, V, n, slots, dtype, seed):
    gen = torch.Generator().manual_seed(seed)
    width = (2 * H * (D + V) + 7) // 8 * 8 + 8
    proj = torch.randn((n, width), generator=gen).to(dtype).to(DEV)
    decays = (0.3 + 0.7 * torch.rand(H, generator=gen)).to(DEV)
    weight = (1.0 + 0.3 * torch.randn(H * V, generator=gen)).to(DEV)
    state = torch.randn((slots, H * D * V + 4), generator=gen).to(DEV)
    return proj, decays, weight, state


def _recurrence(fn, proj, decays, weight, state, batch, H, D, V, dtype, eps=1e-4):
    ops = _ops()
    n = batch.n_tokens
    work = torch.zeros((n, ops.decay_recurrence_work_width(H, D, V)), device=DEV)
    o = torch.zeros((n, H * V), device=DEV)
    mixed = torch.zeros((n, H * V + 9), dtype=dtype, device=DEV)
    fn(proj, decays, state, batch.cu, batch.slots, weight, eps, work, o, mixed[:, 4:4 + H * V], H, D, V,
       single_tokens=all(k == 1 for k in batch.new))
    return mixed


# heads, state rows, value size (rows around the lanes' multiples, columns around a block's)
RECURRENCE_CASES = [(3, 5, 7), (2, 33, 3), (4, 32, 48), (2, 72, 40), (1, 128, 128), (2, 130, 64), (1, 256, 130), (1, 20, 300),
                    (5, 64, 32), (1, 300, 16), (2, 128, 200), (8, 64, 64)]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("case", RECURRENCE_CASES)
def test_decay_recurrence(dtype, case):
    ops = _ops()
    H, D, V = case
    for lengths, new in BATCHES + [([130, 64, 129, 5, 2], [130, 3, 129, 5, 1]), ([65, 63, 300], [65, 63, 300])]:
        batch = Batch(lengths, new, seed=1)
        proj, decays, weight, state = _recurrence_inputs(H, D, V, batch.n_tokens, len(lengths) + 2, dtype, D + V)
        states = [state.clone(), state.clone()]
        got = _recurrence(ops.decay_recurrence, proj, decays, weight, states[0], batch, H, D, V, dtype)
        want = _recurrence(plain_ops.decay_recurrence, proj, decays, weight, states[1], batch, H, D, V, dtype)
        torch.cuda.synchronize()
        _close(got, want, dtype, (case, lengths, "out"))
        top = float(states[1].abs().max())                                              # also the slots and columns that no one owns
        assert float((states[0] - states[1]).abs().max()) <= (3e-6 if dtype == torch.float32 else 1e-2) * top, (case, lengths)


@pytest.mark.parametrize("case", [(3, 32, 48), (2, 64, 64), (1, 96, 40), (4, 128, 128), (2, 128, 8)])
def test_chunks_of_tokens_agree_with_the_scan_to_32_bit(case):
    """The chunked form beside the scan on inputs whose silu is exact in bfloat16 (0 and whole numbers of 20 and more), with
    a state of 32-bit numbers: what is left is the order of the sums. Steps that end inside a chunk, on its edge and just
    beyond; sequences of one token beside long ones; small and large decays, zero and one."""
    ops = _ops()
    H, D, V = case
    for lengths, new in (([64], [64]), ([65, 63, 300], [65, 63, 300]), ([200, 9, 1, 129], [130, 2, 1, 128]), ([17], [17]), ([700, 1], [640, 1])):
        batch = Batch(lengths, new, seed=1)
        gen = torch.Generator().manual_seed(D + len(new))
        n, width = batch.n_tokens, 2 * H * (D + V)
        whole = torch.randint(20, 40, (n, width), generator=gen).float() * (torch.rand((n, width), generator=gen) < 0.3)
        proj = whole.to(torch.bfloat16).to(DEV)
        decays = torch.tensor([0.999, 0.6, 0.0, 1.0][:H], device=DEV)
        state = (1e4 * torch.randn((len(lengths) + 1, H * D * V), generator=gen)).abs().to(DEV)
        results = []
        for without in ((), ("decay_recurrence_chunks",)):
            held, o = state.clone(), torch.zeros((n, H * V), device=DEV)
            work = torch.zeros((n, ops.decay_recurrence_work_width(H, D, V)), device=DEV)
            mixed = torch.zeros((n, H * V), dtype=torch.bfloat16, device=DEV)
            with off(*without):
                ops.decay_recurrence(proj, decays, held, batch.cu, batch.slots, torch.ones(H * V, device=DEV), 1e-5, work, o, mixed,
                                     H, D, V, single_tokens=False)
            results.append((o, held))
        assert float(results[1][0].abs().max()) > 0.0
        for got, want in zip(*results):
            assert torch.allclose(got, want, rtol=3e-6, atol=0.0), (case, new, float(((got - want).abs() / want.abs().clamp_min(1e-20)).max()))


@pytest.mark.parametrize("case", [(2, 12, 10), (1, 128, 128), (2, 100, 36)])
def test_decay_recurrence_carries_its_state_across_any_cut(case):
    """A sequence in one step, and the same cut into two (the second also token by token, in the launch of its own for
    steps of one token): the same results and states to the last bit in 32-bit."""
    ops = _ops()
    H, D, V = case
    n = 21
    proj, decays, weight, state = _recurrence_inputs(H, D, V, n, 3, torch.float32, 9)
    state.zero_()
    whole = state.clone()
    want = _recurrence(ops.decay_recurrence, proj, decays, weight, whole, Batch([n], [n]), H, D, V, torch.float32)
    for cut in range(1, n):
        held = state.clone()
        head = _recurrence(ops.decay_recurrence, proj[:cut], decays, weight, held, Batch([cut], [cut]), H, D, V, torch.float32)
        if cut % 2:
            tail = _recurrence(ops.decay_recurrence, proj[cut:], decays, weight, held, Batch([n], [n - cut]), H, D, V, torch.float32)
        else:
            tail = torch.cat([_recurrence(ops.decay_recurrence, proj[t:t + 1], decays, weight, held, Batch([t + 1], [1]), H, D, V,
                                          torch.float32) for t in range(cut, n)])
        assert torch.equal(torch.cat([head, tail]), want), cut
        assert torch.equal(held, whole), cut


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_decay_recurrence_reads_back_what_it_stored_hundreds_of_tokens_ago(dtype):
    """Token 0 alone writes under state row 0, with a decay of one; the 400 tokens between write under other rows, and the
    last token reads row 0 only: it gets token 0's value back. With the state lost on the way it does not."""
    ops = _ops()
    H, D, V, n = 1, 32, 8, 402
    gen = torch.Generator().manual_seed(2)
    proj = torch.zeros((n, 2 * D + 2 * V))
    proj[:, 1:D] = torch.rand((n, D - 1), generator=gen)                       # q away from row 0
    proj[:, D + 1:2 * D] = torch.randn((n, D - 1), generator=gen)              # k of the other rows
    proj[0, D] = 40.0                                                          # token 0 writes row 0
    proj[:, 2 * D:2 * D + V] = 3.0 * torch.randn((n, V), generator=gen)
    proj[-1, :D] = 0.0
    proj[-1, 0] = 40.0                                                         # the last token reads row 0
    proj = proj.to(dtype).to(DEV)
    decays, weight = torch.ones(1, device=DEV), torch.full((V,), 2.0, device=DEV)      # (a gate of zero halves)
    stored = torch.nn.functional.silu(proj[0, 2 * D:2 * D + V].float())

    def run(lose_at=None):
        state, outs = torch.zeros((1, D * V), device=DEV), []
        for lo, hi in ((0, 150), (150, 151), (151, 300), (300, n)):
            if lose_at == lo:
                state.zero_()
            outs.append(_recurrence(ops.decay_recurrence, proj[lo:hi], decays, weight, state, Batch([hi], [hi - lo]), H, D, V,
                                    dtype, eps=1e-12)[:, 4:4 + V])
        return torch.cat(outs)[-1].float()

    want = stored / torch.sqrt((stored * stored).mean())
    assert torch.allclose(run(), want, atol=1e-4 if dtype == torch.float32 else 0.02)
    assert float((run(lose_at=300) - want).abs().max()) > 0.3


def test_decay_recurrence_fades_by_each_head_s_decay():
    """One write, then reads of the same row: head h gives decay_h^distance of what was written, whatever the cut."""
    ops = _ops()
    H, D, V, n = 3, 64, 16, 140
    decays = torch.tensor([0.5, 0.97, 0.999], device=DEV)
    proj = torch.zeros((n, 2 * H * (D + V)), device=DEV)
    proj[0, H * D:2 * H * D] = 30.0 / D
    proj[0, 2 * H * D:2 * H * D + H * V] = 30.0
    proj[:, :H * D] = 30.0
    for dtype in (torch.float32, torch.bfloat16):
        state = torch.zeros((1, H * D * V), device=DEV)
        for lo, hi in ((0, 64), (64, 65), (65, 129), (129, n)):
            _recurrence(ops.decay_recurrence, proj[lo:hi].to(dtype), decays, torch.ones(H * V, device=DEV), state,
                        Batch([hi], [hi - lo]), H, D, V, dtype)
            k = 30.0 / D
            wrote = k / (1.0 + math.exp(-k)) * 30.0
            want = (wrote * decays ** (hi - 1))[:, None].expand(H, V * D)
            assert torch.allclose(state.view(H, V * D), want, rtol=2e-4 if dtype == torch.float32 else 1e-2, atol=0.0), (dtype, hi)


# ----------------------------------------------------------------------------- queries, keys and values before the cache

@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("case", [(6, 2, 6, 10), (4, 1, 64, 64), (3, 3, 96, 32), (2, 1, 128, 128)])
def test_unit_norm_and_temperature(dtype, case):
    """Norms without a weight per head, a number by position on the queries; with keys and values, and queries alone."""
    ops = _ops()
    heads, groups, dim, vdim = case
    gen = torch.Generator().manual_seed(dim)
    ones, scales = torch.ones(dim, device=DEV), (1.0 + torch.rand(400, generator=gen)).to(DEV)
    for lengths, new in BATCHES:
        batch = Batch(lengths, new, seed=len(lengths))
        for alone in (False, True):
            kw, vw = (0, 0) if alone else (groups * dim, groups * vdim)
            u = torch.randn((batch.n_tokens, heads * dim + kw + vw + 3), generator=gen).to(dtype).to(DEV)
            results = []
            for fn in (ops.norm_rope_cache_write, plain_ops.norm_rope_cache_write):
                k, v = batch.caches(groups, dim, vdim, dtype)
                q = torch.zeros((batch.n_tokens, heads * dim), dtype=dtype, device=DEV)
                fn(u, heads * dim, kw, vw, ones, ones, 1e-3, None, dim, False, batch.tok_pos, batch.tok_seq, q, batch.table,
                   batch.width, k, v, write_cache=not alone, norm_unit=dim, q_scale=scales)
                results.append((q, k, v))
            for got, want in zip(*results):
                _close(got, want, dtype, (case, alone))


# ----------------------------------------------------------------------------- attention with a bias by distance

KERNELS = {"first": (torch.bfloat16, ()), "mma": (torch.bfloat16, ("attention_prefill_tc",)),
           "generic": (torch.bfloat16, ("generic",)), "32-bit": (torch.float32, ())}


def _attend(fn, which, batch, q, k, v, heads, groups, dim, scale, sinks, bias, vdim=None):
    dtype, without = KERNELS[which]
    out = torch.zeros((batch.n_tokens, heads * (vdim or dim)), dtype=dtype, device=DEV)
    with only_generic("generic" in without), off(*(n for n in without if n != "generic")):
        fn(q, k, v, batch.table, batch.width, batch.tok_pos, batch.tok_seq, heads, groups, dim, scale, 0, out=out, sinks=sinks,
           bias=bias, value_dim=vdim, **batch.extra())
    return out


@pytest.mark.parametrize("which", sorted(KERNELS))
@pytest.mark.parametrize("case", [(8, 2, 64, 114), (4, 1, 128, 500), (6, 2, 96, 33), (2, 2, 32, 1), (3, 1, 64, 2000), (10, 1, 128, 64), (4, 2, 128, 130)])
def test_attention_with_a_bias_by_distance(which, case):
    """Whole prompts, later portions and decode steps; biases of the order of the scores and larger; tables that end at once,
    inside a page, inside a tile, and beyond every sequence; groups of more than eight heads."""
    ops = _ops()
    heads, groups, dim, span = case
    dtype = KERNELS[which][0]
    gen = torch.Generator().manual_seed(dim + span)
    sinks = torch.linspace(-3.0, 4.0, heads).to(DEV)
    bias = (2.0 * torch.randn((heads, span), generator=gen)).to(DEV)
    for lengths, new in BATCHES + [([700, 64, 129], [700, 3, 129]), ([1500, 1, 64, 65, 700], [1] * 5)]:
        batch = Batch(lengths, new, seed=3 + len(lengths))
        q = (2.0 * torch.randn((batch.n_tokens, heads * dim), generator=gen)).to(dtype).to(DEV)
        k, v = batch.caches(groups, dim, dim, dtype, seed=3)
        got, want = (_attend(fn, which, batch, q, k, v, heads, groups, dim, dim ** -0.5, sinks, bias)
                     for fn in (ops.attention, plain_ops.attention))
        torch.cuda.synchronize()
        ops.check_device_status()
        _close(got, want, dtype, (case, lengths))


@pytest.mark.parametrize("which", sorted(KERNELS))
@pytest.mark.parametrize("decode", [False, True])
def test_one_distance_stands_out(which, decode):
    """Queries of zero; one distance has a bias of 30, all others none: every query gets the value of the key at exactly that
    distance (each key's value says its position), or a mean of all where there is none; the last column of the table
    stands out at every distance from its own on."""
    ops = _ops()
    dtype, length, dim, heads = KERNELS[which][0], 333, 64, 2
    batch = Batch([length, 90], [1, 1] if decode else [length, 90], seed=7)
    v, k = (torch.zeros((batch.n_pages, 1, PAGE, dim), dtype=dtype, device=DEV) for _ in range(2))
    for b, n in enumerate(batch.lengths):
        for p in range(n):
            page, row = batch.place(b, p)
            v[page, 0, row, 0], v[page, 0, row, 1] = p % 16, p // 16
    q = torch.zeros((batch.n_tokens, heads * dim), dtype=dtype, device=DEV)
    span = 200
    for distance in (0, 1, 14, 15, 16, 62, 63, 64, 65, 127, 128, 129, 198):
        bias = torch.zeros((heads, span), device=DEV)
        bias[:, distance] = 30.0
        out = _attend(ops.attention, which, batch, q, k, v, heads, 1, dim, 0.4, None, bias).float().view(-1, heads, dim)
        for t, p in enumerate(batch.tok_pos.tolist()):
            at = p - distance
            want = (at % 16, at // 16) if at >= 0 else (sum(x % 16 for x in range(p + 1)) / (p + 1), sum(x // 16 for x in range(p + 1)) / (p + 1))
            assert abs(float(out[t, 1, 0]) - want[0]) < 0.08 and abs(float(out[t, 0, 1]) - want[1]) < 0.08, (distance, t, p)
    bias = torch.zeros((heads, span), device=DEV)
    bias[:, -1] = 30.0
    out = _attend(ops.attention, which, batch, q, k, v, heads, 1, dim, 0.4, None, bias).float().view(-1, heads, dim)
    for t, p in enumerate(batch.tok_pos.tolist()):
        seen = p - span + 2 if p >= span - 1 else p + 1                         # keys at least span - 1 back, or all
        assert abs(float(out[t, 0, 1]) - sum(x // 16 for x in range(seen)) / seen) < 0.08, (t, p)


def test_bias_with_values_of_another_size():
    ops = _ops()
    gen = torch.Generator().manual_seed(4)
    for dtype_name in ("32-bit", "first"):
        dtype = KERNELS[dtype_name][0]
        for lengths, new in BATCHES:
            batch = Batch(lengths, new, seed=2)
            q = torch.randn((batch.n_tokens, 4 * 32), generator=gen).to(dtype).to(DEV)
            k, v = batch.caches(2, 32, 20, dtype, seed=3)
            bias, sinks = torch.randn((4, 50), generator=gen).to(DEV), torch.zeros(4, device=DEV)
            got, want = (_attend(fn, dtype_name, batch, q, k, v, 4, 2, 32, 0.2, sinks, bias, 20) for fn in (ops.attention, plain_ops.attention))
            _close(got, want, dtype, lengths)


# ----------------------------------------------------------------------------- latent attention: queries' latent, sinks

@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("case", [(3, 5, 6, 11, 13), (4, 64, 16, 80, 48), (20, 16, 8, 40, 136), (2, 128, 64, 512, 1536)])
def test_latent_write_with_a_latent_of_the_queries(dtype, case):
    ops = _ops()
    H, D, R, C, Q = case
    gen = torch.Generator().manual_seed(D + C)
    gain, q_gain = ((1.0 + 0.3 * torch.randn(n, generator=gen)).to(DEV) for n in (C, Q))
    angle = torch.arange(400, dtype=torch.float64)[:, None] * torch.rand(R // 2, generator=gen, dtype=torch.float64)
    table = torch.cat([angle.cos(), angle.sin()], dim=1).float().to(DEV)
    for lengths, new in BATCHES:
        batch = Batch(lengths, new, seed=len(lengths))
        n = batch.n_tokens
        u = torch.randn((n, Q + C + R + 8), generator=gen).to(dtype).to(DEV)
        heads = torch.randn((n, H * (D + R)), generator=gen).to(dtype).to(DEV)
        for in_place in (True, False):
            results = []
            for m in (ops, plain_ops):
                cache, _ = batch.caches(1, C + R, 0, dtype)
                cq, dense = torch.zeros((n, Q), dtype=dtype, device=DEV), torch.zeros((n, C + R), dtype=dtype, device=DEV)
                mine, queries = heads.clone(), None if in_place else torch.zeros((n, H * (C + R)), dtype=dtype, device=DEV)
                m.latent_write(u, H, D, R, C, gain, 1e-3, table, True, batch.tok_pos, batch.tok_seq, batch.table, batch.width,
                               cache, dense=dense if in_place else None, q_rank=Q, q_gain=q_gain, cq=cq)
                m.latent_rotate(mine, H, D, R, C, table, True, batch.tok_pos, queries=queries)
                results.append([cache, cq, dense, mine] + ([] if in_place else [queries]))
            for i, (got, want) in enumerate(zip(*results)):
                _close(got, want, dtype, (case, in_place, i))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16, "tiles", "generic"])
@pytest.mark.parametrize("case", LATENT_CASES)
def test_latent_attention_with_sinks(dtype, case):
    """Sinks far below, among and far above the scores; whole prompts, later portions and decode steps (one slice and
    several), each head against its own size."""
    ops = _ops()
    without = {"tiles": ("latent_decode_tc",), "generic": ("latent_decode_tc", "latent_tiles")}.get(dtype, ())
    dtype = torch.bfloat16 if without else dtype
    H, C, R = case
    sinks = torch.linspace(-20.0, 20.0, H).to(DEV) if H > 1 else torch.tensor([2.0], device=DEV)
    for lengths, new in BATCHES + [([700, 1, 64, 65, 300], [1] * 5), ([1500], [1])]:
        batch = Batch(lengths, new, seed=3 + len(lengths))
        gen = torch.Generator().manual_seed(C)
        q = (2.0 * torch.randn((batch.n_tokens, H * (C + R)), generator=gen)).to(dtype).to(DEV)
        cache, _ = batch.caches(1, C + R, 0, dtype, seed=4)
        results = []
        for fn in (ops.latent_attention, plain_ops.latent_attention):
            out = torch.zeros((batch.n_tokens, H * C), dtype=dtype, device=DEV)
            with off(*without):
                fn(q, cache, batch.table, batch.width, batch.tok_pos, batch.tok_seq, H, C, R, (C + R) ** -0.5, out, sinks=sinks,
                   **batch.extra())
            results.append(out.view(-1, H, C).float())
        torch.cuda.synchronize()
        ops.check_device_status()
        for h in range(H):
            got, want = results[0][:, h], results[1][:, h]
            top = float(want.abs().max()) + 1e-20
            assert float((got - want).abs().max()) <= (5e-5 if dtype == torch.float32 else 0.03) * top, (case, lengths, h)


@pytest.mark.parametrize("case", EXPANDED_CASES)
def test_latent_prefill_with_sinks(case):
    ops = _ops()
    H, D, R, V, C = case
    sinks = torch.linspace(-20.0, 20.0, H).to(DEV) if H > 1 else torch.tensor([1.5], device=DEV)
    bf16 = torch.bfloat16
    for new in ([70, 5, 130, 64], [1], [300, 257, 1]):
        batch = Batch(new, new, seed=len(new))
        n = batch.n_tokens
        gen = torch.Generator().manual_seed(D + R + n)
        heads = (2.0 * torch.randn((n, H * (D + R)), generator=gen)).to(bf16).to(DEV)
        kv, dense = torch.randn((n, H * (D + V)), generator=gen).to(bf16).to(DEV), torch.randn((n, C + R), generator=gen).to(bf16).to(DEV)
        got, want = (torch.zeros((n, H * V), dtype=bf16, device=DEV) for _ in range(2))
        args = (heads, kv, dense, H, D, R, V, C, (D + R) ** -0.5)
        ops.latent_prefill(*args, got, batch.cu, max(new), batch.order, sinks=sinks)
        plain_ops.latent_prefill(*args, want, batch.cu.cpu(), max(new), sinks=sinks)
        torch.cuda.synchronize()
        ops.check_device_status()
        for h in range(H):
            part = slice(h * V, (h + 1) * V)
            top = float(want[:, part].float().abs().max()) + 1e-20
            assert float((got[:, part].float() - want[:, part].float()).abs().max()) <= 0.03 * top, (case, new, h)


def test_the_sink_s_share_of_latent_rows():
    """Queries of zero: every row has the weight 1 / (n + e^sink), on every kernel and in both forms."""
    ops = _ops()
    sink = torch.full((4,), math.log(7.0), device=DEV)
    for dtype, without in ((torch.float32, ()), (torch.bfloat16, ()), (torch.bfloat16, ("latent_decode_tc",)),
                           (torch.bfloat16, ("latent_decode_tc", "latent_tiles"))):
        for lengths, new in (([100], [100]), ([100, 3], [1, 1]), ([1400], [1])):
            batch = Batch(lengths, new)
            cache, _ = batch.caches(1, 64 + 16, 0, dtype)
            cache[..., :64] = 1.0
            q = torch.zeros((batch.n_tokens, 4 * 80), dtype=dtype, device=DEV)
            out = torch.zeros((batch.n_tokens, 4 * 64), dtype=dtype, device=DEV)
            with off(*without):
                ops.latent_attention(q, cache, batch.table, batch.width, batch.tok_pos, batch.tok_seq, 4, 64, 16, 0.3, out, sinks=sink,
                                     **batch.extra())
            n = (batch.tok_pos + 1).float()[:, None]
            assert torch.allclose(out.float(), (n / (n + 7.0)).expand_as(out), atol=1e-5 if dtype == torch.float32 else 6e-3)
    n, bf16 = 100, torch.bfloat16
    batch = Batch([n], [n])
    kv = torch.ones((n, 4 * 128), dtype=bf16, device=DEV)
    out = torch.zeros((n, 4 * 64), dtype=bf16, device=DEV)
    ops.latent_prefill(torch.zeros((n, 4 * 80), dtype=bf16, device=DEV), kv, torch.ones((n, 48), dtype=bf16, device=DEV), 4, 64, 16, 64, 32,
                       0.3, out, batch.cu, n, batch.order, sinks=sink)
    count = torch.arange(1, n + 1, device=DEV, dtype=torch.float32)[:, None]
    assert torch.allclose(out.float(), (count / (count + 7.0)).expand_as(out), atol=6e-3)


# ----------------------------------------------------------------------------- experts

def _experts(fn, h, router, w_up, w_down, top, **options):
    ops = _ops()
    n, hidden = h.shape
    E, F = w_up.shape[0], w_up.shape[1] // 2
    a = n * top
    ids, order = (torch.zeros(a, dtype=torch.int32, device=DEV) for _ in range(2))
    weights = torch.zeros(a, device=DEV)
    plan = torch.zeros(ops.routed_experts_plan_ints(n, top, E), dtype=torch.int32, device=DEV)
    act = torch.zeros((a, F), dtype=h.dtype, device=DEV)
    y = torch.full((a, hidden), 77.0, device=DEV)
    gathered = torch.zeros((a, hidden), dtype=h.dtype, device=DEV)
    fn(h, router, None, w_up, w_down, top, ids, weights, order, plan, act, y, gathered, scoring=1, **options)
    return y, ids, weights


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("case", [
    # width, expert width, experts, chosen, groups, groups kept
    (40, 12, 6, 3, 3, 2), (128, 64, 8, 2, 4, 1), (128, 96, 4, 1, 1, 1), (32, 16, 1, 1, 1, 1), (256, 128, 16, 4, 8, 3), (136, 40, 8, 8, 2, 2),
    (320, 104, 12, 4, 4, 2), (64, 32, 40, 20, 4, 3), (64, 32, 9, 2, 9, 4)])
def test_clamped_experts_in_groups(dtype, case):
    """The groups' choice and the clamped activation (limits that bite both ways) in all forms of the products."""
    ops = _ops()
    hidden, F, E, top, groups, keep = case
    gen = torch.Generator().manual_seed(hidden + E)
    router = (2.0 * torch.randn((E, hidden), generator=gen) / hidden ** 0.5).to(DEV)
    w_up = (2.0 * torch.randn((E, 2 * F, hidden), generator=gen) / hidden ** 0.5).to(dtype).to(DEV)
    w_down = (torch.randn((E, hidden, F), generator=gen) / F ** 0.5).to(dtype).to(DEV)
    options = dict(groups=groups, keep=keep, weight_scale=1.6, alpha=1.702)
    for n in (1, 7, 70, 600, 48 * E) if E <= 16 else (1, 70):      # few rows an expert, and enough for the tiles of 128 rows
        h = torch.randn((n, hidden), generator=gen).to(dtype).to(DEV)
        for limit in (1.0, 0.0, 30.0):
            got, got_ids, got_weights = _experts(ops.routed_experts, h, router, w_up, w_down, top, limit=limit, **options)
            want, want_ids, want_weights = _experts(plain_ops.routed_experts, h, router, w_up, w_down, top, limit=limit, **options)
            torch.cuda.synchronize()
            same = (got_ids.view(n, top) == want_ids.view(n, top)).all(dim=1)      # a close call may fall either way
            assert int(same.sum()) >= 0.95 * n, (case, n)
            rows = same.repeat_interleave(top)
            assert torch.allclose(got_weights[rows], want_weights[rows], atol=2e-6, rtol=2e-5)
            _close(got[rows], want[rows], dtype, (case, n, limit))
    alone, _, _ = _experts(ops.routed_experts, h[2:3] if n > 2 else h[:1], router, w_up, w_down, top, limit=1.0, **options)
    among, _, _ = _experts(ops.routed_experts, h[:5], router, w_up, w_down, top, limit=1.0, **options)
    assert torch.equal(alone, among.view(-1, top, hidden)[2 if n > 2 else 0])


def test_groups_decide_before_experts_do():
    """Scores made so that a choice without groups, by the groups' sums or by the wrong number of groups gives other
    experts; equal groups and equal experts fall to the lower index."""
    ops = _ops()
    logits = torch.tensor([[5.0, -9.0, 4.0, 3.9, 4.1, -9.0, 1.0, 0.9],         # peaks 5, 4, 4.1, 1; sums would put group 1 before 2
                           [2.0, 2.0, 2.0, 2.0, 2.0, 2.0, 2.0, 2.0],
                           [0.0, 1.0, 0.5, 0.4, 1.0, 0.0, 0.2, 3.0]], device=DEV)
    router = torch.eye(8, device=DEV)
    w_up, w_down = torch.zeros((8, 4, 8), device=DEV), torch.zeros((8, 8, 2), device=DEV)
    for keep, want in ((4, [[0, 4, 2], [0, 1, 2], [7, 1, 4]]), (2, [[0, 4, 1], [0, 1, 2], [7, 1, 6]]), (3, [[0, 4, 2], [0, 1, 2], [7, 1, 4]])):
        _, ids, weights = _experts(ops.routed_experts, logits, router, w_up, w_down, 3, groups=4, keep=keep, limit=1.0)
        assert ids.view(3, 3).tolist() == want, keep
        scores = torch.softmax(logits, -1).gather(1, torch.tensor(want, device=DEV))
        assert torch.allclose(weights.view(3, 3), scores / scores.sum(-1, keepdim=True), atol=1e-6)


# ----------------------------------------------------------------------------- the model

def _setup(tmp_path, which, dtype, change=None, weights_change=None, **engine_options):
    from llm_b200.engine import Engine, load_model
    folder = make_folder(tmp_path, which, torch.bfloat16, change, weights_change)
    config, weights = plain.read_model(folder)
    engine = Engine(load_model(folder, dtype, DEV), **{"max_tokens": 4096, **engine_options})
    return config, weights, engine


def _check_logits(got, want, dtype, what="", sure=None):
    """32-bit: element by element. bfloat16: against the span of the logits; a row at which the plain
    model chose its experts by less than a rounding's reach (`sure` False) is not looked at."""
    got, want = got.float().cpu(), want.float()
    if dtype == torch.float32:
        assert torch.allclose(got, want, atol=4e-4, rtol=1e-4), (what, float((got - want).abs().max()))
        return
    if got.dim() == 1:
        got, want = got[None], want[None]
        sure = None if sure is None else torch.as_tensor(sure).reshape(1)
    if sure is not None:
        got, want = got[sure], want[sure]
    if got.numel() == 0:
        return
    span = float(want.max() - want.min())
    assert float((got - want).abs().max()) <= 0.06 * span, (what, float((got - want).abs().max()), span)
    assert float((got - want).abs().mean()) <= 0.012 * span, what


MARGIN = 0.004          # of softmax scores: what bfloat16 rounding of the router's input reaches


def _sure(config, weights, tokens, dtype):
    """Per position: True up to the first position at which a routed layer chose by less than a rounding's reach (another
    expert there changes what every later position reads from the states and the cache)."""
    if dtype == torch.float32:
        return torch.ones(len(tokens), dtype=torch.bool)
    return torch.cummin(plain.closest_call(config, weights, tokens), dim=0).values > MARGIN


def _all_experts(config):
    """Every expert chosen: no close calls, so every position is compared in bfloat16 too."""
    for layer in config["layers"]:
        if layer["mlp"] is not None:
            r = layer["mlp"]["router"]
            r["experts"] = r["top"] = min(r["experts"], 4)
            r.pop("groups", None)


def test_every_layer_agrees_with_plain(tmp_path):
    """The residual after each layer in 32-bit (a model of the first k layers, for every k, whose last norm has a weight of
    one, and its last layer also without feed-forward)."""
    from llm_b200.engine import Entry
    for which in sorted(CONFIGS):
        depth = len(CONFIGS[which][0]["layers"])
        for k in range(1, depth + 1):
            for mixer_only in (True, False):
                def cut(config, k=k, mixer_only=mixer_only):
                    config["layers"] = config["layers"][:k]
                    if mixer_only:
                        config["layers"][-1]["mlp"] = None
                def plain_final(weights):
                    weights["final.norm"].fill_(1.0)
                config, weights, engine = _setup(tmp_path / f"{which}{k}{mixer_only}", which, torch.float32, cut, plain_final)
                tokens = random_tokens(80, config["vocab"], k)
                want = plain.forward(config, weights, tokens)
                (slot,) = engine.acquire()
                got = engine.step([Entry(slot, tokens, list(range(80)))])
                _check_logits(got, want, torch.float32, (which, k, mixer_only))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("which", sorted(CONFIGS))
def test_whole_decode_pieces_and_batches_agree_with_plain(tmp_path, which, dtype):
    from llm_b200.engine import Entry
    config, weights, engine = _setup(tmp_path, which, dtype, step_tokens=48)
    lengths = [150, 1, 67, 20]
    seqs = [random_tokens(n, config["vocab"], 30 + n) for n in lengths]
    expected = [plain.forward(config, weights, s) for s in seqs]
    sure = [_sure(config, weights, s, dtype) for s in seqs]
    for again in range(2):                                       # the second time reuses slots, pages and states
        slots = engine.acquire(len(seqs))
        heads = [max(1, n - 9 - 2 * i) for i, n in enumerate(lengths)]          # unequal prompts, cut into passes of 48
        logits = engine.step([Entry(s, q[:h], list(range(h))) for s, q, h in zip(slots, seqs, heads)])
        row = 0
        for b, h in enumerate(heads):
            _check_logits(logits[row:row + h], expected[b][:h], dtype, ("prompt", b), sure[b][:h])
            row += h
        live = [b for b in range(len(seqs)) if heads[b] < lengths[b]]
        engine.release([slots[b] for b in range(len(seqs)) if b not in live])
        done = 0
        while live:                                              # decoding together; shorter sequences end earlier
            logits = engine.step([Entry(slots[b], [seqs[b][heads[b] + done]], [0]) for b in live])
            for r, b in enumerate(live):
                at = heads[b] + done
                _check_logits(logits[r], expected[b][at], dtype, ("decode", b, done), sure[b][at])
            done += 1
            ended = [b for b in live if heads[b] + done == lengths[b]]
            engine.release([slots[b] for b in ended])
            live = [b for b in live if b not in ended]
        engine.cache.check()
        engine.check()
        assert engine.cache.slots.n_held == 0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_every_position_in_both_dtypes_however_it_is_cut(tmp_path, dtype):
    """All experts chosen: in one step (the latent attention with keys and values formed), in portions (the cached rows), and
    decoded."""
    from llm_b200.engine import Entry
    config, weights, engine = _setup(tmp_path, "Q", dtype, _all_experts)
    tokens = random_tokens(210, config["vocab"], 12)
    expected = plain.forward(config, weights, tokens)
    for cuts in ([210], [130, 80], [64, 2, 64, 80], [100] + [1] * 110):
        (slot,) = engine.acquire()
        at = 0
        for size in cuts:
            got = engine.step([Entry(slot, tokens[at:at + size], list(range(size)))])
            _check_logits(got, expected[at:at + size], dtype, (cuts[:3], at))
            at += size
        engine.release([slot])
    engine.check()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_long_decoding_passes_page_edges(tmp_path, dtype):
    """One token a step from the first on, 300 steps: pages fill and follow each other, the recurrences' states are carried
    300 times, distances leave the bias tables, and steps are replayed from graphs."""
    from llm_b200.engine import Entry
    config, weights, engine = _setup(tmp_path, "Q", dtype, _all_experts)
    tokens = random_tokens(300, config["vocab"], 77)
    expected = plain.forward(config, weights, tokens)
    (slot,) = engine.acquire()
    for p, token in enumerate(tokens):
        logits = engine.step([Entry(slot, [token], [0])])
        _check_logits(logits[0], expected[p], dtype, p)
    assert engine.graph_replays > 200


@pytest.mark.parametrize("piece", [2, 5, 64])
def test_pieces_down_to_two_tokens(tmp_path, piece):
    from llm_b200.engine import Entry
    for which in ("P", "Q"):
        config, weights, engine = _setup(tmp_path, which, torch.float32)
        tokens = random_tokens(140, config["vocab"], 8)
        expected = plain.forward(config, weights, tokens)
        (slot,) = engine.acquire()
        for start in range(0, len(tokens), piece):
            part = tokens[start:start + piece]
            logits = engine.step([Entry(slot, part, list(range(len(part))))])
            _check_logits(logits, expected[start:start + len(part)], torch.float32, (which, start))


def test_batch_and_cut_change_nothing_in_32_bit(tmp_path):
    """A position's logits alone, among neighbours, and with its prompt cut: equal to the last bit in the
    32-bit path (every reduction's order depends only on the position; states are carried exactly; an
    expert's rows do not depend on the tile they fall into)."""
    from llm_b200.engine import Entry
    for which in ("P", "Q"):
        config, weights, engine = _setup(tmp_path, which, torch.float32)
        seqs = [random_tokens(n, config["vocab"], 60 + n) for n in (50, 13, 31)]
        a, b, c, d = engine.acquire(4)
        alone = engine.step([Entry(a, seqs[0], [49, 20])]).clone()
        together = engine.step([Entry(b, seqs[1], [12]), Entry(c, seqs[0], [49, 20]), Entry(d, seqs[2], [])])
        assert torch.equal(alone, together[1:3]), which
        engine.release([a])
        (e,) = engine.acquire()
        engine.step([Entry(e, seqs[0][:17], [])])
        engine.step([Entry(e, seqs[0][17:21], [])])
        for t in range(21, 30):
            engine.step([Entry(e, [seqs[0][t]], [0])])
        cut = engine.step([Entry(e, seqs[0][30:], [49 - 30])])
        assert torch.equal(alone[0], cut[0]), which


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_passes_walked_from_their_record_agree_with_plain_passes(tmp_path, dtype):
    """The same shape of step five times on other slots, pages and states: the first pass runs through the parts,
    the second is recorded, the later ones are walked natively from the record; a mixed step and a later portion of a
    prompt (another form of the latent attention than its first) likewise."""
    from llm_b200.engine import Entry
    config, weights, engine = _setup(tmp_path, "Q", dtype, _all_experts)
    for again in range(5):
        seqs = [random_tokens(n, config["vocab"], 100 * again + n) for n in (90, 33)]
        slots = engine.acquire(2)
        want = [plain.forward(config, weights, s) for s in seqs]
        logits = engine.step([Entry(slots[0], seqs[0][:40], [0, 39]), Entry(slots[1], seqs[1][:15], [14])])
        _check_logits(logits, torch.stack([want[0][0], want[0][39], want[1][14]]), dtype, ("first", again))
        logits = engine.step([Entry(slots[0], seqs[0][40:80], [0, 39]), Entry(slots[1], seqs[1][15:30], [14])])
        _check_logits(logits, torch.stack([want[0][40], want[0][79], want[1][29]]), dtype, ("later", again))
        mixed = engine.step([Entry(slots[0], seqs[0][80:], [9]), Entry(slots[1], [seqs[1][30]], [0])])
        _check_logits(mixed, torch.stack([want[0][89], want[1][30]]), dtype, ("mixed", again))
        engine.release(slots)
    assert engine.records_run >= 8


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_a_far_key_read_through_another_layer_s_cache(tmp_path, dtype):
    """A layer that reads an earlier layer's keys and values and whose bias makes every key count from one distance on: at
    the position where only the first token is that far back, it decides the layer's result; one position earlier it is one
    of many. In a prompt and decoded, with the distance on both sides of page borders."""
    from llm_b200.engine import Entry
    rows = CONFIGS["S"][1][2]
    for far in (50.0, 157.0, 160.0, 163.0, 405.0):
        edge = next(n for n in range(400) if plain.bucket_of(n, rows, far) == rows - 1)

        def change(config):
            _all_experts(config)
            config["layers"][2]["mixer"]["bias_max"] = far

        def loud(weights):
            weights["l2.mix.rel"].zero_()
            weights["l2.mix.rel"][-1] = 16.0
            weights["l2.mix.o"] *= 4.0
        config, weights, engine = _setup(tmp_path / str(far), "S", dtype, change, loud)
        tokens = random_tokens(edge + 2, config["vocab"], 5)
        other = [(tokens[0] + 1) % config["vocab"]] + tokens[1:]
        moved = {}
        for seq in (tokens, other):
            want = plain.forward(config, weights, seq)
            slot, whole = engine.acquire(2)
            engine.step([Entry(slot, seq[:edge - 1], [])])
            for t in range(edge - 1, edge + 2):
                logits = engine.step([Entry(slot, [seq[t]], [0])])
                _check_logits(logits[0], want[t], dtype, (far, t))
                moved.setdefault(t, []).append(logits[0].float().cpu())
            _check_logits(engine.step([Entry(whole, seq, list(range(edge + 2)))]), want, dtype, (far, "prompt"))
            engine.release([slot, whole])
        before, at = (float((moved[t][0] - moved[t][1]).abs().max()) for t in (edge - 1, edge))
        assert at > 0.5 and at > 4 * before, (far, before, at)


def test_what_a_fault_would_change_shows_in_the_logits(tmp_path):
    """Changes that a fault would make, made on purpose in the plain model: each must move the logits by far
    more than the library differs from the unchanged plain model."""
    from llm_b200.engine import Entry
    config, weights, engine = _setup(tmp_path, "Q", torch.float32)
    tokens = random_tokens(160, config["vocab"], 5)
    want = plain.forward(config, weights, tokens)
    (slot,) = engine.acquire()
    got = engine.step([Entry(slot, tokens, list(range(160)))]).cpu()
    error = float((got - want).abs().max())
    for change in ("mixture turned", "spread", "input weights", "decay", "recurrence norm", "recurrence gate", "key bias", "query bias",
                   "temperature", "temperature's step", "bias far", "bias table", "own keys", "sink", "latent sink", "query latent norm",
                   "latent norm", "base", "limit", "router scale", "groups", "fewer experts", "values", "nothing"):
        other, w = json.loads(json.dumps(config)), dict(weights)
        layers = other["layers"]
        if change == "mixture turned":
            w["l3.hc2.mix"] = weights["l3.hc2.mix"].T.contiguous()
        elif change == "spread":
            w["l7.hc1.out"] = weights["l7.hc1.out"].flip(0)
        elif change == "input weights":
            w["l2.hc1.in"] = weights["l2.hc1.in"].flip(0)
        elif change == "decay":
            layers[7]["mixer"]["decay"] = [0.998, 0.5]
        elif change == "recurrence norm":
            w["l2.mix.norm"] = weights["l2.mix.norm"].flip(0)
        elif change == "recurrence gate":
            w["l2.mix.g"] = weights["l2.mix.g"] * 0.0
        elif change == "key bias":
            w["l0.mix.k.b"] = weights["l0.mix.k.b"] * 0.0
        elif change == "query bias":
            w["l4.mix.q.b"] = weights["l4.mix.q.b"] * 0.0
        elif change == "temperature":
            del layers[0]["mixer"]["q_temp"]
        elif change == "temperature's step":
            layers[6]["mixer"]["q_temp"]["every"] = 99
        elif change == "bias far":
            layers[0]["mixer"]["bias_max"] = 91
        elif change == "bias table":
            w["l3.mix.rel"] = weights["l3.mix.rel"].flip(1)
        elif change == "own keys":
            layers[4]["mixer"]["kv_from"] = 3
            layers[4]["mixer"].update({"dim": 96, "vdim": 96, "heads": 6, "kv_heads": 2})
            for name in ("q", "q.b", "rel", "sink", "o"):
                w["l4.mix." + name] = weights["l3.mix." + name]
        elif change == "sink":
            w["l4.mix.sink"] = weights["l4.mix.sink"] - 50.0
        elif change == "latent sink":
            w["l1.mix.sink"] = weights["l1.mix.sink"] - 50.0
        elif change == "query latent norm":
            w["l5.mix.dq.norm"] = weights["l5.mix.dq.norm"].flip(0)
        elif change == "latent norm":
            w["l1.mix.dkv.norm"] = weights["l1.mix.dkv.norm"].flip(0)
        elif change == "base":
            layers[5]["mixer"]["rot"]["base"] = 710.0
        elif change == "limit":
            layers[7]["mlp"]["expert"]["limit"] = 0.51
        elif change == "router scale":
            layers[2]["mlp"]["router"]["scale"] = 2.45
        elif change == "groups":
            layers[0]["mlp"]["router"]["groups"]["keep"] = 2
        elif change == "fewer experts":
            layers[3]["mlp"]["router"]["top"] = 3
        elif change == "values":
            w["l1.mix.uv"] = weights["l1.mix.uv"].flip(0)
        moved = float((plain.forward(other, w, tokens) - want).abs().max())
        if change == "nothing":
            assert moved == 0.0
        else:
            assert moved > 30 * error, (change, moved, error)


def test_greedy_generation_through_the_entry_point(tmp_path):
    import llm_b200
    folder = make_folder(tmp_path, "Q", torch.bfloat16)
    config, weights = plain.read_model(folder)
    prompts = [random_tokens(n, config["vocab"], 90 + n) for n in (5, 70, 23)]
    llm = llm_b200.LLM(str(folder), dtype="float32", device=DEV, context=256, batch=3)
    got = llm.generate(prompts, max_tokens=8, temperature=0.0, stop_tokens=[], repeat_penalty=1.0)
    for prompt, tokens in zip(prompts, got):
        assert tokens == plain.greedy(config, weights, prompt, 8)
    llm16 = llm_b200.LLM(str(folder), dtype="bfloat16", device=DEV, context=256, batch=3)
    for prompt, tokens in zip(prompts, llm16.generate(prompts, max_tokens=8, temperature=0.0, stop_tokens=[],
                                                      repeat_penalty=1.0)):
        sequence = list(prompt)
        for token in tokens:                                    # every token is a maximum of the plain logits up to rounding
            if not bool(_sure(config, weights, sequence, torch.bfloat16).all()):
                break                                           # an expert chosen by a hair: the plain model may go another way
            logits = plain.forward(config, weights, sequence)[-1]
            assert logits[token] >= logits.max() - 0.06 * float(logits.max() - logits.min())
            sequence.append(token)


def test_trace_replay_program(tmp_path):
    folder = make_folder(tmp_path, "P", torch.bfloat16)
    config, weights = plain.read_model(folder)
    a, b = random_tokens(40, config["vocab"], 1), random_tokens(9, config["vocab"], 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:30], "want": [0, 29]}, {"id": "b", "tokens": b[:8], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": [a[30]], "want": [0]}, {"id": "b", "tokens": [b[8]], "want": [0]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[31:], "want": [8]}], "end": ["a"]}]
    program = Path(__file__).resolve().parent.parent / "bin" / "trace_run"
    out = tmp_path / "out"
    result = subprocess.run([sys.executable, str(program), "--model", str(folder), "--dtype", "float32", "--out", str(out),
                             "--max-tokens", "128"], input="\n".join(json.dumps(s) for s in steps) + "\n",
                            capture_output=True, text=True, timeout=600)
    assert result.returncode == 0, result.stderr[-2000:]
    assert [line for line in result.stdout.splitlines() if line.startswith("done")] == ["done 0", "done 1", "done 2"]
    read = lambda n: torch.frombuffer(bytearray((out / f"{n}.f32").read_bytes()), dtype=torch.float32).view(-1, config["vocab"])
    wa, wb = plain.forward(config, weights, a), plain.forward(config, weights, b)
    _check_logits(read(0), wa[[0, 29]], torch.float32)
    _check_logits(read(1), torch.stack([wa[30], wb[8]]), torch.float32)
    _check_logits(read(2), wa[[39]], torch.float32)
