"""Duvozen on the GPU: every new kernel and kernel option beside its plain statement (also with weights and inputs
made so that one key, a sink, a tap or a lost state shows), and the model through the engine, the generation entry
point and the trace-replay program against the plain whole-sequence implementation, in 32-bit and in bfloat16."""
import json
import math
import subprocess
import sys
from pathlib import Path

import pytest
import torch

import plain_duvozen as plain
import plain_ops
from test_mefolorn_gpu import BATCHES, Batch, _close, only_generic
from tiny_duvozen import CONFIGS, make_folder, random_tokens

pytestmark = pytest.mark.gpu

PAGE = 64
DEV = "cuda:0"


def _ops():
    from llm_b200 import ops
    return ops


class off:
    """Kernel variants switched off while the block runs."""

    def __init__(self, *names):
        self.names = names

    def __enter__(self):
        from llm_b200.ops import tactics
        for n in self.names:
            tactics.disable(n)

    def __exit__(self, *_):
        from llm_b200.ops import tactics
        for n in self.names:
            tactics.enable(n)


# ----------------------------------------------------------------------------- norms on results, convolution of the stream

@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width", [36, 97, 128, 2048, 4100])
def test_layernorm(dtype, width):
    ops = _ops()
    gen = torch.Generator().manual_seed(width)
    x = (2.0 * torch.randn((9, width), generator=gen) + 5.0).to(DEV)               # a mean that matters
    gain = (1.0 + 0.3 * torch.randn(width, generator=gen)).to(DEV)
    rows = torch.tensor([8, 0, 3], dtype=torch.int32, device=DEV)
    _close(ops.layernorm(x, gain, 1e-3, dtype), plain_ops.layernorm(x, gain, 1e-3, dtype), dtype)
    _close(ops.layernorm(x, gain, 1e-3, dtype, rows=rows), plain_ops.layernorm(x, gain, 1e-3, dtype, rows=rows), dtype)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("case", [(36, 4), (97, 3), (128, 3), (256, 1), (2048, 2), (4096, 4), (132, 7), (64, 16), (40, 0)])
def test_input_conv(dtype, case):
    """Batches of unequal steps on shuffled slots; the state is a range of a wider row, and what lies beside it and
    the slots of no one stay as they were."""
    ops = _ops()
    width, K = case
    gen = torch.Generator().manual_seed(width + K)
    taps = torch.randn((K, width), generator=gen).to(DEV) if K else None
    for lengths, new in BATCHES + [([40, 1, 300], [17, 1, 33]), ([16, 15, 2], [16, 15, 2])]:
        batch = Batch(lengths, new, seed=2)
        x = torch.randn((batch.n_tokens, width), generator=gen).to(DEV)
        wide = torch.randn((len(lengths) + 2, 2, max(K - 1, 1), width), generator=gen).to(DEV)
        results = []
        for fn in (ops.input_conv, plain_ops.input_conv):
            held = wide.clone()
            out = torch.zeros((batch.n_tokens, width), dtype=dtype, device=DEV)
            fn(x, taps, held[:, 1] if K > 1 else None, batch.cu, batch.slots, out, max(new))
            results.append((out, held))
        torch.cuda.synchronize()
        _close(results[0][0], results[1][0], dtype, (case, lengths, "out"))
        assert torch.equal(results[0][1], results[1][1]), (case, lengths, "state")        # copies of rows: exact


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("case", [
    # width, taps, result rows a token, a row of its own behind them, norm
    (36, 4, 2, True, "layernorm"), (97, 3, 1, False, "layernorm"), (128, 3, 3, True, "rmsnorm"), (2048, 2, 8, True, "layernorm"),
    (4096, 4, 1, True, "layernorm"), (256, 1, 4, False, "rmsnorm"), (64, 0, 1, True, "layernorm"), (132, 16, 2, False, "layernorm")])
def test_output_norm_add_alone_and_with_the_next_input(dtype, case):
    ops = _ops()
    width, K, terms, extra, kind = case
    gen = torch.Generator().manual_seed(width + terms)
    for n in (1, 5, 33):
        x = torch.randn((n, width), generator=gen).to(DEV)
        y = (torch.randn((n * terms, width), generator=gen) + 2.0).to(DEV)
        more = torch.randn((n, width), generator=gen).to(DEV) if extra else None
        gain = (1.0 + 0.3 * torch.randn(width, generator=gen)).to(DEV)
        taps = torch.randn((K, width), generator=gen).to(DEV) if K else None
        wide = torch.randn((n + 2, 2, max(K - 1, 1), width), generator=gen).to(DEV)
        slots = torch.randperm(n + 2, generator=gen)[:n].to(torch.int32).to(DEV)
        for with_conv in (False, True):
            results = []
            for fn in (ops.output_norm_add_, plain_ops.output_norm_add_):
                stream, held = x.clone(), wide.clone()
                out = torch.zeros((n, width), dtype=dtype, device=DEV)
                conv = (taps, held[:, 0] if K > 1 else None, slots, out) if with_conv else None
                fn(stream, y, gain, 1e-3, kind, terms, extra=more, conv=conv)
                results.append((stream, held, out))
            torch.cuda.synchronize()
            _close(results[0][0], results[1][0], torch.float32, (case, n, "stream"))
            _close(results[0][1], results[1][1], torch.float32, (case, n, "state"))
            _close(results[0][2], results[1][2], dtype, (case, n, "input"))
        # the fused form is the two launches to the last bit
        one, two = x.clone(), x.clone()
        held_one, held_two = wide.clone(), wide.clone()
        out_one, out_two = (torch.zeros((n, width), dtype=dtype, device=DEV) for _ in range(2))
        ops.output_norm_add_(one, y, gain, 1e-3, kind, terms, extra=more, conv=(taps, held_one[:, 0] if K > 1 else None, slots, out_one))
        ops.output_norm_add_(two, y, gain, 1e-3, kind, terms, extra=more)
        cu = torch.arange(n + 1, dtype=torch.int32, device=DEV)
        ops.input_conv(two, taps, held_two[:, 0] if K > 1 else None, cu, slots, out_two, 1)
        assert torch.equal(one, two) and torch.equal(out_one, out_two) and torch.equal(held_one, held_two), (case, n)


def test_a_convolution_is_the_same_however_the_prompt_is_cut():
    ops = _ops()
    width, K, n = 128, 4, 70
    gen = torch.Generator().manual_seed(0)
    x, taps = torch.randn((n, width), generator=gen).to(DEV), torch.randn((K, width), generator=gen).to(DEV)

    def run(cuts):
        state, outs, at = torch.zeros((1, K - 1, width), device=DEV), [], 0
        for size in cuts:
            out = torch.zeros((size, width), device=DEV)
            cu = torch.tensor([0, size], dtype=torch.int32, device=DEV)
            ops.input_conv(x[at:at + size], taps, state, cu, torch.zeros(1, dtype=torch.int32, device=DEV), out, size)
            outs.append(out)
            at += size
        return torch.cat(outs), state

    whole, state = run([n])
    _close(whole, plain.input_conv(x.double().cpu(), taps.t().double().cpu()).to(DEV), torch.float32)
    assert torch.equal(state[0], x[-3:])
    for cuts in ([1] * n, [2] * 35, [1, 3, 66], [17, 16, 37], [69, 1], [5, 1, 1, 1, 62]):
        again, held = run(cuts)
        assert torch.equal(again, whole) and torch.equal(held, state), cuts


# ----------------------------------------------------------------------------- the forget-gated recurrence

def _recurrence_inputs(H, D, V, n, slots, dtype, seed):
    gen = torch.Generator().manual_seed(seed)
    width = (2 * H * D + H * V + 7) // 8 * 8 + 8
    proj = torch.randn((n, width), generator=gen).to(dtype).to(DEV)
    bias = (1.0 + 2.0 * torch.randn(H * D, generator=gen)).to(DEV)
    lower = (0.9 * torch.rand(H * D, generator=gen)).to(DEV)
    weight = (1.0 + 0.3 * torch.randn(V, generator=gen)).to(DEV)
    state = torch.randn((slots, H * D * V + 4), generator=gen).to(DEV)
    return proj, bias, lower, weight, state


def _recurrence(fn, proj, bias, lower, weight, state, batch, H, D, V, dtype, single=None, eps=1e-4):
    ops = _ops()
    n = batch.n_tokens
    work = torch.zeros((n, ops.forget_recurrence_work_width(H, D, V)), device=DEV)
    o = torch.zeros((n, H * V), device=DEV)
    mixed = torch.zeros((n, H * V + 9), dtype=dtype, device=DEV)
    fn(proj, bias, lower, state, batch.cu, batch.slots, weight, eps, work, o, mixed[:, 4:4 + H * V], H, D, V,
       single_tokens=all(k == 1 for k in batch.new) if single is None else single)
    return mixed


# heads, state rows, value size (rows around the lanes' multiples, columns around a block's)
RECURRENCE_CASES = [(3, 5, 7), (2, 33, 3), (4, 32, 48), (2, 72, 40), (1, 128, 128), (2, 130, 64), (1, 256, 130), (1, 20, 300),
                    (5, 64, 32), (1, 300, 16), (2, 128, 200)]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("case", RECURRENCE_CASES)
def test_forget_recurrence(dtype, case):
    ops = _ops()
    H, D, V = case
    for lengths, new in BATCHES + [([130, 64, 129, 5, 2], [130, 3, 129, 5, 1])]:
        batch = Batch(lengths, new, seed=1)
        proj, bias, lower, weight, state = _recurrence_inputs(H, D, V, batch.n_tokens, len(lengths) + 2, dtype, D + V)
        states = [state.clone(), state.clone()]
        got = _recurrence(ops.forget_recurrence, proj, bias, lower, weight, states[0], batch, H, D, V, dtype)
        want = _recurrence(plain_ops.forget_recurrence, proj, bias, lower, weight, states[1], batch, H, D, V, dtype)
        torch.cuda.synchronize()
        _close(got, want, dtype, (case, lengths, "out"))
        _close(states[0], states[1], torch.float32, (case, lengths, "state"))           # also the slots and columns that no one owns


@pytest.mark.parametrize("case", [(2, 12, 10), (1, 128, 128), (2, 100, 36)])
def test_forget_recurrence_carries_its_state_across_any_cut(case):
    """A sequence in one step, and the same cut into two (the second also token by token, in the launch of its own for
    steps of one token): the same results and states to the last bit in 32-bit."""
    ops = _ops()
    H, D, V = case
    n = 21
    proj, bias, lower, weight, state = _recurrence_inputs(H, D, V, n, 3, torch.float32, 9)
    state.zero_()
    whole = state.clone()
    args = (bias, lower, weight)
    want = _recurrence(ops.forget_recurrence, proj, *args, whole, Batch([n], [n]), H, D, V, torch.float32)
    for cut in range(1, n):
        held = state.clone()
        head = _recurrence(ops.forget_recurrence, proj[:cut], *args, held, Batch([cut], [cut]), H, D, V, torch.float32)
        if cut % 2:
            tail = _recurrence(ops.forget_recurrence, proj[cut:], *args, held, Batch([n], [n - cut]), H, D, V, torch.float32)
        else:
            tail = torch.cat([_recurrence(ops.forget_recurrence, proj[t:t + 1], *args, held, Batch([t + 1], [1]), H, D, V, torch.float32)
                              for t in range(cut, n)])
        assert torch.equal(torch.cat([head, tail]), want), cut
        assert torch.equal(held, whole), cut


def test_forget_recurrence_reads_back_what_it_stored_hundreds_of_tokens_ago():
    """Token 0 writes its value under state row 0 (forgetting all of it), whose gate then stays at one; the 400 tokens
    between write under other rows, and the last token reads row 0 only: it gets token 0's value back. With the state
    lost on the way it does not."""
    ops = _ops()
    H, D, V, n, big = 1, 32, 8, 402, 40.0
    gen = torch.Generator().manual_seed(2)
    proj = torch.zeros((n, 2 * D + V), device=DEV)
    proj[:, 1:D] = torch.rand((n, D - 1), generator=gen).to(DEV)                       # q away from row 0
    proj[:, D + 1:2 * D] = torch.randn((n, D - 1), generator=gen).to(DEV)              # f of the other rows
    proj[:, D] = big                                                                   # row 0: sigmoid = 1, kept
    proj[0, D] = -big                                                                  # token 0: forgotten and written
    proj[:, 2 * D:] = 3.0 * torch.randn((n, V), generator=gen).to(DEV)
    proj[-1, :D] = 0.0
    proj[-1, 0] = big                                                                  # the last token reads row 0
    bias, lower, weight = torch.zeros(D, device=DEV), torch.zeros(D, device=DEV), torch.ones(V, device=DEV)
    stored = proj[0, 2 * D:]

    def run(lose_at=None):
        state, outs = torch.zeros((1, D * V), device=DEV), []
        for lo, hi in ((0, 150), (150, 151), (151, 300), (300, n)):
            if lose_at == lo:
                state.zero_()
            outs.append(_recurrence(ops.forget_recurrence, proj[lo:hi], bias, lower, weight, state, Batch([hi], [hi - lo]), H, D, V,
                                    torch.float32, eps=1e-12)[:, 4:4 + V])
        return torch.cat(outs)[-1]

    want = stored / torch.sqrt((stored * stored).mean())
    assert torch.allclose(run(), want, atol=1e-4)
    assert float((run(lose_at=300) - want).abs().max()) > 0.3


# ----------------------------------------------------------------------------- latent attention

@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("case", [
    # heads, unrotated, rotated part, latent, rotated of it, interleaved
    (3, 5, 6, 11, 6, True), (2, 9, 2, 20, 2, True), (4, 32, 16, 80, 8, True), (2, 64, 64, 128, 64, False), (20, 16, 8, 40, 4, False),
    (1, 128, 64, 512, 64, True), (2, 16, 8, 24, 0, True)])
def test_latent_write(dtype, case):
    ops = _ops()
    H, D, R, C, n_rot, interleaved = case
    gen = torch.Generator().manual_seed(D + C)
    gain = (1.0 + 0.3 * torch.randn(C, generator=gen)).to(DEV)
    table = None
    if n_rot:
        angle = torch.arange(400, dtype=torch.float64)[:, None] * torch.rand(n_rot // 2, generator=gen, dtype=torch.float64)
        table = (1.2 * torch.cat([angle.cos(), angle.sin()], dim=1)).float().to(DEV)
    for lengths, new in BATCHES:
        batch = Batch(lengths, new, seed=len(lengths))
        u = torch.randn((batch.n_tokens, H * (D + R) + C + R + 8), generator=gen).to(dtype).to(DEV)
        for form in ("queries", "in place", "shared cache"):
            results = []
            for fn in (ops.latent_write, plain_ops.latent_write):
                cache, _ = batch.caches(1, C + R, 0, dtype, seed=5)
                mine = u.clone()
                queries = torch.zeros((batch.n_tokens, H * (C + R)), dtype=dtype, device=DEV) if form != "in place" else None
                dense = torch.zeros((batch.n_tokens, C + R), dtype=dtype, device=DEV) if form == "in place" else None
                fn(mine, H, D, R, C, gain, 1e-3, table, interleaved, batch.tok_pos, batch.tok_seq, batch.table, batch.width, cache,
                   queries=queries, dense=dense, write_cache=form != "shared cache")
                results.append((mine, cache, queries, dense))
            torch.cuda.synchronize()
            for got, want, what in zip(results[0], results[1], ("projection", "cache", "queries", "dense rows")):
                if got is not None:
                    _close(got, want, dtype, (case, lengths, form, what))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16, "cuda cores"])
@pytest.mark.parametrize("case", [
    # heads, outputs, inner size, columns between heads of x and of the result
    (3, 11, 5, 11, 17), (2, 128, 64, 128, 192), (4, 80, 32, 48, 96), (5, 24, 40, 40, 24), (2, 512, 128, 192, 576), (1, 70, 520, 520, 70),
    (2, 64, 72, 72, 64)])
def test_head_products(dtype, case):
    ops = _ops()
    plainly = dtype == "cuda cores"
    dtype = torch.bfloat16 if plainly else dtype
    H, N, K, x_head, out_head = case
    gen = torch.Generator().manual_seed(N + K)
    w = (torch.randn((H, N, K), generator=gen) / math.sqrt(K)).to(dtype).to(DEV)
    for n in (1, 7, 33, 130):
        x = torch.randn((n, H * x_head + 8), generator=gen).to(dtype).to(DEV)
        got, want = (torch.full((n, H * out_head + 8), 7.0, dtype=dtype, device=DEV) for _ in range(2))
        with off(*(("head_products_mma",) if plainly else ())):
            ops.head_products(x, x_head, w, got, out_head)
        plain_ops.head_products(x, x_head, w, want, out_head)
        torch.cuda.synchronize()
        _close(got, want, dtype, (case, n))
        beside = torch.ones(got.shape[1], dtype=torch.bool)
        for h in range(H):
            beside[h * out_head:h * out_head + N] = False
        assert bool((got[:, beside.to(DEV)] == 7.0).all())


# heads, latent, rotated part
LATENT_CASES = [(3, 11, 6), (4, 80, 16), (2, 128, 64), (20, 40, 8), (40, 64, 32), (16, 256, 64), (33, 512, 64), (1, 512, 128), (70, 96, 32)]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16, "tiles", "generic"])
@pytest.mark.parametrize("case", LATENT_CASES)
def test_latent_attention(dtype, case):
    ops = _ops()
    without = {"tiles": ("latent_decode_tc",), "generic": ("latent_decode_tc", "latent_tiles")}.get(dtype, ())
    dtype = torch.bfloat16 if without else dtype
    H, C, R = case
    for lengths, new in BATCHES + [([400, 64, 129], [3, 3, 129]), ([700, 1, 64, 65, 300], [1] * 5)]:
        batch = Batch(lengths, new, seed=3 + len(lengths))
        gen = torch.Generator().manual_seed(C)
        q = (2.0 * torch.randn((batch.n_tokens, H * (C + R)), generator=gen)).to(dtype).to(DEV)
        cache, _ = batch.caches(1, C + R, 0, dtype, seed=4)
        results = []
        for fn in (ops.latent_attention, plain_ops.latent_attention):
            out = torch.zeros((batch.n_tokens, H * C), dtype=dtype, device=DEV)
            with off(*without):
                fn(q, cache, batch.table, batch.width, batch.tok_pos, batch.tok_seq, H, C, R, (C + R) ** -0.5, out, **batch.extra())
            results.append(out)
        torch.cuda.synchronize()
        ops.check_device_status()
        _close(results[0], results[1], dtype, (case, lengths))


def test_latent_decode_with_scores_that_grow():
    """Scores that rise along the sequence, in some heads and not in others: the exponents' references move again and
    again, each head's at places of its own."""
    ops = _ops()
    for H, C, R, n in ((20, 64, 8, 700), (32, 512, 64, 330), (7, 256, 40, 129)):
        batch = Batch([n, 64, 1], [1, 1, 1], seed=2)
        cache, _ = batch.caches(1, C + R, 0, torch.bfloat16, seed=3, std=0.3)
        for p in range(n):
            page, row = batch.place(0, p)
            cache[page, 0, row, :4] = torch.tensor([p / 20.0, -p / 30.0, (p % 97) / 5.0, 1.0])
        q = torch.zeros((3, H * (C + R)), dtype=torch.bfloat16, device=DEV)
        heads = q.view(3, H, C + R)
        for h in range(H):
            heads[:, h, h % 4] = 1.0 + h / 8.0
        got, want = (torch.zeros((3, H * C), dtype=torch.bfloat16, device=DEV) for _ in range(2))
        for fn, out in ((ops.latent_attention, got), (plain_ops.latent_attention, want)):
            fn(q, cache, batch.table, batch.width, batch.tok_pos, batch.tok_seq, H, C, R, 1.0, out, **batch.extra())
        torch.cuda.synchronize()
        ops.check_device_status()
        _close(got, want, torch.bfloat16, (H, C))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("decode", [False, True])
def test_latent_attention_planted_keys(dtype, decode):
    """One row stands out by its rotated part alone (its latent part scores nothing) and the result is its latent part:
    far back, at page borders, the newest, and one beyond the query, which must not be seen."""
    ops = _ops()
    for H, C in ((20, 72), (20, 64), (3, 128)):
        _latent_planted(ops, dtype, decode, H, C)


def _latent_planted(ops, dtype, decode, H, C):
    R, length = 8, 331
    batch = Batch([length, 40], [1, 1] if decode else [length, 40], seed=11)
    for planted in (0, 1, 31, 32, 63, 64, 255, 256, length - 2, length - 1):
        cache, _ = batch.caches(1, C + R, 0, dtype, seed=6, std=0.1)
        page, row = batch.place(0, planted)
        cache[page, 0, row] = 0.0
        cache[page, 0, row, C:] = 3.0
        cache[page, 0, row, :2] = torch.tensor([5.0, -7.0])
        gen = torch.Generator().manual_seed(4)
        q = (0.1 * torch.randn((batch.n_tokens, H * (C + R)), generator=gen)).to(dtype).to(DEV)
        at = [0] if decode else sorted({planted, length - 1} | ({planted - 1} if planted else set()))
        for t in at:
            q[t] = 0.0
            q[t].view(H, C + R)[:, C:] = 1.0                          # score 24 x 0.8 with the planted row, about 0 with the others
        out = torch.zeros((batch.n_tokens, H * C), dtype=dtype, device=DEV)
        ops.latent_attention(q, cache, batch.table, batch.width, batch.tok_pos, batch.tok_seq, H, C, R, 0.8, out, **batch.extra())
        for t in at:
            sees = decode or t >= planted
            heads = out[t].view(H, C)
            if sees:
                assert torch.allclose(heads[:, :2].float(), torch.tensor([5.0, -7.0], device=DEV).expand(H, 2), atol=0.05), (planted, t)
            else:
                assert float(heads.float().abs().max()) < 1.0, (planted, t)


# heads, unrotated, rotated part, value size, latent
EXPANDED_CASES = [(2, 64, 64, 64, 128), (3, 128, 64, 128, 96), (2, 64, 32, 128, 40), (2, 128, 8, 64, 64), (1, 64, 24, 64, 512), (5, 128, 64, 128, 512)]


@pytest.mark.parametrize("case", EXPANDED_CASES)
def test_latent_prefill_with_keys_and_values_formed(case):
    ops = _ops()
    H, D, R, V, C = case
    for new in ([70, 5, 130, 64], [1], [300, 257, 128, 1], [600], [256, 129]):
        batch = Batch(new, new, seed=len(new))
        n = batch.n_tokens
        gen = torch.Generator().manual_seed(D + R + n)
        bf16 = torch.bfloat16
        proj = (2.0 * torch.randn((n, H * (D + R) + C + R), generator=gen)).to(bf16).to(DEV)
        if proj.shape[1] % 8:
            proj = torch.cat([proj, torch.zeros((n, 8 - proj.shape[1] % 8), dtype=bf16, device=DEV)], dim=1).contiguous()
        kv = torch.randn((n, H * (D + V)), generator=gen).to(bf16).to(DEV)
        dense = torch.randn((n, C + R), generator=gen).to(bf16).to(DEV)
        got, want = (torch.zeros((n, H * V), dtype=bf16, device=DEV) for _ in range(2))
        args = (proj, kv, dense, H, D, R, V, C, (D + R) ** -0.5)
        ops.latent_prefill(*args, got, batch.cu, max(new), batch.order)
        plain_ops.latent_prefill(*args, want, batch.cu.cpu(), max(new))
        torch.cuda.synchronize()
        ops.check_device_status()
        _close(got, want, bf16, (case, new))


def test_latent_prefill_planted_keys_and_growing_scores():
    """Far keys, keys at block borders and the diagonal, one by the shared rotated part alone; and scores that grow along
    the sequence, so that the exponent's reference moves again and again."""
    ops = _ops()
    H, D, R, V, C, n = 2, 64, 16, 64, 24, 520
    bf16 = torch.bfloat16
    batch = Batch([n], [n])
    gen = torch.Generator().manual_seed(1)
    for planted in (0, 63, 64, 127, 128, 255, 256, 511, 519):
        proj = (0.1 * torch.randn((n, H * (D + R) + C + R), generator=gen)).to(bf16).to(DEV)
        kv = (0.1 * torch.randn((n, H * (D + V)), generator=gen)).to(bf16).to(DEV)
        dense = torch.zeros((n, C + R), dtype=bf16, device=DEV)
        dense[planted, C:] = 3.0
        kv.view(n, H, D + V)[planted, :, D:D + 2] = torch.tensor([5.0, -7.0], dtype=bf16, device=DEV)
        q = proj[:, :H * (D + R)].view(n, H, D + R)
        q[:, :, :D] = 0.0
        q[:, :, D:] = 1.0
        out = torch.zeros((n, H * V), dtype=bf16, device=DEV)
        ops.latent_prefill(proj, kv, dense, H, D, R, V, C, 0.5, out, batch.cu, n, batch.order)
        heads = out.view(n, H, V).float()
        assert torch.allclose(heads[planted:, :, :2], torch.tensor([5.0, -7.0], device=DEV).expand(n - planted, H, 2), atol=0.06), planted
        if planted:
            assert float(heads[:planted].abs().max()) < 1.0
    proj = torch.ones((n, H * (D + R) + C + R), dtype=bf16, device=DEV)
    kv = (torch.arange(n, device=DEV)[:, None] / 40.0 + torch.randn((n, H * (D + V)), generator=gen).to(DEV) * 0.3).to(bf16)
    dense = torch.zeros((n, C + R), dtype=bf16, device=DEV)
    got, want = (torch.zeros((n, H * V), dtype=bf16, device=DEV) for _ in range(2))
    ops.latent_prefill(proj, kv, dense, H, D, R, V, C, 0.25, got, batch.cu, n, batch.order)
    plain_ops.latent_prefill(proj, kv, dense, H, D, R, V, C, 0.25, want, batch.cu.cpu(), n)
    _close(got, want, bf16)


# ----------------------------------------------------------------------------- attention with learned sinks

@pytest.mark.parametrize("which", ["first", "mma", "generic", "32-bit"])
@pytest.mark.parametrize("case", [(8, 2, 64), (4, 1, 128), (6, 2, 96), (2, 2, 32)])
def test_attention_with_learned_sinks_on_every_kernel(which, case):
    """Sinks far below, among and far above the scores; whole prompts, later portions and decode steps; the tensor-core
    kernels, those one rank below, and the one for any sizes."""
    ops = _ops()
    heads, groups, dim = case
    dtype = torch.float32 if which == "32-bit" else torch.bfloat16
    gen = torch.Generator().manual_seed(dim)
    sinks = torch.linspace(-30.0, 40.0, heads).to(DEV)
    for lengths, new in BATCHES + [([700, 64, 129], [700, 3, 129]), ([1500, 1, 64, 65, 700], [1] * 5)]:
        batch = Batch(lengths, new, seed=3 + len(lengths))
        q = (2.0 * torch.randn((batch.n_tokens, heads * dim), generator=gen)).to(dtype).to(DEV)
        k_cache, v_cache = batch.caches(groups, dim, dim, dtype, seed=3)
        results = []
        for fn in (ops.attention, plain_ops.attention):
            out = torch.zeros((batch.n_tokens, heads * dim), dtype=dtype, device=DEV)
            with only_generic(which == "generic"), off(*(("attention_prefill_tc",) if which in ("mma", "generic") else ())):
                fn(q, k_cache, v_cache, batch.table, batch.width, batch.tok_pos, batch.tok_seq, heads, groups, dim, dim ** -0.5, 0,
                   out=out, sinks=sinks, **batch.extra())
            results.append(out)
        torch.cuda.synchronize()
        for h in range(heads):                               # head by head: a large sink makes a head's results tiny
            part = slice(h * dim, (h + 1) * dim)
            got, want = results[0][:, part].float(), results[1][:, part].float()
            top = float(want.abs().max()) + 1e-20
            assert float((got - want).abs().max()) <= (5e-5 if dtype == torch.float32 else 0.03) * top, (case, lengths, h)


def test_the_sink_s_share():
    """Queries of zero: every key has the weight 1 / (n + e^sink)."""
    ops = _ops()
    batch = Batch([100], [100])
    sink = math.log(7.0)
    for dtype, dim in ((torch.float32, 16), (torch.bfloat16, 64), (torch.bfloat16, 96)):
        q = torch.zeros((100, 2 * dim), dtype=dtype, device=DEV)
        k, v = batch.caches(1, dim, dim, dtype)
        v.fill_(1.0)
        out = torch.zeros((100, 2 * dim), dtype=dtype, device=DEV)
        ops.attention(q, k, v, batch.table, batch.width, batch.tok_pos, batch.tok_seq, 2, 1, dim, 0.3, 0, out=out,
                      sinks=torch.full((2,), sink, device=DEV), **batch.extra())
        n = torch.arange(1, 101, device=DEV, dtype=torch.float32)[:, None]
        assert torch.allclose(out.float(), (n / (n + 7.0)).expand_as(out), atol=1e-5 if dtype == torch.float32 else 6e-3)


# ----------------------------------------------------------------------------- feed-forward

@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("m,width,ff", [(1, 64, 32), (8, 256, 160), (70, 128, 96), (300, 512, 512), (16, 4096, 256), (5, 36, 18)])
def test_gelu_in_the_gated_epilogue_and_alone(dtype, m, width, ff):
    ops = _ops()
    gen = torch.Generator().manual_seed(m + ff)
    x = torch.randn((m, width), generator=gen).to(dtype).to(DEV)
    gate, up = (2.0 * torch.randn((ff, width), generator=gen) / math.sqrt(width) for _ in range(2))
    gate_up = (torch.cat([gate, up]).to(dtype).to(DEV))
    product = (x.float() @ gate_up.float().T).to(dtype)
    for gelu in (False, True):
        _close(ops.swiglu(product, gelu=gelu), plain_ops.swiglu(product, gelu=gelu), dtype, (m, gelu))
    if ops.glu_fusable(2 * ff, width, dtype):
        w = torch.stack([gate.view(-1, 16, width), up.view(-1, 16, width)], dim=1).reshape(2 * ff, width).to(dtype).to(DEV).contiguous()
        for glu in (True, "gelu"):
            _close(ops.linear(x, w, glu=glu), plain_ops.linear(x, w, glu=glu), dtype, (m, glu))


def test_gelu_far_from_zero():
    ops = _ops()
    z = torch.tensor([-1e4, -30.0, -5.0, -0.5, 0.0, 0.5, 5.0, 30.0, 1e4], device=DEV)
    row = torch.cat([z, torch.ones_like(z)])[None].contiguous()
    want = 0.5 * z.double() * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z.double() + 0.044715 * z.double() ** 3)))
    assert torch.allclose(ops.swiglu(row, gelu=True)[0].double(), want, atol=1e-5, rtol=1e-6)


def _experts(fn, h, router, w_up, w_down, top, on_input=True):
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
    fn(h, router, None, w_up, w_down, top, ids, weights, order, plan, act, y, gathered, scoring=2, weight_on_input=on_input)
    return y, ids, weights


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("case", [
    # width, expert width, experts, chosen
    (40, 12, 5, 3), (128, 64, 8, 2), (128, 96, 4, 1), (32, 16, 1, 1), (256, 128, 16, 4), (136, 40, 7, 7), (320, 104, 12, 4), (64, 32, 40, 20)])
def test_experts_with_sigmoid_scores_and_the_weight_on_their_input(dtype, case):
    ops = _ops()
    hidden, F, E, top = case
    gen = torch.Generator().manual_seed(hidden + E)
    router = (2.0 * torch.randn((E, hidden), generator=gen) / hidden ** 0.5).to(DEV)
    w_up = (2.0 * torch.randn((E, 2 * F, hidden), generator=gen) / hidden ** 0.5).to(dtype).to(DEV)
    w_down = (torch.randn((E, hidden, F), generator=gen) / F ** 0.5).to(dtype).to(DEV)
    for n in (1, 7, 70, 600, 48 * E) if E <= 16 else (1, 70):      # few rows an expert, and enough for the tiles of 128 rows
        h = torch.randn((n, hidden), generator=gen).to(dtype).to(DEV)
        for on_input in (True, False):
            got, got_ids, got_weights = _experts(ops.routed_experts, h, router, w_up, w_down, top, on_input)
            want, want_ids, want_weights = _experts(plain_ops.routed_experts, h, router, w_up, w_down, top, on_input)
            torch.cuda.synchronize()
            same = (got_ids.view(n, top) == want_ids.view(n, top)).all(dim=1)      # a close call may fall either way
            assert int(same.sum()) >= 0.95 * n, (case, n)
            rows = same.repeat_interleave(top)
            assert torch.allclose(got_weights[rows], want_weights[rows], atol=2e-6, rtol=2e-5)
            _close(got[rows], want[rows], dtype, (case, n, on_input))
    # the same rows whatever else is in the batch
    alone, _, _ = _experts(ops.routed_experts, h[2:3], router, w_up, w_down, top)
    among, _, _ = _experts(ops.routed_experts, h[:5], router, w_up, w_down, top)
    assert torch.equal(alone, among.view(5, top, hidden)[2])


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


MARGIN = 0.01           # of sigmoid scores: what bfloat16 rounding of the router's input reaches


def _sure(config, weights, tokens, dtype):
    """Per position: True up to the first position at which a routed layer chose by less than a rounding's reach (another
    expert there changes what every later position reads from the states and the cache)."""
    if dtype == torch.float32:
        return torch.ones(len(tokens), dtype=torch.bool)
    return torch.cummin(plain.closest_call(config, weights, tokens), dim=0).values > MARGIN


def test_every_layer_agrees_with_plain(tmp_path):
    """The residual stream after each layer in 32-bit (a model of the first k layers, for every k, whose
    last norm has a weight of one, and its last layer also without feed-forward)."""
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
@pytest.mark.parametrize("which", ["P", "Q", "R"])
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
def test_dense_feed_forwards_in_both_dtypes(tmp_path, dtype):
    """All layers with dense feed-forwards: no choice of experts, so every position is compared in bfloat16 too, in one
    step (prompts from their first token: keys and values formed), in portions (the cached rows), and decoded."""
    from llm_b200.engine import Entry

    def dense(config):
        for i, layer in enumerate(config["layers"]):
            layer["mlp"] = {"kind": "dense", "ff": 96 + 32 * (i % 3)}
    config, weights, engine = _setup(tmp_path, "Q", dtype, dense)
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


@pytest.mark.parametrize("heads", [8, 24, 40])
@pytest.mark.parametrize("rank", [64, 128, 256, 512])
def test_decode_steps_whose_kernels_follow_closely(tmp_path, heads, rank):
    """A model of latent layers alone, decoded as a batch through captured steps: every kernel starts while the one in
    front of it ends, so a load in front of the wait for it would read the step before."""
    from llm_b200.engine import Entry
    from tiny_duvozen import _latent

    def latent_only(config):
        config["layers"] = [{"type": "latent_attention", "mlp": None,
                             "mixer": _latent(heads, 64, 64, 24, rank, 10000.0, (4.0, 100, 8.0, 1.0))}] * 2
    config, weights, engine = _setup(tmp_path, "Q", torch.bfloat16, latent_only)
    lengths = (129, 190, 40)
    seqs = [random_tokens(n + 12, config["vocab"], n) for n in lengths]
    expected = [plain.forward(config, weights, s) for s in seqs]
    slots = engine.acquire(3)
    engine.step([Entry(s, q[:n], []) for s, q, n in zip(slots, seqs, lengths)])
    for k in range(12):
        logits = engine.step([Entry(s, [q[n + k]], [0]) for s, q, n in zip(slots, seqs, lengths)])
        _check_logits(logits, torch.stack([e[n + k] for e, n in zip(expected, lengths)]), torch.bfloat16, k)
    assert engine.graph_replays > 5


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_long_decoding_passes_page_edges(tmp_path, dtype):
    """One token a step from the first on, 300 steps: pages fill and follow each other, the recurrences' states and the
    stream's last rows are carried 300 times, and steps are replayed from graphs."""
    from llm_b200.engine import Entry

    def dense(config):
        for layer in config["layers"]:
            layer["mlp"] = {"kind": "dense", "ff": 96}
    config, weights, engine = _setup(tmp_path, "Q", dtype, dense)
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
            engine.step([Entry(e, [seqs[0][t]], [])])
        cut = engine.step([Entry(e, seqs[0][30:], [49 - 30])])
        assert torch.equal(alone[0], cut[0]), which


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_passes_walked_from_their_record_agree_with_plain_passes(tmp_path, dtype):
    """The same shape of step five times on other slots, pages and states: the first pass runs through the parts,
    the second is recorded, the later ones are walked natively from the record; a mixed step and a later portion of a
    prompt (another form of the latent attention than its first) likewise."""
    from llm_b200.engine import Entry
    config, weights, engine = _setup(tmp_path, "Q", dtype)
    for again in range(5):
        seqs = [random_tokens(n, config["vocab"], 100 * again + n) for n in (90, 33)]
        sure = [_sure(config, weights, s, dtype) for s in seqs]
        slots = engine.acquire(2)
        want = [plain.forward(config, weights, s) for s in seqs]
        logits = engine.step([Entry(slots[0], seqs[0][:40], [0, 39]), Entry(slots[1], seqs[1][:15], [14])])
        _check_logits(logits, torch.stack([want[0][0], want[0][39], want[1][14]]), dtype, ("first", again),
                      torch.stack([sure[0][0], sure[0][39], sure[1][14]]))
        logits = engine.step([Entry(slots[0], seqs[0][40:80], [0, 39]), Entry(slots[1], seqs[1][15:30], [14])])
        _check_logits(logits, torch.stack([want[0][40], want[0][79], want[1][29]]), dtype, ("later", again),
                      torch.stack([sure[0][40], sure[0][79], sure[1][29]]))
        mixed = engine.step([Entry(slots[0], seqs[0][80:], [9]), Entry(slots[1], [seqs[1][30]], [0])])
        _check_logits(mixed, torch.stack([want[0][89], want[1][30]]), dtype, ("mixed", again), torch.stack([sure[0][89], sure[1][30]]))
        engine.release(slots)
    assert engine.records_run >= 8


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
    for change in ("taps", "no convolution", "lower bound", "gate bias", "head norm", "bands", "rotated part", "latent norm", "sink",
                   "gate", "query norm", "shared expert", "fewer experts", "logit scale", "values", "nothing"):
        other, w = json.loads(json.dumps(config)), dict(weights)
        if change == "taps":
            w["l3.canon1"] = weights["l3.canon1"].flip(1)
        elif change == "no convolution":
            w["l4.canon2"] = weights["l4.canon2"] * 0.0
        elif change == "lower bound":
            w["l2.mix.lower"] = weights["l2.mix.lower"] * 0.0
        elif change == "gate bias":
            w["l2.mix.f.b"] = weights["l2.mix.f.b"] * 0.0
        elif change == "head norm":
            w["l5.mix.norm"] = weights["l5.mix.norm"].flip(0)
        elif change == "bands":
            del other["layers"][0]["mixer"]["rot"]["scaling"]
        elif change == "rotated part":
            other["layers"][1]["mixer"]["rot"]["dims"] = 64
        elif change == "latent norm":
            w["l3.mix.dkv.norm"] = weights["l3.mix.dkv.norm"].flip(0)
        elif change == "sink":
            w["l4.mix.sink"] = weights["l4.mix.sink"] - 50.0
        elif change == "gate":
            w["l1.mix.g"] = weights["l1.mix.g"] * 0.0
        elif change == "query norm":
            w["l1.mix.q.norm"] = weights["l1.mix.q.norm"].flip(0)
        elif change == "shared expert":
            w["l2.mlp.shared.down"] = weights["l2.mlp.shared.down"] * 0.0
        elif change == "fewer experts":
            other["layers"][4]["mlp"]["router"]["top"] = 3
        elif change == "logit scale":
            other["logit_scale"] = 1.51
        elif change == "values":
            w["l6.mix.uv"] = weights["l6.mix.uv"].flip(0)
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
