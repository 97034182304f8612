"""Randomly drawn tiny Duvozen configurations (seeded): any order of the three mixers, widths that the 16-byte paths
take and widths they do not, head, latent and value sizes that the tensor-core kernels take and sizes no tile takes,
groups of 1 to 8 heads, rotated parts shorter than a head, scaled frequencies or not, states with fewer and more rows
than columns, one to eight taps, one to all of 1 to 40 experts with and without a shared one, dense feed-forwards, layers
without. Each runs a batch of unequal prompts, a later portion of one of them, and then decodes, shorter requests
leaving earlier, in 32-bit and in bfloat16, against the plain implementation."""
import math
import random

import pytest
import torch

import plain_duvozen as plain
from test_zemozen_random_gpu import close
from tiny_duvozen import random_weights, write_folder

pytestmark = pytest.mark.gpu

DEV = "cuda:0"
MARGIN = 0.02           # of sigmoid scores: what bfloat16 rounding of the router's input reaches


def draw_config(rng) -> dict:
    width = rng.choice([36, 48, 64, 100, 136, 160, 260, 320])

    def rotation(unit):
        return {"base": rng.choice([100.0, 10000.0, 1e6]), "dims": max(2, rng.choice([unit, unit, unit // 2]) // 2 * 2)}

    def attention():
        kv = rng.choice([1, 2, 3, 4])
        dim = rng.choice([8, 10, 16, 24, 32, 48, 64, 64, 96, 128])
        return {"heads": kv * rng.choice([1, 2, 3, 8] if kv < 3 else [1, 2]), "kv_heads": kv, "dim": dim,
                "vdim": rng.choice([dim, dim, dim, 8, 20, 72]), "scale": rng.choice([1.0 / math.sqrt(dim), 0.13]), "rot": rotation(dim)}

    def latent():
        dim, rot_dim = rng.choice([8, 10, 16, 32, 64, 64, 128]), rng.choice([2, 4, 8, 16, 24, 32, 64])
        rot = {"base": rng.choice([1000.0, 10000.0, 5e5]), "dims": rot_dim}
        if rng.random() < 0.7:
            rot["scaling"] = {"factor": rng.choice([2.0, 5.0, 20.0]), "original": rng.choice([64, 500, 2048]),
                              "fast": rng.choice([8.0, 24.0]), "slow": rng.choice([0.5, 2.0])}
        return {"heads": rng.choice([1, 2, 5, 8, 17, 24, 40]), "dim": dim, "rot_dim": rot_dim, "vdim": rng.choice([dim, 8, 20, 64, 128]),
                "kv_rank": rng.choice([12, 24, 40, 64, 64, 96, 128, 160, 256, 300]), "rot": rot,
                "scale": rng.choice([1.0 / math.sqrt(dim + rot_dim), 0.09])}

    def recurrence():
        return {"heads": rng.choice([1, 2, 3, 6]), "dim": rng.choice([4, 7, 16, 33, 40, 64, 100, 128, 140]),
                "vdim": rng.choice([4, 6, 16, 36, 64, 130])}

    def feed_forward():
        kind = rng.random()
        if kind < 0.12:
            return None
        if kind < 0.5:
            return {"kind": "dense", "ff": rng.choice([8, 20, 64, 72, 160])}
        experts = rng.choice([1, 2, 3, 8, 16, 40])
        out = {"kind": "moe", "router": {"experts": experts, "top": min(experts, rng.choice([1, 2, 4, experts if experts <= 8 else 6]))},
               "expert": {"ff": rng.choice([8, 20, 32, 64, 72, 96])}}
        if rng.random() < 0.7:
            out["shared"] = {"ff": rng.choice([8, 36, 64, 128])}
        return out

    kinds = [("attention", attention), ("latent_attention", latent), ("hgrn2", recurrence)]
    layers = []
    for _ in range(rng.choice([1, 2, 3, 4, 5])):
        kind, mixer = rng.choice(kinds)
        layers.append({"type": kind, "mixer": mixer(), "mlp": feed_forward()})
    return {"architecture": "Duvozen", "vocab": rng.choice([61, 128, 300, 1000]), "width": width,
            "norm": {"eps": rng.choice([1e-5, 1e-6, 1e-3])}, "embedding": {"scale": rng.choice([0.3, 1.0, 4.0])},
            "logit_scale": rng.choice([0.5, 1.0, 3.0]), "canon": {"taps": rng.choice([1, 2, 3, 4, 5, 8])}, "layers": layers}


@pytest.mark.parametrize("case", range(200, 236))
def test_random_configuration(tmp_path, case):
    from llm_b200.engine import Engine, Entry, load_model
    rng = random.Random(52100 + case)
    raw = draw_config(rng)
    folder = write_folder(tmp_path / "model", raw, random_weights(raw, 700 + case))
    config, weights = plain.read_model(folder)
    lengths = [rng.choice([1, 3, 17, 64, 65, 127, 128, 129, 200, 300]) for _ in range(rng.choice([1, 2, 3, 5]))]
    later = rng.choice([2, 5, 40])                                  # tokens the first sequence brings in a portion of its own
    extra = [rng.choice([1, 2, 8, 33]) for _ in lengths]
    gen = torch.Generator().manual_seed(case)
    seqs = [torch.randint(0, raw["vocab"], (n + (later if b == 0 else 0) + e,), generator=gen).tolist()
            for b, (n, e) in enumerate(zip(lengths, extra))]
    expected, margins = [], []
    for s in seqs:
        per_layer = []
        expected.append(plain.forward(config, weights, s, margins=per_layer))
        # bfloat16: from the first position on at which an expert was chosen by less than rounding reaches, a sequence is
        # not compared (another expert there changes what every later position reads from the state and the cache)
        margins.append(torch.cummin(torch.stack(per_layer).min(dim=0).values, dim=0).values > MARGIN if per_layer
                       else torch.ones(len(s), dtype=torch.bool))
    for dtype in (torch.float32, torch.bfloat16):
        sure = [None if dtype == torch.float32 else m for m in margins]
        engine = Engine(load_model(folder, dtype, DEV), max_tokens=64 * 8 * len(seqs), max_slots=len(seqs))

        def check(got, b, first, count, what):
            assert close(got, expected[b][first:first + count], dtype, None if sure[b] is None else sure[b][first:first + count]), \
                (raw, dtype, what, b, first, lengths)
        slots = engine.acquire(len(seqs))
        logits = engine.step([Entry(s, q[:n], list(range(n))) for s, q, n in zip(slots, seqs, lengths)])
        at = 0
        for b, n in enumerate(lengths):
            check(logits[at:at + n], b, 0, n, "prompt")
            at += n
        starts = list(lengths)
        check(engine.step([Entry(slots[0], seqs[0][starts[0]:starts[0] + later], list(range(later)))]), 0, starts[0], later, "portion")
        starts[0] += later
        live = list(range(len(seqs)))
        for k in range(max(extra)):
            ended = [b for b in live if k >= extra[b]]
            engine.release([slots[b] for b in ended])
            live = [b for b in live if b not in ended]
            if not live:
                break
            logits = engine.step([Entry(slots[b], [seqs[b][starts[b] + k]], [0]) for b in live])
            for row, b in enumerate(live):
                check(logits[row:row + 1], b, starts[b] + k, 1, ("step", k))
        engine.release([slots[b] for b in live])
        engine.cache.check()
        engine.check()
