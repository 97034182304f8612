"""Randomly drawn tiny Renapel configurations (seeded): any order of the three mixers, one to six streams and none, widths
that the 16-byte paths take and widths they do not, head, latent and value sizes that the tensor-core kernels take and
sizes no tile takes, groups of 1 to 10 heads, bias tables of 2 to 64 rows with far and near last distances, temperatures or
none, keys read from any earlier attention of the same sizes, decays from 0 to 1, states with fewer and more rows than
columns, one to all of 1 to 40 experts from one to all of their groups, layers without. Each runs a batch of unequal prompts,
a later portion of one of them, and then decodes, shorter requests leaving earlier, in 32-bit and in bfloat16, against the
plain implementation."""
import math
import random

import pytest
import torch

import plain_renapel as plain
from test_zemozen_random_gpu import close
from tiny_renapel import random_weights, write_folder

pytestmark = pytest.mark.gpu

DEV = "cuda:0"
MARGIN = 0.006          # of softmax scores: what bfloat16 rounding of the router's input reaches


def draw_config(rng):
    """(configuration, rows of the bias table by layer)"""
    width = rng.choice([36, 48, 64, 100, 136, 160, 260, 320])

    def attention():
        kv = rng.choice([1, 2, 3, 4])
        dim = rng.choice([8, 10, 16, 24, 32, 48, 64, 64, 96, 128])
        out = {"heads": kv * rng.choice([1, 2, 3, 10] if kv < 3 else [1, 2]), "kv_heads": kv, "dim": dim,
               "vdim": rng.choice([dim, dim, dim, 8, 20, 72]), "scale": rng.choice([1.0 / math.sqrt(dim), 0.13])}
        return around(out)

    def around(mixer):
        """What a layer that reads another's keys has of its own."""
        mixer.pop("q_temp", None)
        mixer["bias_max"] = rng.choice([33, 40, 64, 100, 128, 1000, 77.5])
        if rng.random() < 0.7:
            mixer["q_temp"] = {"coef": rng.choice([0.1, 0.5, 1.0]), "every": rng.choice([1, 7, 64, 100])}
        return mixer

    def latent():
        dim, rot_dim = rng.choice([8, 10, 16, 32, 64, 64, 128]), rng.choice([2, 4, 8, 16, 24, 32, 64])
        return {"heads": rng.choice([1, 2, 5, 8, 17, 24, 40]), "dim": dim, "rot_dim": rot_dim, "vdim": rng.choice([dim, 8, 20, 64, 128]),
                "kv_rank": rng.choice([12, 24, 40, 64, 64, 96, 128, 160, 256, 300]), "q_rank": rng.choice([7, 24, 64, 100, 136]),
                "rot": {"base": rng.choice([100.0, 10000.0, 5e5]), "dims": rot_dim}, "scale": rng.choice([1.0 / math.sqrt(dim + rot_dim), 0.09])}

    def lightning():
        heads = rng.choice([1, 2, 3, 6])
        return {"heads": heads, "dim": rng.choice([4, 7, 16, 33, 40, 64, 100, 128, 140]), "vdim": rng.choice([4, 6, 16, 36, 64, 130]),
                "decay": [rng.choice([0.0, 0.3, 0.8, 0.97, 0.9995]) for _ in range(heads)]}

    def feed_forward():
        if rng.random() < 0.15:
            return None
        count = rng.choice([1, 1, 2, 3, 4])
        size = rng.choice([1, 2, 3, 8, 10])
        keep = rng.choice([1, count, max(1, count - 1)])
        top = min(keep * size, rng.choice([1, 2, 4, keep * size if keep * size <= 8 else 6]))
        router = {"experts": count * size, "top": top, "scale": rng.choice([1.0, 0.4, 2.5])}
        if count > 1 or rng.random() < 0.5:
            router["groups"] = {"count": count, "keep": keep}
        return {"kind": "moe", "router": router, "expert": {"ff": rng.choice([8, 20, 32, 64, 72, 96]), "limit": rng.choice([0.5, 1.0, 7.0])}}

    layers, rows = [], {}
    for i in range(rng.choice([1, 2, 3, 4, 5])):
        kind = rng.choice(["attention", "attention", "latent_attention", "lightning"])
        mixer = {"attention": attention, "latent_attention": latent, "lightning": lightning}[kind]()
        owners = [j for j in range(i) if layers[j]["type"] == "attention" and "kv_from" not in layers[j]["mixer"]]
        if kind == "attention":
            if owners and rng.random() < 0.6:
                j = rng.choice(owners)
                mixer = around(dict(layers[j]["mixer"]))
                mixer["kv_from"] = j
            rows[i] = rng.choice([2, 5, 8, 16, 32, 33, 64])
        layers.append({"type": kind, "mixer": mixer, "mlp": feed_forward()})
    config = {"architecture": "Renapel", "vocab": rng.choice([61, 128, 300, 1000]), "width": width,
              "norm": {"eps": rng.choice([1e-5, 1e-6, 1e-3])}, "layers": layers}
    streams = rng.choice([1, 2, 3, 4, 4, 5, 6, None])
    if streams is not None:
        config["streams"] = streams
    return config, rows


@pytest.mark.parametrize("case", range(200, 236))
def test_random_configuration(tmp_path, case):
    from llm_b200.engine import Engine, Entry, load_model
    rng = random.Random(73100 + case)
    raw, rows = draw_config(rng)
    folder = write_folder(tmp_path / "model", raw, random_weights(raw, 700 + case, rows=rows))
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
